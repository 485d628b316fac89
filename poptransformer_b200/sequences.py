"""Decoders whose sequences have positions of their own: what they share besides their layers.

A model's class brings its weights (`_load`), the caches and states of its layers (`_alloc_layers`), its activation buffers
(`_row_buffers`) and its layers (`_layers`, `_head`).  This base runs them in two ways over the same kernels, caches and weights.
The decode loop of the other models (`run`, `step`, `prefill`, `capture`): one id container, all rows at the same position, greedy.
And sequences with positions of their own (`open`, `extend`, `close`): each call takes the next tokens of any number of sequences
and returns logits."""
import contextlib
import copy
from types import SimpleNamespace

import numpy as np
import torch

from . import ops
from .cache import SequenceSlots
from .loop import DecodeLoop


class Weights:
    """Look-ups in a state dict with shape checks, on the decoder's device and in its element type."""

    def __init__(self, sd, device, dtype):
        self.sd, self.device, self.dtype = sd, device, dtype

    def __contains__(self, key):
        return key in self.sd

    def _get(self, key, shape):
        if key not in self.sd:
            raise ops.PtError(f"{key}: no such tensor")
        t = self.sd[key]
        if tuple(t.shape) != tuple(shape):
            raise ops.PtError(f"{key}: shape {tuple(t.shape)}, expected {tuple(shape)}")
        return t.to(self.device)

    def f32(self, key, shape):
        return self._get(key, shape).to(torch.float32).contiguous()

    def mat(self, key, shape):
        return self._get(key, shape).to(self.dtype)

    def lin(self, keys, shapes, **kw):
        """One linear of several matrices with the same input, their outputs one after the other."""
        ws = [self.mat(k, s) for k, s in zip(keys, shapes)]
        return ops.DenseLinear(torch.cat(ws, 0) if len(ws) > 1 else ws[0], self.dtype, **kw)


class JointRows:
    """Matrices that read the same activations, gathered row by row into one linear."""

    def __init__(self, width, dtype, device):
        self.width, self.dtype, self.device, self.parts, self.biases, self.n = width, dtype, device, [], [], 0

    def add(self, rows, bias=None):
        """bias: fp32 [rows] (default zeros)."""
        self.parts.append(rows)
        self.biases.append(torch.zeros(len(rows), dtype=torch.float32, device=self.device) if bias is None else bias)
        self.n += len(rows)

    def column(self, multiple=8):
        """First column of what is added next: zero rows come before it up to a multiple (8: a 16-byte boundary)."""
        if self.n % multiple:
            self.add(torch.zeros((-self.n % multiple, self.width), dtype=self.dtype, device=self.device))
        return self.n

    def linear(self, biased=False, **kw):
        return ops.DenseLinear(torch.cat(self.parts, 0), self.dtype, bias=torch.cat(self.biases) if biased else None, **kw)


class SequenceDecoder(DecodeLoop):
    _side_stream = None
    PROMPT_TOKENS = 8192     # most packed prompt tokens of one pass (longer prompts go in portions)

    def __init__(self, cfg, state_dict, batch, device="cuda", dtype="bfloat16", page_size=64, pad_id=None, eos_id=-1, early_stop=False, n_pages=None,
                 plain=False):
        """batch: rows of the id container, and the most sequences that are open at a time.  n_pages: size of the page pool (default:
        max_len positions for every sequence, which the decode loop needs).  plain: use the any-size kernels even where the
        tensor-core ones apply (for comparisons)."""
        self.cfg, self.batch, self.device = cfg, batch, device
        self.dtype = {"bfloat16": torch.bfloat16, "float32": torch.float32}[dtype] if isinstance(dtype, str) else dtype
        self.pad_id, self.eos_id, self.plain = (cfg.vocab - 1 if pad_id is None else pad_id), eos_id, bool(plain)
        self._init_loop(device, early_stop)
        self._state_opts = dict(page_size=page_size, n_pages=n_pages)
        self._load(Weights(state_dict, device, self.dtype))
        self._alloc_state()

    # ---- what a model brings ----------------------------------------------------------------------
    def _load(self, w):
        raise NotImplementedError

    def _alloc_layers(self):
        """Caches and recurrent states of all layers, for self.batch slots."""
        raise NotImplementedError

    def _row_buffers(self, rows):
        """Activation buffers for up to `rows` packed tokens (an object with `rows`)."""
        raise NotImplementedError

    def _layers(self, r, view, longest, ids, ids_ld=1, step=None, pos_out=None, layer_sums=None):
        """All layers over the packed tokens of `view` (`longest`: most tokens of one sequence), up to the last sublayer's output."""
        raise NotImplementedError

    def _head(self, r, n, out, row_index=None, layer_sums=None, n_tok=0):
        """Logits of `n` rows (all of them, or the ones row_index names) after `_layers`."""
        raise NotImplementedError

    def _linear_workspaces(self, r, rows, linears):
        r.lin_ws = r.gemm_ws = None
        if self.dtype == torch.bfloat16:
            L = ops._lib.lib()
            n = max(L.pt_linear_workspace_bytes(min(rows, x.skinny_rows), x.n_out, max(16, x.ld // 256)) for x in linears)     # at least 256 k per slice
            r.lin_ws = torch.zeros(n, dtype=torch.uint8, device=self.device)
            if rows > ops.DenseLinear.SKINNY_ROWS:   # k-slices only while there are fewer tiles than SMs: 40 MB hold every such product's
                n = min(max(L.pt_gemm_workspace_bytes(rows, x.n_out, 8) for x in linears), (40 << 20) + 65536)
                r.gemm_ws = torch.zeros(n, dtype=torch.uint8, device=self.device)

    def _attn_workspace(self, shapes):
        """shapes: (heads, value width, window, kept first tokens) of the attention layers."""
        if not shapes:
            return None
        n = max(ops._lib.lib().pt_window_attn_workspace_bytes(self.batch, h, v, self._state_opts["page_size"], self.cfg.max_len, w, k) for h, v, w, k in shapes)
        return torch.zeros(n, dtype=torch.uint8, device=self.device)

    # ---- state ----------------------------------------------------------------------------------
    def new_stream(self):
        """A second decode stream over the same weights: its own id container, slots, caches, recurrent state and CUDA graph."""
        s = copy.copy(self)
        s._init_loop(self.device, self.early_stop)
        s._alloc_state()
        return s

    def resize(self, batch, n_pages=None):
        """Rebuilds the state for another number of sequences (and size of the page pool); none may be open."""
        if self.slots.length and not self._loop_rows:
            raise ops.PtError("resize: sequences are open")
        self.batch, self._state_opts["n_pages"] = batch, n_pages
        self._alloc_state()

    def _alloc_state(self):
        c, dev, B = self.cfg, self.device, self.batch
        i32 = dict(dtype=torch.int32, device=dev)
        self.slots = SequenceSlots(B, c.max_len, self._state_opts["page_size"], self._state_opts["n_pages"], dev)
        self._alloc_layers()
        self.ids = torch.full((B, c.max_len), self.pad_id, **i32)
        self.step_t, self.stop_mask = torch.zeros(1, **i32), torch.zeros(B, **i32)
        self.error_flag = torch.zeros(1, **i32)
        self.pos = torch.zeros(B, **i32)
        self.row = torch.arange(B + 1, **i32)
        self.next_val, self.next_ids = torch.empty((B, 1), dtype=torch.float32, device=dev), torch.empty((B, 1), **i32)
        self.rows_decode = self._row_buffers(B)
        self.rows_prompt = None
        self.logits = torch.empty((B, c.vocab), dtype=torch.float32, device=dev)
        self.graph = None
        self._loop_rows = False
        torch.cuda.synchronize()

    def _linear(self, lin, x, out, rows, out_ld, r, **kw):
        lin(x, out, rows, out_ld, linear_ws=r.lin_ws, gemm_ws=r.gemm_ws, error_flag=self.error_flag, **kw)

    @contextlib.contextmanager
    def _beside(self):
        """What is launched inside runs beside what follows on the current stream, until `_join`.  (In a captured graph: a branch.)"""
        if self._side_stream is None:
            self._side_stream = torch.cuda.Stream(self.device)
        self._side_stream.wait_stream(torch.cuda.current_stream())
        with torch.cuda.stream(self._side_stream):
            yield

    def _join(self):
        torch.cuda.current_stream().wait_stream(self._side_stream)

    # ---- the decode loop ------------------------------------------------------------------------
    def _need_loop_rows(self):
        """Rows of the id container = slots 0 .. batch - 1 with all their pages."""
        if not self._loop_rows:
            self.slots.close_all()
            for b in range(self.batch):
                self.slots.extend(self.slots.open(), self.cfg.max_len)
            self._loop_rows = True

    def reset(self, input_ids):
        """input_ids int32 [batch, max_len] (host or device), right-padded with pad_id; step <- 0."""
        self._need_loop_rows()
        self.ids.copy_(torch.as_tensor(input_ids, dtype=torch.int32).to(self.device, non_blocking=True))
        self.step_t.zero_()
        self.stop_mask.zero_()

    def capture(self):
        """Captures one loop iteration in a CUDA graph.  The recurrent state is that of the running generation: call before `reset`."""
        self._need_loop_rows()
        super().capture()

    def enqueue_step(self):
        c, B, L_ = self.cfg, self.batch, ops._lib.lib()
        view = ops.batch_view(B, B, self.row, self.pos, self.row, self.row)
        self._layers(self.rows_decode, view, 1, self.ids, ids_ld=c.max_len, step=self.step_t, pos_out=self.pos)
        self._head(self.rows_decode, B, self.logits)
        ops.check(L_.pt_topk(ops._ptr(self.logits), B, c.vocab, 1, ops.DT_F32, ops._ptr(self.next_val), ops._ptr(self.next_ids), ops._stream()), "topk")
        ops.step_containers(self.ids, self.step_t, self.next_ids, self.pad_id, self.eos_id, self.stop_mask, done_flag=self._loop_done_flag())

    def step(self):
        if self.graph is not None:
            self.graph.replay()
        else:
            self.enqueue_step()

    def prefill(self, n_tokens=None, chunk=1024):
        """Ingests the first `n_tokens` positions of every row in passes of at most `chunk` positions instead of one loop iteration
        per token (default: one less than the shortest prompt); the next `step()` is loop iteration `n_tokens`.  Call right after
        `reset()`.  Returns the number of positions ingested."""
        c, B = self.cfg, self.batch
        if n_tokens is None:
            n_tokens = int((self.ids != self.pad_id).to(torch.int32).cumprod(1).sum(1).min().item()) - 1
        n = int(n_tokens)
        if n <= 0:
            return 0
        if n >= c.max_len:
            raise ops.PtError(f"prefill: n_tokens={n} leaves no decode position (max_len={c.max_len})")
        ids = self.ids[:, :n].cpu().numpy()
        for s0 in range(0, n, chunk):
            part = [(b, ids[b, s0:s0 + chunk], s0, []) for b in range(B)]
            for p in self._passes(part):
                self._run_pass(p)
        self.step_t.fill_(n)
        if self.eos_id >= 0:      # the stop mask the loop would have built: it looks at the id one position ahead
            self.stop_mask |= (self.ids[:, 1:n + 1] == self.eos_id).any(1).to(torch.int32)
        return n

    # ---- sequences with positions of their own ----------------------------------------------------
    def open(self):
        """A new sequence; returns its handle."""
        if self._loop_rows:
            self.slots.close_all()
            self._loop_rows = False
        return self.slots.open()

    def close(self, seq):
        """Ends a sequence and returns its slot and pages."""
        self.slots.close(seq)

    def extend(self, entries, layer_sums=None):
        """The next tokens of some sequences as one batch.  entries: [(handle, token ids, wanted places)]; a place counts from the
        first of the entry's tokens.  Returns fp32 logits [wanted places in the order of the entries, vocab] on the device."""
        c = self.cfg
        out = torch.empty((sum(len(w) for _, _, w in entries), c.vocab), dtype=torch.float32, device=self.device)
        parts, row = [], 0
        for seq, tokens, want in entries:
            tokens = np.asarray(tokens, dtype=np.int32)
            if tokens.ndim != 1 or not tokens.size or tokens.min() < 0 or tokens.max() >= c.vocab:
                raise ops.PtError("extend: an entry needs token ids inside the vocabulary")
            if any(w < 0 or w >= tokens.size for w in want):
                raise ops.PtError("extend: a wanted place is outside the entry's tokens")
            parts.append((seq, tokens, self.slots.extend(seq, tokens.size), [(w, row + k) for k, w in enumerate(want)]))
            row += len(want)
        for p in self._passes(parts):
            self._run_pass(p, out, layer_sums)
        if int(self.error_flag.item()):
            raise ops.PtError(f"device-side error flag {int(self.error_flag.item())}")
        return out

    def _passes(self, parts):
        """Cuts [(slot, tokens, start, [(place, output row)])] into passes of at most PROMPT_TOKENS packed tokens."""
        cur, room = [], self.PROMPT_TOKENS
        for slot, tokens, start, want in parts:
            at = 0
            while at < len(tokens):
                if room == 0:
                    yield cur
                    cur, room = [], self.PROMPT_TOKENS
                k = min(room, len(tokens) - at)
                cur.append((slot, tokens[at:at + k], start + at, [(w - at, o) for w, o in want if at <= w < at + k]))
                room -= k
                at += k
        if cur:
            yield cur

    def _run_pass(self, part, out=None, layer_sums=None):
        n_seq, lens = len(part), [len(t) for _, t, _, _ in part]
        n = sum(lens)
        cu = np.concatenate([[0], np.cumsum(lens)]).astype(np.int32)
        rows = [cu[s] + w for s, (_, _, _, want) in enumerate(part) for w, _ in want]
        dest = [o for _, _, _, want in part for _, o in want]
        ctx = np.concatenate([[0], np.cumsum([s + n for (_, _, s, _), n in zip(part, lens)])])      # all positions so far, sequence after sequence
        fields = [np.concatenate([t for _, t, _, _ in part]), np.repeat(np.arange(n_seq), lens), cu, [s for _, _, s, _ in part], [s for s, _, _, _ in part],
                  rows, dest, ctx]
        sizes = [ops.pad_to(len(f), 4) for f in fields]              # every array on a 16-byte boundary of one upload
        host = np.zeros(sum(sizes), dtype=np.int32)
        at = np.concatenate([[0], np.cumsum(sizes)])
        for f, a in zip(fields, at):
            host[a:a + len(f)] = f
        dev = torch.from_numpy(host).to(self.device)
        ids, tok_seq, cu_d, start, slot, rows_d, dest_d, ctx_d = (dev[a:a + len(f)] for f, a in zip(fields, at))
        if n <= self.rows_decode.rows:
            r = self.rows_decode
        else:
            if self.rows_prompt is None or self.rows_prompt.rows < n:
                self.rows_prompt = None
                self.rows_prompt = self._row_buffers(n)
            r = self.rows_prompt
        view = ops.batch_view(n_seq, n, cu_d, start, slot, tok_seq)
        view.ctx_cu, view.n_ctx = ctx_d, int(ctx[-1])
        self._layers(r, view, max(lens), ids, layer_sums=layer_sums)
        k = len(rows)
        logits = torch.empty((k, self.cfg.vocab), dtype=torch.float32, device=self.device) if k else None
        self._head(r, k, logits, row_index=rows_d if k else None, layer_sums=layer_sums, n_tok=n)
        if k:
            out[dest_d.long()] = logits
