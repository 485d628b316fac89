"""Sabisun: a small hybrid decoder (attention and state-space layers in any order) with hyper-connected residual streams.

Per layer, twice (mixer, feed-forward): the sublayer reads a learned combination of `streams` fp32 residual streams, RMS-normalises
it, and its output is written back to all streams together with a learned mixing of the streams (csrc/hyper.cu).
  attention   grouped heads with key / value widths of their own, a sliding window with kept first tokens, a softmax sink, no
              rotation; a layer with `kv_from` has only queries and reads the named layer's cache (csrc/window_attn.cu)
  mamba2      input projection -> causal convolution -> matrix-state recurrence -> gate -> group norm (csrc/ssm.cu)
  dense       W_down relu(W_up h)^2
The output layer is the embedding table, with a factor on the logits.

Every size and constant comes from the configuration; layers may differ in all of them.  dtype bfloat16: matrix products and
their inputs are bfloat16, accumulation, residual streams, norms, softmax, recurrent state and what enters it are float32.
float32: everything is true 32-bit.

The decoder runs in two ways over the same kernels, caches and weights.  The decode loop of the other models (`run`, `step`,
`prefill`, `capture`): one id container, all rows at the same position, greedy.  And sequences with positions of their own
(`open`, `extend`, `close`): each call takes the next tokens of any number of sequences and returns logits."""
import copy
from types import SimpleNamespace

import numpy as np
import torch

from . import ops
from .cache import SequenceSlots
from .loop import DecodeLoop


class SabisunConfig:
    """The parsed config.json plus the longest sequence the decoder is built for."""

    def __init__(self, config, max_len):
        self.max_len = int(max_len)
        self.vocab, self.width, self.streams = int(config["vocab"]), int(config["width"]), int(config.get("streams", 1))
        self.eps = float(config["norm"]["eps"])
        self.residual_mult, self.logit_scale = float(config.get("residual_mult", 1.0)), float(config.get("logit_scale", 1.0))
        self.layers = []
        for i, lay in enumerate(config["layers"]):
            m = lay["mixer"]
            if lay["type"] == "attention":
                mask = m.get("mask") or {}
                mixer = SimpleNamespace(kind="attention", heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                                        scale=float(m["scale"]), window=int(mask.get("size", 0)), keep_first=int(mask.get("keep_first", 0)),
                                        kv_from=m.get("kv_from"))
                if mixer.kv_from is not None:
                    src = self.layers[mixer.kv_from].mixer if 0 <= mixer.kv_from < i else None
                    if src is None or src.kind != "attention" or src.kv_from is not None or (src.kv_heads, src.dim, src.vdim) != (
                            mixer.kv_heads, mixer.dim, mixer.vdim):
                        raise ops.PtError(f"layer {i}: kv_from={mixer.kv_from} is not an earlier attention layer with keys of the same shape")
                if mixer.heads % mixer.kv_heads:
                    raise ops.PtError(f"layer {i}: {mixer.heads} heads do not divide over {mixer.kv_heads} key/value heads")
            elif lay["type"] == "mamba2":
                mixer = SimpleNamespace(kind="mamba2", heads=int(m["heads"]), vdim=int(m["vdim"]), state=int(m["state"]), groups=int(m["groups"]),
                                        taps=int(m["conv"]), norm_groups=int(m["norm_groups"]))
                mixer.inner = mixer.heads * mixer.vdim
                mixer.channels = mixer.inner + 2 * mixer.groups * mixer.state
                mixer.proj = mixer.inner + mixer.channels + mixer.heads
                if mixer.heads % mixer.groups or mixer.inner % mixer.norm_groups:
                    raise ops.PtError(f"layer {i}: {mixer.heads} heads / {mixer.groups} groups / {mixer.norm_groups} norm groups do not divide evenly")
            else:
                raise ops.PtError(f"layer {i}: unknown mixer {lay['type']!r}")
            mlp = lay.get("mlp")
            if mlp is not None and mlp.get("kind", "dense") != "dense":
                raise ops.PtError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
            self.layers.append(SimpleNamespace(mixer=mixer, ff=int(mlp["ff"]) if mlp is not None else 0))


class SabisunDecoder(DecodeLoop):
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
        self._load(state_dict)
        self._alloc_state()

    # ---- weights --------------------------------------------------------------------------------
    def _load(self, sd):
        c, dt = self.cfg, self.dtype

        def f32(key, shape):
            t = sd[key].to(self.device).to(torch.float32).contiguous()
            if tuple(t.shape) != shape:
                raise ops.PtError(f"{key}: shape {tuple(t.shape)}, expected {shape}")
            return t

        def lin(keys, shapes, **kw):
            ws = []
            for k, s in zip(keys, shapes):
                if tuple(sd[k].shape) != s:
                    raise ops.PtError(f"{k}: shape {tuple(sd[k].shape)}, expected {s}")
                ws.append(sd[k].to(self.device).to(dt))
            return ops.DenseLinear(torch.cat(ws, 0) if len(ws) > 1 else ws[0], dt, **kw)

        def hyper(p, q):
            s = c.streams
            if p + f"hc{q}.in" not in sd and s == 1:
                one = torch.ones(1, dtype=torch.float32, device=self.device)
                return SimpleNamespace(w_in=one, w_out=one, mix=one.view(1, 1))
            return SimpleNamespace(w_in=f32(p + f"hc{q}.in", (s,)), w_out=f32(p + f"hc{q}.out", (s,)), mix=f32(p + f"hc{q}.mix", (s, s)))

        W = c.width
        self.head = lin(["embed"], [(c.vocab, W)], keep=True)     # also the look-up table (rows padded like the head's k)
        self.table = self.head.w
        self.final_norm = f32("final.norm", (W,))
        self.subs = []                                                # sublayers in order: mixer, feed-forward, mixer, ...
        for i, lay in enumerate(c.layers):
            p, m = f"l{i}.", lay.mixer
            sub = SimpleNamespace(kind=m.kind, layer=i, m=m, norm=f32(p + "norm1", (W,)), hc=hyper(p, 1))
            if m.kind == "attention":
                keys, shapes = [p + "mix.q"], [(m.heads * m.dim, W)]
                if m.kv_from is None:
                    keys += [p + "mix.k", p + "mix.v"]
                    shapes += [(m.kv_heads * m.dim, W), (m.kv_heads * m.vdim, W)]
                sub.proj = lin(keys, shapes)
                sub.sink = f32(p + "mix.sink", (m.heads,)) if p + "mix.sink" in sd else None
                sub.out = lin([p + "mix.o"], [(W, m.heads * m.vdim)])
            else:
                sub.proj = lin([p + "mix.in"], [(m.proj, W)])
                sub.out = lin([p + "mix.o"], [(W, m.inner)])
                sub.w = SimpleNamespace(heads=m.heads, vdim=m.vdim, state=m.state, groups=m.groups, taps=m.taps, norm_groups=m.norm_groups, eps=c.eps,
                                        conv_w=f32(p + "mix.conv", (m.channels, m.taps)), conv_b=f32(p + "mix.conv.b", (m.channels,)),
                                        dt_bias=f32(p + "mix.dt_bias", (m.heads,)), A_log=f32(p + "mix.A_log", (m.heads,)), D=f32(p + "mix.D", (m.heads,)),
                                        norm_w=f32(p + "mix.norm", (m.inner,)))
            sub.ld = ops.pad_to(sub.proj.n_out, 8)                    # row stride of the projection's output
            self.subs.append(sub)
            if lay.ff:
                up_rows = ops.pad_to(lay.ff, ops.DenseLinear.K_PAD) if dt == torch.bfloat16 else lay.ff
                ff = SimpleNamespace(kind="dense", layer=i, norm=f32(p + "norm2", (W,)), hc=hyper(p, 2), proj=lin([p + "mlp.up"], [(lay.ff, W)], pad_rows=up_rows),
                                     out=lin([p + "mlp.down"], [(W, lay.ff)]))
                ff.ld = ff.out.ld
                self.subs.append(ff)

    def weight_bytes(self):
        """Algorithmic weight bytes one decode step streams (every linear once)."""
        return sum(s.proj.nbytes + s.out.nbytes for s in self.subs) + self.head.nbytes

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
        c, dev, B, dt = self.cfg, self.device, self.batch, self.dtype
        page_size, n_pages = self._state_opts["page_size"], self._state_opts["n_pages"]
        i32 = dict(dtype=torch.int32, device=dev)
        self.slots = SequenceSlots(B, c.max_len, page_size, n_pages, dev)
        self.caches, self.rings, self.states = {}, {}, {}
        for i, lay in enumerate(c.layers):
            m = lay.mixer
            if m.kind == "mamba2":
                self.rings[i] = torch.zeros((B, m.taps, m.channels), dtype=dt, device=dev)
                self.states[i] = torch.zeros((B, m.heads, m.state, m.vdim), dtype=torch.float32, device=dev)
            elif m.kv_from is None:
                self.caches[i] = ops.PagedKVCache(B, m.kv_heads, m.dim, c.max_len, page_size, dev, self.slots.page_table, v_dim=m.vdim, dtype=dt,
                                                  n_pages=self.slots.n_pages)
            else:
                self.caches[i] = self.caches[m.kv_from]
        self.ids = torch.full((B, c.max_len), self.pad_id, **i32)
        self.step_t, self.stop_mask = torch.zeros(1, **i32), torch.zeros(B, **i32)
        self.error_flag = torch.zeros(1, **i32)
        self.pos = torch.zeros(B, **i32)
        self.row = torch.arange(B + 1, **i32)
        self.next_val, self.next_ids = torch.empty((B, 1), dtype=torch.float32, device=dev), torch.empty((B, 1), **i32)
        self.rows_decode = self._row_buffers(B)
        self.rows_prompt = None
        self.logits = torch.empty((B, c.vocab), dtype=torch.float32, device=dev)
        sizes = [(s.m.heads, s.m.vdim, s.m.window, s.m.keep_first) for s in self.subs if s.kind == "attention"]
        self.attn_ws = None
        if sizes:
            n = max(ops._lib.lib().pt_window_attn_workspace_bytes(B, h, v, page_size, c.max_len, w, k) for h, v, w, k in sizes)
            self.attn_ws = torch.zeros(n, dtype=torch.uint8, device=dev)
        self.graph = None
        self._loop_rows = False
        torch.cuda.synchronize()

    def _row_buffers(self, rows):
        """Activation buffers for up to `rows` packed tokens."""
        c, dev, dt = self.cfg, self.device, self.dtype
        f32 = dict(dtype=torch.float32, device=dev)
        r = SimpleNamespace(rows=rows)
        r.xs = torch.empty((rows, c.streams, c.width), **f32)
        r.h = torch.empty(rows * max(self.head.ld, *(s.proj.ld for s in self.subs)), dtype=dt, device=dev)
        r.a = torch.empty(rows * max(s.ld for s in self.subs), dtype=dt, device=dev)           # projection outputs
        r.b = torch.empty(rows * max(s.out.ld for s in self.subs), dtype=dt, device=dev)       # mixer outputs
        r.y = torch.empty((rows, c.width), **f32)                                              # sublayer outputs
        mm = [s.m for s in self.subs if s.kind == "mamba2"]
        r.xbc = torch.empty(rows * max((m.channels for m in mm), default=1), dtype=dt, device=dev)
        r.dt = torch.empty(rows * max((m.heads for m in mm), default=1), **f32)
        r.yin = torch.empty(rows * max((m.inner for m in mm), default=1), **f32)
        r.lin_ws = r.gemm_ws = r.ssm_ws = None
        if dt == torch.bfloat16:
            L = ops._lib.lib()
            lins = [self.head] + [x for s in self.subs for x in (s.proj, s.out)]
            skinny = min(rows, ops.DenseLinear.SKINNY_ROWS)
            n = max(L.pt_linear_workspace_bytes(skinny, x.n_out, max(16, x.ld // 256)) for x in lins)     # at least 256 k per slice
            r.lin_ws = torch.zeros(n, dtype=torch.uint8, device=dev)
            if rows > ops.DenseLinear.SKINNY_ROWS:   # k-slices only while there are fewer tiles than SMs: 40 MB hold every such product's
                n = min(max(L.pt_gemm_workspace_bytes(rows, x.n_out, 8) for x in lins), (40 << 20) + 65536)
                r.gemm_ws = torch.zeros(n, dtype=torch.uint8, device=dev)
            if mm:
                n = max(L.pt_ssm_workspace_bytes(rows, min(self.batch, rows), m.heads, m.vdim, m.state) for m in mm)
                r.ssm_ws = torch.empty(n, dtype=torch.uint8, device=dev)
        return r

    # ---- the layers -----------------------------------------------------------------------------
    def _linear(self, lin, x, out, rows, out_ld, r, **kw):
        lin(x, out, rows, out_ld, linear_ws=r.lin_ws, gemm_ws=r.gemm_ws, error_flag=self.error_flag, **kw)

    def _layers(self, r, view, longest, ids, ids_ld=1, step=None, pos_out=None, layer_sums=None):
        """All layers over the packed tokens of `view` (`longest`: most tokens of one sequence).  Leaves the streams before the last
        sublayer's write in r.xs and that sublayer's output in r.y; `_head` finishes."""
        c, n = self.cfg, view.n_tok
        first = self.subs[0]
        ops.hyper(r.xs, n, c.eps, norm_w=first.norm, h=r.h, h_ld=first.proj.ld, w_in=first.hc.w_in, table=self.table, vocab=c.vocab, ids=ids, ids_ld=ids_ld,
                  step=step, pos_out=pos_out)
        for k, s in enumerate(self.subs):
            if k:
                prev = self.subs[k - 1]
                sums = None
                if layer_sums is not None and prev.layer != s.layer:
                    sums = torch.empty((n, c.width), dtype=torch.float32, device=self.device)
                    layer_sums.append(sums)
                ops.hyper(r.xs, n, c.eps, norm_w=s.norm, h=r.h, h_ld=s.proj.ld, w_in=s.hc.w_in, y=r.y, y_ld=c.width, mix=prev.hc.mix, w_out=prev.hc.w_out,
                          mult=c.residual_mult, sum_out=sums)
            if s.kind == "dense":
                self._linear(s.proj, r.h, r.a, n, s.ld, r, epilogue=ops.EPI_RELU2)
                self._linear(s.out, r.a, r.y, n, c.width, r)
                continue
            self._linear(s.proj, r.h, r.a, n, s.ld, r)
            if s.kind == "attention":
                m = s.m
                ops.window_attn(view, r.a, s.ld, self.caches[s.layer], r.b, s.out.ld, m.heads, m.scale, m.window, m.keep_first, s.sink,
                                append=m.kv_from is None, max_tokens_per_seq=longest, workspace=self.attn_ws, error_flag=self.error_flag, plain=self.plain)
            else:
                ops.ssm(view, r.a, s.ld, r.b, s.out.ld, s.w, self.rings[s.layer], self.states[s.layer], r.yin, r.xbc, r.dt, r.ssm_ws,
                        plain=self.plain)
            self._linear(s.out, r.b, r.y, n, c.width, r)

    def _head(self, r, n, out, row_index=None, layer_sums=None, n_tok=0):
        """Logits of `n` rows (all of them, or the ones row_index names) after `_layers`."""
        c, last = self.cfg, self.subs[-1]
        kw = dict(y=r.y, y_ld=c.width, mix=last.hc.mix, w_out=last.hc.w_out, mult=c.residual_mult)
        if layer_sums is not None:
            layer_sums.append(torch.empty((n_tok, c.width), dtype=torch.float32, device=self.device))
            ops.hyper(r.xs, n_tok, c.eps, sum_out=layer_sums[-1], **kw)
        if n:
            ops.hyper(r.xs, n, c.eps, norm_w=self.final_norm, h=r.h, h_ld=self.head.ld, row_index=row_index, **kw)
            self._linear(self.head, r.h, out, n, c.vocab, r, alpha=c.logit_scale)

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
        fields = [np.concatenate([t for _, t, _, _ in part]), np.repeat(np.arange(n_seq), lens), cu, [s for _, _, s, _ in part], [s for s, _, _, _ in part],
                  rows, dest]
        sizes = [ops.pad_to(len(f), 4) for f in fields]              # every array on a 16-byte boundary of one upload
        host = np.zeros(sum(sizes), dtype=np.int32)
        at = np.concatenate([[0], np.cumsum(sizes)])
        for f, a in zip(fields, at):
            host[a:a + len(f)] = f
        dev = torch.from_numpy(host).to(self.device)
        ids, tok_seq, cu_d, start, slot, rows_d, dest_d = (dev[a:a + len(f)] for f, a in zip(fields, at))
        if n <= self.rows_decode.rows:
            r = self.rows_decode
        else:
            if self.rows_prompt is None or self.rows_prompt.rows < n:
                self.rows_prompt = None
                self.rows_prompt = self._row_buffers(n)
            r = self.rows_prompt
        self._layers(r, ops.batch_view(n_seq, n, cu_d, start, slot, tok_seq), max(lens), ids, layer_sums=layer_sums)
        k = len(rows)
        logits = torch.empty((k, self.cfg.vocab), dtype=torch.float32, device=self.device) if k else None
        self._head(r, k, logits, row_index=rows_d if k else None, layer_sums=layer_sums, n_tok=n)
        if k:
            out[dest_d.long()] = logits
