"""Padetar: a small decoder with two mixers side by side in every layer, experts, and a per-layer input from the token itself.

One fp32 residual stream; a sublayer reads it as it is, and its output is RMS-normalised before it is added (csrc/post_norm.cu).
Per layer:
  parallel    left_scale * attention + right_scale * matrix memory of the same input.  Attention: grouped heads whose values are the
              keys as projected, per-head norm of q and k, rotation with scaled frequencies (csrc/window_attn.cu).  Matrix memory: the
              mLSTM recurrence with capped exponential gates (csrc/mlstm.cu).
  moe         a router picks `top` of the experts (clamped gated units) per token, weights are the softmax over the chosen; a shared
              expert runs for every token (csrc/moe.cu and the grouped linears)
  side        the layer's part of a second embedding of the token, gated by the residual stream

The products of a sublayer that share their input are one linear: q, k and the memory's q, k, v, output gate and log gates; the
shared expert's gate and up rows and the router.  Log gates and router logits leave it in fp32.  The two mixers' output projections
are one linear over both mixers' outputs side by side, which carry left_scale and right_scale already.

Every size and constant comes from the configuration; layers may differ in all of them.  dtype bfloat16: matrix products and their
inputs are bfloat16, accumulation, residual stream, norms, rotation, softmax, router, gates and recurrent state are float32.
float32: everything is true 32-bit."""
import math
from types import SimpleNamespace

import numpy as np
import torch

from . import ops
from .experts import Experts
from .sequences import SequenceDecoder


def rope_frequencies(dims, base, scaling=None):
    """Radians per position of every pair, float64.  scaling: factor, low, high, original (the frequency bands of Llama 3.1)."""
    f = float(base) ** (-2.0 * np.arange(dims // 2) / dims)
    if scaling:
        wave = 2.0 * math.pi / f
        long, short = scaling["original"] / scaling["low"], scaling["original"] / scaling["high"]
        s = (scaling["original"] / wave - scaling["low"]) / (scaling["high"] - scaling["low"])
        f = np.where(wave < short, f, np.where(wave > long, f / scaling["factor"], (1.0 - s) * f / scaling["factor"] + s * f))
    return f


class PadetarConfig:
    """The parsed config.json plus the longest sequence the decoder is built for."""

    def __init__(self, config, max_len):
        self.max_len = int(max_len)
        self.vocab, self.width, self.eps = int(config["vocab"]), int(config["width"]), float(config["norm"]["eps"])
        self.side = int((config.get("token_side") or {}).get("dim", 0))
        self.layers = []
        for i, lay in enumerate(config["layers"]):
            if lay["type"] != "parallel":
                raise ops.PtError(f"layer {i}: unknown mixer {lay['type']!r}")
            m, mlp = lay["mixer"], lay.get("mlp")
            a, b = m["left"], m["right"]
            rot = a["rot"]
            sc = rot.get("scaling")
            left = SimpleNamespace(heads=int(a["heads"]), kv_heads=int(a["kv_heads"]), dim=int(a["dim"]), scale=float(a["scale"]), rot_dims=int(rot["dims"]),
                                   rot=(int(rot["dims"]), float(rot["base"]), tuple(float(sc[k]) for k in ("factor", "low", "high", "original")) if sc else None))
            if int(a.get("vdim", left.dim)) != left.dim:
                raise ops.PtError(f"layer {i}: values are keys, but vdim={a['vdim']} is not dim={left.dim}")
            if left.heads % left.kv_heads:
                raise ops.PtError(f"layer {i}: {left.heads} heads do not divide over {left.kv_heads} key/value heads")
            if left.rot_dims % 2 or not 0 <= left.rot_dims <= left.dim:
                raise ops.PtError(f"layer {i}: {left.rot_dims} rotated dimensions of {left.dim}")
            right = SimpleNamespace(heads=int(b["heads"]), dim=int(b["dim"]), vdim=int(b["vdim"]), cap=float(b["gate_cap"]))
            layer = SimpleNamespace(left=left, right=right, left_scale=float(m["left_scale"]), right_scale=float(m["right_scale"]), moe=None)
            if mlp is not None:
                if mlp.get("kind", "moe") != "moe":
                    raise ops.PtError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
                shared = mlp.get("shared")
                layer.moe = SimpleNamespace(experts=int(mlp["router"]["experts"]), top=int(mlp["router"]["top"]), ff=int(mlp["expert"]["ff"]),
                                            limit=float(mlp["expert"]["limit"]), shared_ff=int(shared["ff"]) if shared else 0,
                                            shared_limit=float(shared["limit"]) if shared else 0.0)
                if not 1 <= layer.moe.top <= layer.moe.experts:
                    raise ops.PtError(f"layer {i}: {layer.moe.top} of {layer.moe.experts} experts")
            self.layers.append(layer)


class PadetarDecoder(SequenceDecoder):
    # ---- weights --------------------------------------------------------------------------------
    def _load(self, w):
        c, dt, f32, mat = self.cfg, self.dtype, w.f32, w.mat
        W = c.width
        pad = ops.DenseLinear.K_PAD if dt == torch.bfloat16 else 16        # features of a gated product: the padded input of the next
        zeros = lambda rows, cols=W: torch.zeros((rows, cols), dtype=dt, device=self.device)

        def down(key, ff):
            full = zeros(W, ops.pad_to(ff, pad))
            full[:, :ff] = mat(key, (W, ff))
            return full

        self.table = mat("embed", (c.vocab, W)).contiguous()
        self.final_norm = f32("final.norm", (W,))
        self.head = w.lin(["head"], [(c.vocab, W)])
        self.h_ld = self.head.ld
        ropes = {}
        self.subs = []                                                # sublayers in order: mixer, experts, side input, mixer, ...
        for i, lay in enumerate(c.layers):
            p, a, b = f"l{i}.", lay.left, lay.right
            L, R = p + "mix.left.", p + "mix.right."
            # ---- the two mixers
            sub = SimpleNamespace(kind="mixer", layer=i, lay=lay, norm=f32(p + "norm1", (W,)))
            parts = [mat(L + "q", (a.heads * a.dim, W)), mat(L + "k", (a.kv_heads * a.dim, W))]
            left_cols = sum(len(x) for x in parts)
            parts.append(zeros(-left_cols % 8))
            sub.cols = []                                             # first columns of the memory's q, k, v and output gate
            for name, n in (("q", b.heads * b.dim), ("k", b.heads * b.dim), ("v", b.heads * b.vdim), ("g", b.heads * b.vdim)):
                sub.cols.append(sum(len(x) for x in parts))
                parts.append(mat(R + name, (n, W)))
            parts.append(zeros(-sum(len(x) for x in parts) % 32))
            split = sum(len(x) for x in parts)
            parts += [mat(R + n, (b.heads, W)) for n in ("i", "f")]
            bias = torch.zeros(split + 2 * b.heads, dtype=torch.float32, device=self.device)
            bias[:left_cols] = torch.cat([f32(L + "q.b", (a.heads * a.dim,)), f32(L + "k.b", (a.kv_heads * a.dim,))])
            bias[split:] = torch.cat([f32(R + n + ".b", (b.heads,)) for n in ("i", "f")])
            sub.proj = ops.DenseLinear(torch.cat(parts, 0), dt, bias=bias, split=split)
            sub.ld = ops.pad_to(split, 8)
            sub.q_norm, sub.k_norm = f32(L + "q.norm", (a.dim,)), f32(L + "k.norm", (a.dim,))
            if a.rot not in ropes:
                dims, base, sc = a.rot
                ang = np.arange(c.max_len)[:, None] * rope_frequencies(dims, base, dict(zip(("factor", "low", "high", "original"), sc)) if sc else None)
                ropes[a.rot] = torch.from_numpy(np.stack([np.cos(ang), np.sin(ang)], -1).astype(np.float32)).to(self.device) if dims else None
            sub.rope = ropes[a.rot]
            sub.mem = SimpleNamespace(heads=b.heads, dim=b.dim, vdim=b.vdim, cap=b.cap, eps=c.eps, norm_w=f32(R + "norm", (b.heads * b.vdim,)))
            sub.right_col = ops.pad_to(a.heads * a.dim, 8)            # the outputs of both mixers, side by side
            outs = [mat(L + "o", (W, a.heads * a.dim)), zeros(W, sub.right_col - a.heads * a.dim), mat(R + "o", (W, b.heads * b.vdim))]
            sub.out = ops.DenseLinear(torch.cat(outs, 1), dt, bias=lay.left_scale * f32(L + "o.b", (W,)))
            self.subs.append(sub)
            # ---- experts
            if lay.moe:
                m, M = lay.moe, p + "mlp."
                sub = SimpleNamespace(kind="moe", layer=i, m=m, norm=f32(p + "norm2", (W,)), sff=ops.pad_to(m.shared_ff, pad), down=None)
                rows = []
                if m.shared_ff:
                    rows.append(ops.glu_rows(*(mat(M + "shared." + n, (m.shared_ff, W)) for n in ("gate", "up")), sub.sff))
                    sub.down = ops.DenseLinear(down(M + "shared.down", m.shared_ff), dt)
                split = sum(len(x) for x in rows)
                bias = torch.zeros(split + m.experts, dtype=torch.float32, device=self.device)
                bias[split:] = f32(M + "router.b", (m.experts,))
                sub.proj = ops.DenseLinear(torch.cat(rows + [mat(M + "router", (m.experts, W))], 0), dt, bias=bias, split=split, limit=m.shared_limit)
                gates, ups = ([mat(M + f"e{e}." + n, (m.ff, W)) for e in range(m.experts)] for n in ("gate", "up"))
                sub.experts = Experts(dt, m.top, gates, ups, [mat(M + f"e{e}.down", (W, m.ff)) for e in range(m.experts)], limit=m.limit)
                self.subs.append(sub)
            # ---- side input
            if c.side:
                S = p + "side."
                sub = SimpleNamespace(kind="side", layer=i, norm=f32(S + "norm", (W,)), out=w.lin([S + "proj"], [(W, c.side)]))
                sub.ld = sub.out.ld
                sub.proj = w.lin([S + "gate"], [(c.side, W)], pad_rows=sub.ld)
                self.subs.append(sub)
        if c.side:      # [vocab, layers, side], every layer's part padded like the input of its projection
            self.side_ld = self.subs[-1].ld
            t = torch.zeros((c.vocab, len(c.layers), self.side_ld), dtype=dt, device=self.device)
            t[:, :, :c.side] = mat("side.embed", (c.vocab, len(c.layers) * c.side)).view(c.vocab, len(c.layers), c.side)
            self.side_table = t.view(c.vocab, -1)

    def _linears(self):
        return [self.head] + [x for s in self.subs for x in (s.proj, s.down if s.kind == "moe" else s.out) if x is not None]

    def expert_groups(self):
        return [s.experts for s in self.subs if s.kind == "moe"]

    def fixed_bytes(self):
        """Weight bytes that every decode step streams, whatever the experts."""
        return sum(x.nbytes for x in self._linears())

    def weight_bytes(self, rows=1):
        """Algorithmic weight bytes one decode step of `rows` tokens streams: every linear once, of the experts as many as the rows
        can choose at most."""
        return self.fixed_bytes() + sum(e.step_bytes(rows) for e in self.expert_groups())

    # ---- state ----------------------------------------------------------------------------------
    def _alloc_layers(self):
        c, dev, B = self.cfg, self.device, self.batch
        L, page_size = ops._lib.lib(), self._state_opts["page_size"]
        self.caches, self.states, self.norms = {}, {}, {}
        for i, lay in enumerate(c.layers):
            a, b = lay.left, lay.right
            self.caches[i] = ops.PagedKVCache(B, a.kv_heads, a.dim, c.max_len, page_size, dev, self.slots.page_table, dtype=self.dtype, n_pages=self.slots.n_pages)
            self.states[i], self.norms[i] = (torch.zeros((B, L.pt_mlstm_state_floats(b.heads, b.dim, b.vdim, k)), dtype=torch.float32, device=dev) for k in (0, 1))
        self.attn_ws = self._attn_workspace([(lay.left.heads, lay.left.dim, 0, 0) for lay in c.layers])

    def _row_buffers(self, rows):
        c, dev, dt = self.cfg, self.device, self.dtype
        f32, i32 = dict(dtype=torch.float32, device=dev), dict(dtype=torch.int32, device=dev)
        mixers, moes = [s for s in self.subs if s.kind == "mixer"], [s for s in self.subs if s.kind == "moe"]
        r = SimpleNamespace(rows=rows)
        r.x = torch.empty((rows, c.width), **f32)                                              # residual stream
        r.h = torch.empty(rows * self.h_ld, dtype=dt, device=dev)
        r.tok = torch.empty(rows, **i32)
        r.a = torch.empty(rows * max(s.sff if s.kind == "moe" else s.ld for s in self.subs), dtype=dt, device=dev)        # projection outputs
        r.b = torch.empty(rows * max(s.out.ld for s in mixers), dtype=dt, device=dev)          # mixer outputs
        r.y = torch.empty((rows, c.width), **f32)                                              # sublayer outputs
        r.o = torch.empty(rows * max(s.mem.heads * s.mem.vdim for s in mixers), **f32)
        r.gates = torch.empty(rows * max(2 * s.mem.heads for s in mixers), **f32)
        self._linear_workspaces(r, rows, self._linears())
        r.beside = SimpleNamespace(lin_ws=None, gemm_ws=None)                                  # of the shared expert, which runs beside the others
        if any(s.down for s in moes):
            self._linear_workspaces(r.beside, rows, [s.down for s in moes if s.down])
        L = ops._lib.lib()
        n = max(L.pt_mlstm_workspace_bytes(rows + 1, min(self.batch, rows), s.mem.heads, s.mem.dim, s.mem.vdim) for s in mixers)
        r.mem_ws = torch.zeros(n, dtype=torch.uint8, device=dev)
        if moes:
            Experts.buffers(r, rows, [s.experts for s in moes], self.h_ld, dev)
        return r

    # ---- the layers -----------------------------------------------------------------------------
    def _mixer(self, s, r, view, longest):
        n, lay, a = view.n_tok, s.lay, s.lay.left
        self._linear(s.proj, r.h, r.a, n, s.ld, r, out2=r.gates, out2_ld=2 * s.mem.heads, pdl=1)
        with self._beside():          # the two mixers read and write columns of their own
            ops.mlstm(view, r.a, s.ld, s.cols, r.gates, 2 * s.mem.heads, r.b[s.right_col:], s.out.ld, s.mem, self.states[s.layer], self.norms[s.layer], r.o, r.mem_ws,
                      out_scale=lay.right_scale, out_cols=s.out.ld - s.right_col, plain=self.plain)
        ops.window_attn(view, r.a, s.ld, self.caches[s.layer], r.b, s.out.ld, a.heads, a.scale, max_tokens_per_seq=longest, workspace=self.attn_ws,
                        error_flag=self.error_flag, plain=self.plain, values_are_keys=True, q_norm=s.q_norm, k_norm=s.k_norm, eps=self.cfg.eps, rope=s.rope,
                        rope_dims=a.rot_dims, out_scale=lay.left_scale, out_cols=s.right_col)
        self._join()
        self._linear(s.out, r.b, r.y, n, self.cfg.width, r)
        return dict(y=r.y, y_ld=self.cfg.width)

    def _experts(self, s, r, view, longest):
        n, m, W = view.n_tok, s.m, self.cfg.width
        self._linear(s.proj, r.h, r.a, n, s.sff, r, epilogue=ops.EPI_GLU if s.down else ops.EPI_STORE, out2=r.logits, out2_ld=m.experts, pdl=1)
        if s.down:
            with self._beside():
                self._linear(s.down, r.a, r.y, n, W, r.beside)
        pairs = s.experts(r, n, self.h_ld, self.error_flag)
        if s.down:
            self._join()
        return dict(y=r.y if s.down else None, y_ld=W, **pairs)

    def _side(self, s, r, view, longest):
        n, W = view.n_tok, self.cfg.width
        self._linear(s.proj, r.h, r.a, n, s.ld, r, epilogue=ops.EPI_GELU_MUL, mul=(self.side_table, self.side_table.shape[1], s.layer * self.side_ld), mul_ids=r.tok, pdl=1)
        self._linear(s.out, r.a, r.y, n, W, r, pdl=1)
        return dict(y=r.y, y_ld=W)

    def _layers(self, r, view, longest, ids, ids_ld=1, step=None, pos_out=None, layer_sums=None):
        """Leaves the stream before the last sublayer's output is added in r.x, and what is to be added in r.pending; `_head` finishes."""
        c, n = self.cfg, view.n_tok
        ops.post_norm(n, c.width, c.eps, self.dtype, x_out=r.x, h=r.h, h_ld=self.h_ld, table=self.table, vocab=c.vocab, ids=ids, ids_ld=ids_ld, step=step,
                      pos_out=pos_out, id_out=r.tok)
        run = {"mixer": self._mixer, "moe": self._experts, "side": self._side}
        r.pending = None
        for s in self.subs:
            if r.pending is not None:
                ops.post_norm(n, c.width, c.eps, self.dtype, x_in=r.x, x_out=r.x, h=r.h, h_ld=self.h_ld, **r.pending)
                if layer_sums is not None and s.kind == "mixer":
                    layer_sums.append(r.x[:n].clone())
            r.pending = run[s.kind](s, r, view, longest)
            r.pending["norm_w"] = s.norm

    def _head(self, r, n, out, row_index=None, layer_sums=None, n_tok=0):
        c = self.cfg
        if layer_sums is not None:
            layer_sums.append(torch.empty((n_tok, c.width), dtype=torch.float32, device=self.device))
            ops.post_norm(n_tok, c.width, c.eps, self.dtype, x_in=r.x, x_out=layer_sums[-1], **r.pending)
        if n:
            ops.post_norm(n, c.width, c.eps, self.dtype, x_in=r.x, h=r.h, h_ld=self.h_ld, final_w=self.final_norm, row_index=row_index, **r.pending)
            self._linear(self.head, r.h, out, n, c.vocab, r, pdl=1)
