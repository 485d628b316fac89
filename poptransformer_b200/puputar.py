"""Puputar: a small decoder of latent attention layers beside feed-forwards that read a norm of their own, with a token shift.

One fp32 residual stream.  A layer reads two RMS norms of it, each over groups of neighbouring dimensions: the mixer takes the first,
mixed element by element with the same norm of the token before (a part of every layer's state), the feed-forward the second; both
outputs are added at once (csrc/shift_norm.cu).  Mixers and feed-forwards, in any order:
  latent_attention    queries through a latent; keys and values from a cached latent plus one rotated key part shared by all heads; a gate
                      per head (latent.py, csrc/latent.cu).  Decode steps stay in the latent's space, prompts project the context up
  latent_attention_2  a gate per output.  The layer may read the latents that an earlier one caches, with its own queries and up-projections
  dense               one matrix up, the xIELU unit, one down, with biases
  moe                 softmax scores, chosen with a correction among the best groups of experts; relu^2 units, and identity experts that
                      give the input back (experts.py, csrc/moe.cu)

The products that share the mixer's input are one linear (both latents and the gate), and a dense feed-forward's down projection is one
linear with the mixer's output projection, over both inputs side by side.  The feed-forward runs beside the mixer.  Identity experts cost
no product: the residual step adds their share of the feed-forward's input.

Every size and constant comes from the configuration; layers may differ in all of them.  dtype bfloat16: matrix products and their
inputs are bfloat16, accumulation, residual stream, norms, token shift and its state, rotation, scores, softmax and router are
float32.  float32: everything is true 32-bit."""
from types import SimpleNamespace

import numpy as np
import torch

from . import ops
from .experts import Experts
from .latent import LatentAttention, latent_mixer
from .sequences import JointRows, SequenceDecoder

GATE_PER_VALUE = {"latent_attention": False, "latent_attention_2": True}


class PuputarConfig:
    """The parsed config.json plus the longest sequence the decoder is built for."""

    def __init__(self, config, max_len):
        self.max_len = int(max_len)
        self.vocab, self.width = int(config["vocab"]), int(config["width"])
        self.eps, self.groups = float(config["norm"]["eps"]), int(config["norm"]["groups"])
        if self.groups < 1 or self.width % self.groups:
            raise ops.PtError(f"a width of {self.width} in {self.groups} groups")
        self.layers = []
        for i, lay in enumerate(config["layers"]):
            kind, m, mlp = lay["type"], lay["mixer"], lay.get("mlp")
            if kind not in GATE_PER_VALUE:
                raise ops.PtError(f"layer {i}: unknown mixer {kind!r}")
            layer = latent_mixer(i, kind, m)
            layer.kv_from, layer.ff, layer.moe = m.get("kv_from"), 0, None
            if layer.kv_from is not None:
                if not 0 <= layer.kv_from < i or self.layers[layer.kv_from].kv_from is not None:
                    raise ops.PtError(f"layer {i}: layer {layer.kv_from} caches nothing that it could read")
                source = self.layers[layer.kv_from]
                if (source.rank, source.rot_dim, source.base) != (layer.rank, layer.rot_dim, layer.base):
                    raise ops.PtError(f"layer {i}: layer {layer.kv_from} caches latents of another shape or rotation")
            if mlp is not None:
                if mlp["kind"] == "dense":
                    layer.ff = int(mlp["ff"])
                elif mlp["kind"] == "moe":
                    layer.moe = self._router(i, mlp)
                else:
                    raise ops.PtError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
            self.layers.append(layer)

    @staticmethod
    def _router(i, mlp):
        r = mlp["router"]
        groups = r.get("groups") or {"count": 1, "keep": 1}
        moe = SimpleNamespace(experts=int(r["experts"]), top=int(r["top"]), ff=int(mlp["expert"]["ff"]), identity=int(r.get("identity") or 0), groups=int(groups["count"]),
                              keep=int(groups["keep"]))
        n = moe.experts + moe.identity
        if moe.experts < 1 or moe.groups < 1 or n % moe.groups or not 1 <= moe.keep <= moe.groups:
            raise ops.PtError(f"layer {i}: {moe.keep} of {moe.groups} groups of {n} experts")
        if not 1 <= moe.top <= n // moe.groups * moe.keep:
            raise ops.PtError(f"layer {i}: {moe.top} of the {n // moe.groups * moe.keep} experts in {moe.keep} groups")
        return moe


class PuputarDecoder(SequenceDecoder):
    # ---- weights --------------------------------------------------------------------------------
    def _load(self, w):
        c, dt, dev, f32, mat = self.cfg, self.dtype, self.device, w.f32, w.mat
        W = c.width
        zeros = lambda rows, cols: torch.zeros((rows, cols), dtype=dt, device=dev)
        self.table = mat("embed", (c.vocab, W)).contiguous()
        self.head = w.lin(["head"], [(c.vocab, W)])
        self.h_ld = self.head.ld
        self.embed_norm, self.final_norm = f32("embed.norm", (W,)), f32("final.norm", (W,))
        ropes, self.subs = {}, []
        for i, lay in enumerate(c.layers):
            p, M = f"l{i}.", f"l{i}.mix."
            sub = SimpleNamespace(layer=i, lay=lay, norm1=f32(p + "norm1", (W,)), shift=f32(p + "shift", (W,)), norm2=None, ff=None, router=None, experts=None)
            rows = JointRows(W, dt, dev)
            sub.lat = LatentAttention(w, M, lay, W, rows, ropes, c.max_len, gate_per_value=GATE_PER_VALUE[lay.kind], interleaved=True, own=lay.kv_from is None)
            sub.cache = i if lay.kv_from is None else lay.kv_from
            rows.column(32)                      # (the GEMM's fast epilogue takes whole groups of 32 outputs)
            sub.proj = rows.linear()
            sub.ld = ops.pad_to(sub.proj.n_out, 8)
            if lay.ff or lay.moe:
                sub.norm2 = f32(p + "norm2", (W,))
            if lay.moe:
                moe, Q = lay.moe, p + "mlp."
                n = moe.experts + moe.identity
                sub.router = ops.DenseLinear(mat(Q + "router", (n, W)), dt)
                ups, downs = ([mat(Q + f"e{e}.{name}", shape) for e in range(moe.experts)] for name, shape in (("up", (moe.ff, W)), ("down", (W, moe.ff))))
                sub.experts = Experts(dt, moe.top, None, ups, downs, score=ops.MOE_SOFTMAX_ALL, correction=f32(Q + "correction", (n,)), groups=moe.groups, keep=moe.keep,
                                      identity=moe.identity)
            # ---- outputs: the mixer's columns, then the dense feed-forward's
            mixed = lay.heads * lay.vdim
            sub.ff_col = ops.pad_to(mixed, 8)
            outs, out_bias = [mat(M + "o", (W, mixed))], None
            if lay.ff:
                features = ops.pad_to(sub.ff_col + lay.ff, ops.DenseLinear.K_PAD if dt == torch.bfloat16 else 8) - sub.ff_col
                p_, q_ = f32(p + "mlp.act", (2,)).double().cpu().numpy()
                sub.ff = ops.DenseLinear(mat(p + "mlp.up", (lay.ff, W)), dt, pad_rows=features, bias=f32(p + "mlp.up.b", (lay.ff,)),
                                         xielu=(float(np.logaddexp(0.0, p_)), float(0.5 + np.logaddexp(0.0, q_))))
                outs += [zeros(W, sub.ff_col - mixed), mat(p + "mlp.down", (W, lay.ff)), zeros(W, features - lay.ff)]
                out_bias = f32(p + "mlp.down.b", (W,))
            sub.out = ops.DenseLinear(torch.cat(outs, 1), dt, bias=out_bias)
            sub.mix_cols = sub.ff_col if lay.ff else sub.out.ld
            self.subs.append(sub)
        self.lats = [s.lat for s in self.subs]

    def _linears(self):
        return [self.head] + [x for s in self.subs for x in (s.proj, s.ff, s.router, s.lat.uq, s.out) if x is not None]

    def expert_groups(self):
        return [s.experts for s in self.subs if s.experts]

    def fixed_bytes(self):
        """Weight bytes that every decode step streams, whatever the experts: the linears and the latents' per-head up-projections."""
        return sum(x.nbytes for x in self._linears()) + sum(s.lat.head_bytes for s in self.subs)

    def weight_bytes(self, rows=1):
        """Algorithmic weight bytes one decode step of `rows` tokens streams, of the experts as many as the rows can choose at most."""
        return self.fixed_bytes() + sum(e.step_bytes(rows) for e in self.expert_groups())

    # ---- state ----------------------------------------------------------------------------------
    def _alloc_layers(self):
        own = {s.layer: s.lat.new_cache(self) for s in self.subs if s.cache == s.layer}
        self.caches = {s.layer: own[s.cache] for s in self.subs}
        # the last token's norm of every layer and slot, and where a pass with several tokens per sequence leaves the next ones
        self.shift_state, self.shift_next = (torch.zeros((len(self.subs), self.batch, self.cfg.width), dtype=torch.float32, device=self.device) for _ in range(2))

    def _row_buffers(self, rows):
        c, dev, dt = self.cfg, self.device, self.dtype
        f32, act = dict(dtype=torch.float32, device=dev), dict(dtype=dt, device=dev)
        moes = [s for s in self.subs if s.experts]
        r = SimpleNamespace(rows=rows)
        r.xs = [torch.empty((rows, c.width), **f32) for _ in range(2)]                         # residual stream, before and after a step
        r.h = torch.empty(rows * self.h_ld, **act)                                             # the mixer's input
        r.hs = [torch.empty(rows * self.h_ld, **act) for _ in range(2)]                        # the feed-forward's, of this layer and the one before
        r.a = torch.empty(rows * max(s.ld for s in self.subs), **act)                          # projection outputs
        r.b = torch.empty(rows * max(s.out.ld for s in self.subs), **act)                      # mixer outputs, a dense feed-forward's features
        r.y = torch.empty((rows, c.width), **f32)                                              # sublayer outputs
        self._linear_workspaces(r, rows, self._linears())
        r.beside = SimpleNamespace(lin_ws=None, gemm_ws=None)                                  # of the feed-forward, which runs beside the mixer
        if moes or any(s.ff for s in self.subs):
            self._linear_workspaces(r.beside, rows, [x for s in self.subs for x in (s.ff, s.router) if x] + [x for s in moes for x in (s.experts.up, s.experts.back)])
        if moes:
            Experts.buffers(r, rows, [s.experts for s in moes], self.h_ld, dev, r.beside)
        LatentAttention.buffers(r, rows, self.lats, self)
        return r

    # ---- the layers -----------------------------------------------------------------------------
    def _residual(self, r, view, k, **kw):
        """The step in front of layer k: its two inputs (the second where it has a feed-forward) and the stream in r.xs[k % 2]."""
        s, n, W, c = self.subs[k], view.n_tok, self.cfg.width, self.cfg
        single = n == view.n_seq
        state = self.shift_state[k]
        second = dict(w2=s.norm2, h2=r.hs[k % 2], h2_ld=self.h_ld) if s.norm2 is not None else {}
        ops.shift_norm(view, n, W, c.groups, c.eps, self.dtype, x_out=r.xs[k % 2], w1=s.norm1, shift=s.shift, h1=r.h, h1_ld=self.h_ld, state_in=state,
                       state_out=state if single else self.shift_next[k], state_by_seq=not single, **second, **kw)

    def _layer(self, k, r, view, longest):
        """Mixer and feed-forward of layer k; returns what is to be added to the stream."""
        s, n, W, h2 = self.subs[k], view.n_tok, self.cfg.width, r.hs[k % 2]
        pending = dict(y=r.y, y_ld=W)
        if s.ff or s.experts:
            with self._beside():
                if s.ff:
                    self._linear(s.ff, h2, r.b[s.ff_col:], n, s.out.ld, r.beside, epilogue=ops.EPI_XIELU)
                else:
                    self._linear(s.router, h2, r.logits, n, s.experts.logits, r.beside)
                    pending.update(s.experts(r, n, self.h_ld, self.error_flag, r.beside, h=h2), self_rows=h2, self_ld=self.h_ld)
        self._linear(s.proj, r.h, r.a, n, s.ld, r, pdl=1)
        s.lat(self, r, view, longest, r.a, s.ld, self.caches[k], r.b, s.out.ld, s.mix_cols, self.lats)
        if s.ff:
            self._join()
        self._linear(s.out, r.b, r.y, n, W, r, pdl=0 if s.ff else 1)
        if s.experts:
            self._join()
        return pending

    def _layers(self, r, view, longest, ids, ids_ld=1, step=None, pos_out=None, layer_sums=None):
        """Leaves the stream before the last layer's outputs are added in r.xs, and what is to be added in r.pending; `_head` finishes."""
        n = view.n_tok
        self._residual(r, view, 0, table=self.table, vocab=self.cfg.vocab, ids=ids, ids_ld=ids_ld, step=step, pos_out=pos_out, embed_w=self.embed_norm)
        for k in range(len(self.subs)):
            if k:
                self._residual(r, view, k, x_in=r.xs[(k - 1) % 2], **r.pending)
                if layer_sums is not None:
                    layer_sums.append(r.xs[k % 2][:n].clone())
            r.pending = self._layer(k, r, view, longest)
        if n != view.n_seq:
            _, _, slot, _ = view.keep
            self.shift_state.index_copy_(1, slot.long(), self.shift_next[:, :view.n_seq])

    def _head(self, r, n, out, row_index=None, layer_sums=None, n_tok=0):
        c, last = self.cfg, dict(x_in=r.xs[(len(self.subs) - 1) % 2], **r.pending)
        if layer_sums is not None:
            layer_sums.append(torch.empty((n_tok, c.width), dtype=torch.float32, device=self.device))
            ops.shift_norm(None, n_tok, c.width, c.groups, c.eps, self.dtype, x_out=layer_sums[-1], **last)
        if n:
            ops.shift_norm(None, n, c.width, c.groups, c.eps, self.dtype, w2=self.final_norm, h2=r.h, h2_ld=self.h_ld, row_index=row_index, **last)
            self._linear(self.head, r.h, out, n, c.vocab, r, pdl=1)
