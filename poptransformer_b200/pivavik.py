"""Pivavik: a small decoder whose layers run their mixer and their feed-forward side by side, and of which a stretch runs several times.

One fp32 residual stream; a layer reads one RMS norm of it (weights stored as their distance from one) and adds mixer and feed-forward at
once (csrc/post_norm.cu).  Mixers and feed-forwards, in any order:
  latent_attention  queries through a latent; keys and values from a cached latent plus one rotated key part shared by all heads; a gate
                    per head (latent.py, csrc/latent.cu).  Decode steps stay in the latent's space, prompts project the context up
  attention         grouped heads with biases, a sliding window, a softcap on the scores, a gate per element; no rotation
                    (csrc/window_attn.cu)
  dense             gelu gated unit with biases
  moe               sigmoid router scores of the `top` experts weigh the experts' inputs (experts.py, csrc/moe.cu)
The looped layers run `times` passes over the same weights, each pass with caches of its own; before a pass the stream is mixed with the
embedding output by one product, whose bias is the pass's step vector.  The output layer is the embedding table, with a softcap.

The products that share a layer's norm are one linear (both latents and the gate, or q, k, v and the gate, and the router, whose logits
leave it in fp32), and a dense feed-forward's down projection is one linear with the mixer's output projection, over both inputs side
by side.  The feed-forward runs beside the mixer.

Every size and constant comes from the configuration; layers may differ in all of them.  dtype bfloat16: matrix products and their
inputs are bfloat16, accumulation, residual stream, norms, rotation, scores, softmax and router are float32.  float32: everything is
true 32-bit."""
from types import SimpleNamespace

import torch

from . import ops
from .experts import Experts
from .latent import LatentAttention, latent_mixer
from .sequences import JointRows, SequenceDecoder


class PivavikConfig:
    """The parsed config.json plus the longest sequence the decoder is built for."""

    def __init__(self, config, max_len):
        self.max_len = int(max_len)
        self.vocab, self.width, self.eps = int(config["vocab"]), int(config["width"]), float(config["norm"]["eps"])
        self.logit_softcap = float(config.get("logit_softcap") or 0.0)
        self.layers = []
        for i, lay in enumerate(config["layers"]):
            kind, m, mlp = lay["type"], lay["mixer"], lay.get("mlp")
            if kind == "latent_attention":
                layer = latent_mixer(i, kind, m)
            elif kind == "attention":
                layer = SimpleNamespace(kind=kind, heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), scale=float(m["scale"]))
                layer.kv_heads, layer.window, layer.softcap = int(m["kv_heads"]), int((m.get("mask") or {}).get("size") or 0), float(m.get("softcap") or 0.0)
                if layer.heads % layer.kv_heads:
                    raise ops.PtError(f"layer {i}: {layer.heads} heads do not divide over {layer.kv_heads} key/value heads")
            else:
                raise ops.PtError(f"layer {i}: unknown mixer {kind!r}")
            layer.ff, layer.moe = 0, None
            if mlp is not None:
                if mlp["kind"] == "dense":
                    layer.ff = int(mlp["ff"])
                elif mlp["kind"] == "moe":
                    layer.moe = SimpleNamespace(experts=int(mlp["router"]["experts"]), top=int(mlp["router"]["top"]), ff=int(mlp["expert"]["ff"]))
                    if not 1 <= layer.moe.top <= layer.moe.experts:
                        raise ops.PtError(f"layer {i}: {layer.moe.top} of {layer.moe.experts} experts")
                else:
                    raise ops.PtError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
            self.layers.append(layer)
        loop, n = config.get("loop"), len(self.layers)
        self.loop = (int(loop["start"]), int(loop["stop"]), int(loop["times"])) if loop else None
        if self.loop and not (0 <= self.loop[0] < self.loop[1] <= n and self.loop[2] >= 1):
            raise ops.PtError(f"a loop over layers {self.loop[0]} .. {self.loop[1]} of {n}, {self.loop[2]} times")

    def runs(self):
        """(layer, the pass that starts with it or None) in the order the layers run."""
        start, stop, times = self.loop or (0, 0, 0)
        out = [(i, None) for i in range(start)]
        for t in range(times):
            out += [(i, t if i == start else None) for i in range(start, stop)]
        return out + [(i, None) for i in range(stop, len(self.layers))]


class PivavikDecoder(SequenceDecoder):
    # ---- weights --------------------------------------------------------------------------------
    def _load(self, w):
        c, dt, dev, f32, mat = self.cfg, self.dtype, self.device, w.f32, w.mat
        W = c.width
        bf16 = dt == torch.bfloat16
        zeros = lambda rows, cols: torch.zeros((rows, cols), dtype=dt, device=dev)
        self.head = w.lin(["embed"], [(c.vocab, W)], keep=True, limit=c.logit_softcap)     # also the look-up table
        self.table, self.h_ld = self.head.w, self.head.ld
        self.embed_norm, self.final_norm = 1.0 + f32("embed.norm", (W,)), 1.0 + f32("final.norm", (W,))
        if c.loop:
            self.loop_in, self.loop_step = w.lin(["loop.in"], [(W, 2 * W)]), f32("loop.step", (c.loop[2], W))
        ropes, self.subs = {}, []
        for i, lay in enumerate(c.layers):
            p, M = f"l{i}.", f"l{i}.mix."
            sub = SimpleNamespace(layer=i, lay=lay, norm=1.0 + f32(p + "norm1", (W,)), ff=None, experts=None)
            rows = JointRows(W, dt, dev)
            H, D, V = lay.heads, lay.dim, lay.vdim
            if lay.kind == "attention":
                for name, n in (("q", H * D), ("k", lay.kv_heads * D), ("v", lay.kv_heads * V)):
                    rows.add(mat(M + name, (n, W)), f32(M + name + ".b", (n,)))
                sub.gate_col = rows.column()
                rows.add(mat(M + "g", (H * V, W)))
            else:
                sub.lat = LatentAttention(w, M, lay, W, rows, ropes, c.max_len)
            split = None
            if lay.moe:
                E, F = lay.moe.experts, lay.moe.ff
                split = rows.column(32)
                rows.add(mat(p + "mlp.router", (E, W)))
                gates, ups = ([mat(p + f"mlp.e{e}.{n}", (F, W)) for e in range(E)] for n in ("gate", "up"))
                sub.experts = Experts(dt, lay.moe.top, gates, ups, [mat(p + f"mlp.e{e}.down", (W, F)) for e in range(E)], glu=ops.GLU_SILU, score=ops.MOE_SIGMOID,
                                      weigh_input=True)
            sub.proj = rows.linear(biased=lay.kind == "attention", split=split)
            sub.ld = ops.pad_to(sub.proj.n_out if split is None else split, 8)
            # ---- outputs: the mixer's columns, then the dense feed-forward's
            sub.ff_col = ops.pad_to(H * V, 8)
            outs, out_bias = [mat(M + "o", (W, H * V))], None
            if lay.ff:
                ld = ops.pad_to(sub.ff_col + lay.ff, ops.DenseLinear.K_PAD if bf16 else 8)
                features = ld - sub.ff_col
                gate, up = (mat(p + f"mlp.{n}", (lay.ff, W)) for n in ("gate", "up"))
                gate_b, up_b = (f32(p + f"mlp.{n}.b", (lay.ff,))[:, None] for n in ("gate", "up"))
                sub.ff = ops.DenseLinear(ops.glu_rows(gate, up, features), dt, bias=ops.glu_rows(gate_b, up_b, features)[:, 0].contiguous(), glu=ops.GLU_GELU)
                outs += [zeros(W, sub.ff_col - H * V), mat(p + "mlp.down", (W, lay.ff)), zeros(W, features - lay.ff)]
                out_bias = f32(p + "mlp.down.b", (W,))
            sub.out = ops.DenseLinear(torch.cat(outs, 1), dt, bias=out_bias)
            sub.mix_cols = sub.ff_col if lay.ff else sub.out.ld
            self.subs.append(sub)
        self.runs = [SimpleNamespace(sub=self.subs[i], index=k, entry=t) for k, (i, t) in enumerate(c.runs())]

    def _linears(self):
        """Every linear once per time a token runs through it."""
        once = [self.head] + [self.loop_in for r in self.runs if r.entry is not None]
        return once + [x for r in self.runs for x in (r.sub.proj, r.sub.ff, r.sub.lat.uq if r.sub.lay.kind != "attention" else None, r.sub.out) if x is not None]

    def expert_groups(self):
        return [r.sub.experts for r in self.runs if r.sub.experts]

    def fixed_bytes(self):
        """Weight bytes that every decode step streams, whatever the experts: the linears and the latents' per-head up-projections."""
        return sum(x.nbytes for x in self._linears()) + sum(r.sub.lat.head_bytes for r in self.runs if r.sub.lay.kind != "attention")

    def weight_bytes(self, rows=1):
        """Algorithmic weight bytes one decode step of `rows` tokens streams, of the experts as many as the rows can choose at most."""
        return self.fixed_bytes() + sum(e.step_bytes(rows) for e in self.expert_groups())

    # ---- state ----------------------------------------------------------------------------------
    def _alloc_layers(self):
        c, B = self.cfg, self.batch
        self.caches = {}                                              # a run's own (the passes of a loop share weights, not positions)
        for r in self.runs:
            lay = r.sub.lay
            kw = dict(page_size=self._state_opts["page_size"], device=self.device, page_table=self.slots.page_table, dtype=self.dtype, n_pages=self.slots.n_pages)
            if lay.kind == "latent_attention":
                self.caches[r.index] = r.sub.lat.new_cache(self)
            else:
                self.caches[r.index] = ops.PagedKVCache(B, lay.kv_heads, lay.dim, c.max_len, v_dim=lay.vdim, **kw)
        self.attn_ws = self._attn_workspace([(s.lay.heads, s.lay.vdim, s.lay.window, 0) for s in self.subs if s.lay.kind == "attention"])

    def _row_buffers(self, rows):
        c, dev, dt = self.cfg, self.device, self.dtype
        f32, act = dict(dtype=torch.float32, device=dev), dict(dtype=dt, device=dev)
        moes = [s for s in self.subs if s.experts]
        r = SimpleNamespace(rows=rows)
        r.x = torch.empty((rows, c.width), **f32)                                              # residual stream
        r.h = torch.empty(rows * self.h_ld, **act)
        r.a = torch.empty(rows * max(s.ld for s in self.subs), **act)                          # projection outputs
        r.b = torch.empty(rows * max(s.out.ld for s in self.subs), **act)                      # mixer outputs, a dense feed-forward's features
        r.y = torch.empty((rows, c.width), **f32)                                              # sublayer outputs
        r.loop = torch.empty(rows * self.loop_in.ld, **act) if c.loop else None                # [stream | embedding output]
        self._linear_workspaces(r, rows, self._linears())
        r.beside = SimpleNamespace(lin_ws=None, gemm_ws=None)                                  # of the feed-forward, which runs beside the mixer
        if moes or any(s.ff for s in self.subs):
            self._linear_workspaces(r.beside, rows, [s.ff for s in self.subs if s.ff] + [x for s in moes for x in (s.experts.up, s.experts.back)])
        if moes:
            Experts.buffers(r, rows, [s.experts for s in moes], self.h_ld, dev, r.beside)
        LatentAttention.buffers(r, rows, self._latents(), self)
        return r

    def _latents(self):
        return [s.lat for s in self.subs if s.lay.kind == "latent_attention"]

    # ---- the layers -----------------------------------------------------------------------------
    def _latent_attention(self, run, r, view, longest):
        s = run.sub
        s.lat(self, r, view, longest, r.a, s.ld, self.caches[run.index], r.b, s.out.ld, s.mix_cols, self._latents())

    def _attention(self, run, r, view, longest):
        s, lay = run.sub, run.sub.lay
        ops.window_attn(view, r.a, s.ld, self.caches[run.index], r.b, s.out.ld, lay.heads, lay.scale, lay.window, max_tokens_per_seq=longest, workspace=self.attn_ws,
                        error_flag=self.error_flag, plain=self.plain, out_cols=s.mix_cols, softcap=lay.softcap, gate=r.a[s.gate_col:], gate_ld=s.ld)

    def _layer(self, run, r, view, longest):
        """Mixer and feed-forward of the norm in r.h; returns what is to be added to the stream."""
        s, n, W = run.sub, view.n_tok, self.cfg.width
        E = s.lay.moe.experts if s.experts else 0
        self._linear(s.proj, r.h, r.a, n, s.ld, r, out2=r.logits if E else None, out2_ld=E, pdl=1)
        pending = dict(y=r.y, y_ld=W)
        if s.ff or s.experts:
            with self._beside():
                if s.ff:
                    self._linear(s.ff, r.h, r.b[s.ff_col:], n, s.out.ld, r.beside, epilogue=ops.EPI_GLU)
                else:
                    pending.update(s.experts(r, n, self.h_ld, self.error_flag, r.beside))
        (self._attention if s.lay.kind == "attention" else self._latent_attention)(run, r, view, longest)
        if s.ff:
            self._join()
        self._linear(s.out, r.b, r.y, n, W, r, pdl=0 if s.ff else 1)
        if s.experts:
            self._join()
        return pending

    def _layers(self, r, view, longest, ids, ids_ld=1, step=None, pos_out=None, layer_sums=None):
        """Leaves the stream before the last layer's outputs are added in r.x, and what is to be added in r.pending; `_head` finishes."""
        c, n, W = self.cfg, view.n_tok, self.cfg.width

        def then(run):
            """Where a residual step puts what `run` reads: the loop's product takes the stream itself."""
            if run.entry is not None:
                return dict(h=r.loop, h_ld=self.loop_in.ld, h_cols=W)
            return dict(h=r.h, h_ld=self.h_ld, final_w=run.sub.norm)

        keep = dict(copy=r.loop[W:], copy_ld=self.loop_in.ld, copy_cols=self.loop_in.ld - W) if c.loop else {}
        ops.post_norm(n, W, c.eps, self.dtype, x_out=r.x, table=self.table, vocab=c.vocab, ids=ids, ids_ld=ids_ld, step=step, pos_out=pos_out, norm_w=self.embed_norm,
                      **keep, **then(self.runs[0]))
        for k, run in enumerate(self.runs):
            if k:
                ops.post_norm(n, W, c.eps, self.dtype, x_in=r.x, x_out=r.x, **r.pending, **then(run))
                if layer_sums is not None:
                    layer_sums.append(r.x[:n].clone())
            if run.entry is not None:
                self._linear(self.loop_in, r.loop, r.x, n, W, r, bias=self.loop_step[run.entry], pdl=1)
                ops.post_norm(n, W, c.eps, self.dtype, x_in=r.x, h=r.h, h_ld=self.h_ld, final_w=run.sub.norm)
            r.pending = self._layer(run, r, view, longest)

    def _head(self, r, n, out, row_index=None, layer_sums=None, n_tok=0):
        c = self.cfg
        if layer_sums is not None:
            layer_sums.append(torch.empty((n_tok, c.width), dtype=torch.float32, device=self.device))
            ops.post_norm(n_tok, c.width, c.eps, self.dtype, x_in=r.x, x_out=layer_sums[-1], **r.pending)
        if n:
            ops.post_norm(n, c.width, c.eps, self.dtype, x_in=r.x, h=r.h, h_ld=self.h_ld, final_w=self.final_norm, row_index=row_index, **r.pending)
            self._linear(self.head, r.h, out, n, c.vocab, r, epilogue=ops.EPI_SOFTCAP if c.logit_softcap else ops.EPI_STORE, pdl=1)
