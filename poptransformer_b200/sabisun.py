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
float32: everything is true 32-bit."""
from types import SimpleNamespace

import torch

from . import ops
from .sequences import SequenceDecoder


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


class SabisunDecoder(SequenceDecoder):
    # ---- weights --------------------------------------------------------------------------------
    def _load(self, w):
        c, dt, f32, lin = self.cfg, self.dtype, w.f32, w.lin

        def hyper(p, q):
            s = c.streams
            if p + f"hc{q}.in" not in w and s == 1:
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
                sub.sink = f32(p + "mix.sink", (m.heads,)) if p + "mix.sink" in w else None
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
    def _alloc_layers(self):
        c, dev, B, dt = self.cfg, self.device, self.batch, self.dtype
        page_size = self._state_opts["page_size"]
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
        self.attn_ws = self._attn_workspace([(s.m.heads, s.m.vdim, s.m.window, s.m.keep_first) for s in self.subs if s.kind == "attention"])

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
        self._linear_workspaces(r, rows, [self.head] + [x for s in self.subs for x in (s.proj, s.out)])
        r.ssm_ws = None
        if mm and dt == torch.bfloat16:
            n = max(ops._lib.lib().pt_ssm_workspace_bytes(rows, min(self.batch, rows), m.heads, m.vdim, m.state) for m in mm)
            r.ssm_ws = torch.empty(n, dtype=torch.uint8, device=dev)
        return r

    # ---- the layers -----------------------------------------------------------------------------
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
