"""Latent attention as a decoder's layer uses it: weight preparation, buffers, and the launches between the layer's input projection and
its output projection (csrc/latent.cu; csrc/window_attn.cu over rows of the context for prompts on tensor cores)."""
from types import SimpleNamespace

import numpy as np
import torch

from . import ops
from .padetar import rope_frequencies


def latent_mixer(i, kind, m):
    """The sizes and constants of a latent mixer's configuration."""
    rot = m["rot"]
    lay = SimpleNamespace(kind=kind, heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), scale=float(m["scale"]), q_rank=int(m["q_rank"]), rank=int(m["kv_rank"]),
                          rot_dim=int(m["rot_dim"]), base=float(rot["base"]))
    if int(rot["dims"]) != lay.rot_dim or lay.rot_dim % 2:
        raise ops.PtError(f"layer {i}: {rot['dims']} rotated dimensions of a rotated part of {lay.rot_dim}")
    return lay


class LatentAttention:
    """One layer's latent attention.

    w: the decoder's weights, M: the tensors' prefix, lay: a latent_mixer; rows: the layer's input projection (sequences.JointRows), which
    takes the down-projections and the gate.  gate_per_value: a gate per output instead of one per head.  interleaved: dimensions 2 i and
    2 i + 1 of the rotated part are a pair (the kernels pair i with i + rot_dim / 2: the rows of the weights are put in that order, which
    no score notices).  own: the layer caches latents of its own; otherwise `cache` is called with another layer's.  ropes: rotation
    tables of the decoder, shared by layers that rotate alike."""

    def __init__(self, w, M, lay, width, rows, ropes, max_len, gate_per_value=False, interleaved=False, own=True):
        dt, dev, H, D, V, R, rank = w.dtype, w.device, lay.heads, lay.dim, lay.vdim, lay.rot_dim, lay.rank
        bf16 = dt == torch.bfloat16
        self.lay, self.gate_per_value = lay, gate_per_value
        order = torch.cat([torch.arange(0, R, 2), torch.arange(1, R, 2)]) if interleaved else torch.arange(R)
        order = order.to(dev)
        self.q_col = rows.column()
        rows.add(w.mat(M + "dq", (lay.q_rank, width)))
        self.kv_col = None
        if own:
            self.kv_col = rows.column()
            down = w.mat(M + "dkv", (rank + R, width))
            rows.add(torch.cat([down[:rank], down[rank:][order]]))
        self.gate_col = rows.column()
        rows.add(w.mat(M + "g", (H * V if gate_per_value else H, width)))
        uq = w.mat(M + "uq", (H * (D + R), lay.q_rank)).view(H, D + R, lay.q_rank)
        self.uq = ops.DenseLinear(torch.cat([uq[:, D:][:, order], uq[:, :D]], 1).reshape(-1, lay.q_rank), dt)       # a head: the rotated part first
        self.q_ld = ops.pad_to(self.uq.n_out, 8)
        uk, uv = w.mat(M + "uk", (H * D, rank)), w.mat(M + "uv", (H * V, rank))
        self.w = SimpleNamespace(heads=H, dim=D, rot_dim=R, vdim=V, rank=rank, q_rank=lay.q_rank, q_norm=w.f32(M + "dq.norm", (lay.q_rank,)),
                                 kv_norm=w.f32(M + "dkv.norm", (rank,)) if own else None, w_k=uk.view(H, D, rank).transpose(1, 2).contiguous(), w_v=uv.view(H, V, rank).contiguous())
        # prompts on tensor cores: keys and values of the whole context by one product
        self.up = ops.DenseLinear(torch.cat([uk, uv], 0), dt) if bf16 and R and not any(x % 8 for x in (D, R, V, rank)) and D + R <= 256 and V <= 128 else None
        if (R, lay.base) not in ropes:
            ang = np.arange(max_len)[:, None] * rope_frequencies(R, lay.base)
            ropes[R, lay.base] = torch.from_numpy(np.stack([np.cos(ang), np.sin(ang)], -1).astype(np.float32)).to(dev) if R else None
        self.rope = ropes[R, lay.base]

    @property
    def head_bytes(self):
        """Weight bytes of the per-head up-projections as decode steps read them."""
        return sum(x.numel() * x.element_size() for x in (self.w.w_k, self.w.w_v))

    def new_cache(self, dec):
        return ops.latent_cache(dec.batch, self.w, dec.cfg.max_len, page_size=dec._state_opts["page_size"], device=dec.device, page_table=dec.slots.page_table, dtype=dec.dtype,
                                n_pages=dec.slots.n_pages)

    @staticmethod
    def buffers(r, rows, layers, dec):
        """Adds to `r` what `layers` (of one decoder) need for up to `rows` tokens."""
        r.lat_ws = r.ctx = None
        if layers:
            size = lambda n: torch.empty(rows * n, dtype=dec.dtype, device=dec.device)
            r.q, r.cq = size(max(s.q_ld for s in layers)), size(max(s.uq.ld for s in layers))
            if rows <= dec.batch or dec.plain or any(s.up is None for s in layers):
                r.lat_ws = torch.empty(max(ops.latent_workspace_bytes(rows, s.w, dec.dtype) for s in layers), dtype=torch.uint8, device=dec.device)

    @staticmethod
    def _context(r, rows, layers, dec):
        """Buffers for `rows` rows of context that prompts project up."""
        if r.ctx is None or r.ctx.rows < rows:
            r.ctx = None
            ups = [s for s in layers if s.up]
            size = lambda n: torch.empty(rows * n, dtype=dec.dtype, device=dec.device)
            r.ctx = SimpleNamespace(rows=rows, shared=size(max(s.w.rot_dim for s in ups)), latent=size(max(s.up.ld for s in ups)), kv=size(max(s.up.n_out for s in ups)))
            dec._linear_workspaces(r.ctx, rows, [s.up for s in ups])
        return r.ctx

    def __call__(self, dec, r, view, longest, rows, ld, cache, out, out_ld, out_cols, layers):
        """From the input projection's rows (row stride ld) to the heads' outputs in `out`, columns up to out_cols; `layers`: all of the
        decoder's (for the size of shared buffers)."""
        n, w, lay = view.n_tok, self.w, self.lay
        ops.latent_prep(view, rows, ld, self.q_col, self.kv_col, w, r.cq, self.uq.ld, cache, dec.cfg.eps, self.rope, dec.error_flag)
        dec._linear(self.uq, r.cq, r.q, n, self.q_ld, r, pdl=1)
        gate = dict(gate=rows[self.gate_col:], gate_ld=ld)
        if n == view.n_seq or self.up is None or dec.plain:
            ops.latent_attn(view, r.q, self.q_ld, w, cache, out, out_ld, lay.scale, self.rope, r.lat_ws, out_cols=out_cols, error_flag=dec.error_flag, plain=dec.plain,
                            gate_per_value=self.gate_per_value, **gate)
            return
        ctx = self._context(r, view.n_ctx, layers, dec)
        ops.latent_context(view, view.ctx_cu, view.n_ctx, w, cache, ctx.shared, ctx.latent, self.up.ld)
        dec._linear(self.up, ctx.latent, ctx.kv, view.n_ctx, self.up.n_out, ctx)
        keys = SimpleNamespace(k=ctx.kv, v=ctx.kv[w.heads * w.dim:], shared=ctx.shared, ld=self.up.n_out, shared_dim=w.rot_dim, cu=view.ctx_cu, dim=w.dim + w.rot_dim, vdim=w.vdim)
        ops.window_attn(view, r.q, self.q_ld, cache, out, out_ld, w.heads, lay.scale, append=False, max_tokens_per_seq=longest, error_flag=dec.error_flag, rope=self.rope,
                        rope_dims=w.rot_dim, out_cols=out_cols, gate_per_head=not self.gate_per_value, context=keys, **gate)
