"""One latent attention call site for the kernels' tests."""
from types import SimpleNamespace

import numpy as np
import torch

from oracle import pivavik_np as ref
from seq_util import as_type, bf16, i32, rel, view_of

F32, BF16 = torch.float32, torch.bfloat16


class LatentSite:
    """One latent attention call site between its projections, over a cache whose pages lie in shuffled order."""

    def __init__(self, dev, dt, n_slots, H, D, R, V, rank, q_rank, max_len, base=100.0, scale=None, seed=0, page=64, per_value=False, of=None):
        """per_value: a gate per output instead of one per head.  of: another site whose cached latents this one reads."""
        from poptransformer_b200 import ops
        from poptransformer_b200.padetar import rope_frequencies
        self.ops, self.dev, self.dt, self.base, self.eps, self.per_value, self.of = ops, dev, dt, base, 1e-3, per_value, of
        self.gates = H * V if per_value else H
        r = np.random.default_rng(seed)
        self.H, self.D, self.R, self.V, self.rank, self.q_rank, self.scale = H, D, R, V, rank, q_rank, 2.0 * (D + R) ** -0.5 if scale is None else scale
        self.uk, self.uv = bf16(r.standard_normal((H, D, rank)) * rank ** -0.5), bf16(r.standard_normal((H, V, rank)) * rank ** -0.5)
        self.qn, self.kn = 1 + 0.3 * r.standard_normal(q_rank), 1 + 0.3 * r.standard_normal(rank) if of is None else of.kn
        self.w = SimpleNamespace(heads=H, dim=D, rot_dim=R, vdim=V, rank=rank, q_rank=q_rank, q_norm=as_type(self.qn, F32, dev), kv_norm=as_type(self.kn, F32, dev),
                                 w_k=as_type(self.uk.transpose(0, 2, 1), dt, dev), w_v=as_type(self.uv, dt, dev))
        self.up = ops.DenseLinear(as_type(np.concatenate([self.uk.reshape(-1, rank), self.uv.reshape(-1, rank)]), dt, dev), dt)
        a = np.arange(max_len)[:, None] * rope_frequencies(R, base)
        self.rope = as_type(np.stack([np.cos(a), np.sin(a)], -1), F32, dev)
        self.flag = torch.zeros(1, dtype=torch.int32, device=dev)
        if of is not None:
            self.cache = of.cache
            return
        pages = -(-max_len // page)
        table = np.random.default_rng(seed).permutation(n_slots * pages).reshape(n_slots, pages)
        self.cache = ops.latent_cache(n_slots, self.w, max_len, page, dev, i32(table, dev), dtype=dt)
        self.cache.pool.fill_(float("nan"))                   # nothing may be read that was not written

    def inputs(self, n, seed):
        """Rows of the projection [query latent | latent | key part | gates], and queries (as if they came from the query latent)."""
        r = np.random.default_rng(seed)
        return bf16(r.standard_normal((n, self.q_rank + self.rank + self.R + self.gates))), bf16(r.standard_normal((n, self.H, self.D + self.R)))

    def __call__(self, x, q, lens, starts, slots, plain, check_cq=True):
        ops, dev, T, w = self.ops, self.dev, len(x), self.w
        cols = [0, ops.pad_to(self.q_rank, 8)]
        cols.append(cols[1] + ops.pad_to(self.rank + self.R, 8))
        ld = cols[2] + ops.pad_to(self.gates, 8)
        buf = torch.zeros((T, ld), dtype=self.dt, device=dev)
        for c, part in zip(cols, np.split(x, np.cumsum([self.q_rank, self.rank + self.R]), axis=1)):
            buf[:, c:c + part.shape[1]] = as_type(part, self.dt, dev)
        view, cq = view_of(lens, starts, slots, dev), torch.full((T, self.q_rank + 5), float("nan"), dtype=self.dt, device=dev)
        ops.latent_prep(view, buf, ld, 0, cols[1] if self.of is None else None, w, cq, self.q_rank + 5, self.cache, self.eps, self.rope, self.flag)
        if check_cq:
            assert rel(cq[:, :self.q_rank].float().cpu(), ref.rms(x[:, :self.q_rank].astype(np.float64), self.eps) * self.qn) < (1e-6 if self.dt == F32 else 4e-3)
            assert not cq[:, self.q_rank:].any()
        q_ld = ops.pad_to(self.H * (self.D + self.R), 8)
        qb = torch.zeros((T, q_ld), dtype=self.dt, device=dev)
        qb[:, :self.H * (self.D + self.R)] = as_type(np.concatenate([q[..., self.D:], q[..., :self.D]], -1).reshape(T, -1), self.dt, dev)
        out_cols = ops.pad_to(self.H * self.V, 64)
        out = torch.full((T, out_cols + 8), float("nan"), dtype=self.dt, device=dev)
        gate = dict(gate=buf.view(-1)[cols[2]:], gate_ld=ld)
        wide = self.dt == BF16 and not plain and not any(v % 8 for v in (self.D, self.R, self.V, self.rank)) and self.D + self.R <= 256 and self.V <= 128
        if wide and T > len(lens):          # prompts: the context projected up
            ends = [s + n for s, n in zip(starts, lens)]
            n_ctx, cu = sum(ends), i32(np.concatenate([[0], np.cumsum(ends)]), dev)
            nan = lambda n: torch.full((n_ctx, n), float("nan"), dtype=BF16, device=dev)
            shared, lat, kv = nan(self.R), nan(self.up.ld), nan(self.up.n_out)
            ops.latent_context(view, cu, n_ctx, w, self.cache, shared, lat, self.up.ld)
            L = ops._lib.lib()
            self.up(lat, kv, n_ctx, self.up.n_out, linear_ws=torch.zeros(L.pt_linear_workspace_bytes(min(n_ctx, 32), self.up.n_out, 16), dtype=torch.uint8, device=dev))
            rows = SimpleNamespace(k=kv, v=kv.view(-1)[self.H * self.D:], shared=shared, ld=self.up.n_out, shared_dim=self.R, cu=cu, dim=self.D + self.R, vdim=self.V)
            ops.window_attn(view, qb, q_ld, self.cache, out, out_cols + 8, self.H, self.scale, append=False, max_tokens_per_seq=max(lens), error_flag=self.flag, rope=self.rope,
                            rope_dims=self.R, out_cols=out_cols, gate_per_head=not self.per_value, context=rows, **gate)
        else:
            ws = torch.full((ops.latent_workspace_bytes(T, w, self.dt),), 255, dtype=torch.uint8, device=dev)
            ops.latent_attn(view, qb, q_ld, w, self.cache, out, out_cols + 8, self.scale, self.rope, ws, out_cols=out_cols, error_flag=self.flag, plain=plain, gate_per_value=self.per_value, **gate)
        assert out[:, out_cols:].isnan().all() and not out[:, self.H * self.V:out_cols].any() and int(self.flag.item()) == 0
        return out[:, :self.H * self.V].float().cpu().numpy()

    def oracle(self, x, q, cached=None):
        """cached: the rows of the site whose latents this one reads."""
        T = len(x)
        x, q = x.astype(np.float64), q.astype(np.float64)
        split = np.cumsum([self.q_rank, self.rank, self.R])
        g = np.split(x, split, axis=1)[3]
        _, c, kr, _ = np.split(x if cached is None else cached.astype(np.float64), np.cumsum([self.q_rank if cached is None else self.of.q_rank, self.rank, self.R]), axis=1)
        c = ref.rms(c, self.eps) * self.kn
        k = np.concatenate([np.einsum("hdr,tr->thd", self.uk, c), np.repeat(ref.rotate(kr[:, None], self.base), self.H, 1)], -1)
        q = np.concatenate([q[..., :self.D], ref.rotate(q[..., self.D:], self.base)], -1)
        o = ref.masked_attention(q, k, np.einsum("hvr,tr->thv", self.uv, c), self.scale)
        return (o.reshape(T, -1) * ref.sigmoid(g) if self.per_value else o * ref.sigmoid(g)[..., None]).reshape(T, -1)

    def run(self, x, q, takes, slots, plain):
        got, at = [[] for _ in x], [0] * len(x)
        for take in takes:
            cut = lambda t: np.concatenate([t[i][at[i]:at[i] + n] for i, n in enumerate(take)])
            for i, part in enumerate(np.split(self(cut(x), cut(q), take, at, slots, plain), np.cumsum(take)[:-1])):
                got[i].append(part)
                at[i] += take[i]
        assert at == [len(t) for t in x]
        return [np.concatenate(g) for g in got]
