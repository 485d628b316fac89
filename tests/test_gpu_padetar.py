"""Padetar on the GPU against the plain restatement (oracle/padetar_np.py): every mechanism alone, then whole models in prompts,
portions, batches and decoding, with slots and pages that are used again, and greedy generation through the decode loop."""
import json
import os
import subprocess
import sys
from types import SimpleNamespace

import numpy as np
import pytest
import torch

from oracle import padetar_np as ref
from padetar_util import CONFIGS, config, decoder, layer, weights
from seq_util import PagedAttention, as_type, bf16, greedy_ok, i32, prompt, rel, run_cut, view_of, write_model

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = {"float32": 2e-5, "bfloat16": 2.5e-2}       # rms of the difference over the rms of the logits, whole model
F32, BF16 = torch.float32, torch.bfloat16


# ------------------------------------------------------------------------------------------ residual stream
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("width", [33, 96, 2052])
def test_post_norm(cuda, dtype, width):
    from poptransformer_b200 import ops
    r = np.random.default_rng(1)
    rows, vocab, top, ld, eps = 6, 11, 3, width + 7, 1e-3
    tol = 1e-6 if dtype == F32 else 4e-3
    f = lambda a: as_type(a, F32, cuda)
    table = bf16(r.standard_normal((vocab, width)))
    ids = r.integers(0, vocab, (rows, 4))
    x = torch.full((rows, width), float("nan"), device=cuda)
    h = torch.full((rows, ld), float("nan"), dtype=dtype, device=cuda)
    pos, tok = (torch.full((rows,), -1, dtype=torch.int32, device=cuda) for _ in range(2))
    ops.post_norm(rows, width, eps, dtype, x_out=x, h=h, h_ld=ld, table=as_type(table, dtype, cuda), ids=i32(ids, cuda), ids_ld=4, step=i32([2], cuda), pos_out=pos, id_out=tok)
    assert np.array_equal(x.cpu().numpy(), table[ids[:, 2]]) and np.array_equal(h[:, :width].float().cpu().numpy(), table[ids[:, 2]]) and not h[:, width:].any()
    assert (pos == 2).all() and np.array_equal(tok.cpu().numpy(), ids[:, 2])
    X, y, nw, fw = (r.standard_normal(s).astype(np.float32) for s in ((rows, width), (rows, width), width, width))
    py, pw = r.standard_normal((20, width)).astype(np.float32), r.uniform(0, 1, (rows, top)).astype(np.float32)
    rows_of = r.permutation(20)[:rows * top].reshape(rows, top)
    for dense, pairs, placed in ((True, False, False), (True, True, True), (False, True, True), (True, True, False)):
        where = rows_of if placed else np.arange(rows * top).reshape(rows, top)
        Y = (y if dense else 0) + (np.einsum("tk,tkw->tw", pw, py[where]) if pairs else 0)
        N = X + ref.rms(np.asarray(Y, np.float64), eps) * nw
        kw = dict(y=f(y) if dense else None, y_ld=width, norm_w=f(nw))
        if pairs:
            kw.update(pair_y=f(py), pair_ld=width, top=top, pair_w=f(pw), pair_row=i32(where, cuda) if placed else None)
        x.copy_(f(X))
        ops.post_norm(rows, width, eps, dtype, x_in=x, x_out=x, h=h, h_ld=ld, **kw)
        assert rel(x.cpu(), N) < 1e-6 and rel(h[:, :width].float().cpu(), N) < tol and not h[:, width:].any()
        x.copy_(f(X))
        pick = [4, 1, 4]
        ops.post_norm(3, width, eps, dtype, x_in=x, h=h, h_ld=ld, final_w=f(fw), row_index=i32(pick, cuda), **kw)      # the end of the model
        assert rel(h[:3, :width].float().cpu(), (ref.rms(N, eps) * fw)[pick]) < tol and torch.equal(x, f(X))
        sums = torch.empty_like(x)
        ops.post_norm(rows, width, eps, dtype, x_in=x, x_out=sums, **kw)
        assert rel(sums.cpu(), N) < 1e-6 and torch.equal(x, f(X))


# ------------------------------------------------------------------------------------------ linears
def epilogue_cases(r, n, rows, split):
    """(name, epilogue, features written, oracle of [rows, split] sums)."""
    from poptransformer_b200 import ops
    side, ids = bf16(r.standard_normal((9, 3 * split))), r.integers(0, 9, rows)
    unzip = lambda v: v.reshape(rows, -1, 2, 8)
    return [("store", ops.EPI_STORE, split, lambda v: v, None), ("relu2", ops.EPI_RELU2, split, lambda v: np.maximum(v, 0) ** 2, None),
            ("glu", ops.EPI_GLU, split // 2, lambda v: ref.clamped_glu(unzip(v)[:, :, 0].reshape(rows, -1), unzip(v)[:, :, 1].reshape(rows, -1), 0.8), None),
            ("gelu-mul", ops.EPI_GELU_MUL, split, lambda v: ref.gelu_tanh(v) * side[ids, split:2 * split], (side, ids))]


@pytest.mark.parametrize("rows", [1, 5, 8, 33, 70, 257])
@pytest.mark.parametrize("n,split,k", [(64, None, 40), (160, None, 96), (167, 128, 328), (35, 32, 64), (96, None, 2048), (261, 256, 1100)])
def test_linear_epilogues(cuda, rows, n, split, k):
    """Bias, the four epilogues, and outputs that leave in fp32 behind them; with and without k-slices, in both types and all three kernels."""
    from poptransformer_b200 import ops
    r = np.random.default_rng(2)
    L = ops._lib.lib()
    x, w, b = bf16(r.standard_normal((rows, k))), bf16(r.standard_normal((n, k)) * k ** -0.5), r.standard_normal(n).astype(np.float32)
    sums = 0.7 * (x.astype(np.float64) @ w.T) + b
    flag = torch.zeros(1, dtype=torch.int32, device=cuda)
    ws = dict(linear_ws=torch.zeros(L.pt_linear_workspace_bytes(min(rows, 32), n, 32), dtype=torch.uint8, device=cuda),
              gemm_ws=torch.zeros(L.pt_gemm_workspace_bytes(rows, n, 8), dtype=torch.uint8, device=cuda), error_flag=flag)
    cut = n if split is None else split
    for dt in (F32, BF16):
        for name, epi, feats, f, mul in epilogue_cases(r, n, rows, cut):
            lin = ops.DenseLinear(as_type(w, dt, cuda), dt, bias=as_type(b, F32, cuda), split=split, limit=0.8)
            xp = torch.zeros((rows, lin.ld), dtype=dt, device=cuda)
            xp[:, :k] = as_type(x, dt, cuda)
            out2 = torch.full((rows, n - cut + 3), -7.0, device=cuda)
            kw = dict(mul=(as_type(mul[0], dt, cuda), 3 * cut, cut), mul_ids=i32(mul[1], cuda)) if mul else {}
            for odt in {dt, F32} if not mul else {dt}:
                out = torch.full((rows, feats + 5), -7.0, dtype=odt, device=cuda)
                lin(xp, out, rows, feats + 5, epilogue=epi, alpha=0.7, out2=out2, out2_ld=n - cut + 3, **kw, **ws)
                assert rel(out[:, :feats].float().cpu(), f(sums[:, :cut])) < (5e-6 if odt == F32 else 6e-3), (dt, odt, name)
                assert (out[:, feats:] == -7).all()
                if split is not None:
                    assert rel(out2[:, :n - cut].cpu(), sums[:, cut:]) < 5e-6 and (out2[:, n - cut:] == -7).all(), (dt, name)
    assert int(flag.item()) == 0


@pytest.mark.parametrize("n,k", [(48, 40), (272, 96), (128, 1344)])
@pytest.mark.parametrize("tile", [1, 16, 32, 64, 128])
def test_grouped_linear(cuda, tile, n, k):
    """Every tile of rows has a weight matrix of its own; tiles without one are left alone."""
    from poptransformer_b200 import ops
    r = np.random.default_rng(3)
    G = 5
    L = ops._lib.lib()
    w = [bf16(r.standard_normal((n, k)) * k ** -0.5) for _ in range(G)]
    group_of = np.array([3, 0, 4, 3, 1, 3, 2] if tile == 1 else [3, 0, -1, 3, 1, -1, 2, -1])
    rows = len(group_of) * tile
    for dt in (F32, BF16):
        if dt == F32 and tile != 64:
            continue
        up, plain = (ops.GroupedLinear([as_type(m, dt, cuda) for m in w], dt, limit=lim) for lim in (0.8, 0.0))
        for x_div in (1, 3) if tile == 1 else (1,):
            x = bf16(r.standard_normal((-(-rows // x_div), k)))
            xp = torch.zeros((len(x), up.ld), dtype=dt, device=cuda)
            xp[:, :k] = as_type(x, dt, cuda)
            flag = torch.zeros(1, dtype=torch.int32, device=cuda)
            ws = dict(linear_ws=torch.zeros(L.pt_linear_workspace_bytes(rows, n, 4), dtype=torch.uint8, device=cuda),
                      gemm_ws=torch.zeros(L.pt_gemm_workspace_bytes(rows, n, 8), dtype=torch.uint8, device=cuda), error_flag=flag)
            for lin, epi, feats in ((plain, ops.EPI_STORE, n), (up, ops.EPI_GLU, n // 2)):
                for odt in {dt, F32}:
                    out = torch.full((rows, feats + 1), -7.0, dtype=odt, device=cuda)
                    lin(xp, out, rows, feats + 1, tile, i32(group_of, cuda), x_div=x_div, epilogue=epi, **ws)
                    got = out.float().cpu().numpy()
                    for t, g in enumerate(group_of):
                        mine = got[t * tile:(t + 1) * tile]
                        if g < 0:
                            assert (mine == -7).all()
                            continue
                        v = x[np.arange(t * tile, (t + 1) * tile) // x_div].astype(np.float64) @ w[g].T
                        if epi == ops.EPI_GLU:
                            v = v.reshape(tile, -1, 2, 8)
                            v = ref.clamped_glu(v[:, :, 0].reshape(tile, -1), v[:, :, 1].reshape(tile, -1), 0.8)
                        assert rel(mine[:, :feats], v) < (5e-6 if odt == F32 else 6e-3) and (mine[:, feats:] == -7).all()
            assert int(flag.item()) == 0


def test_glu_rows_and_clamps(cuda):
    """Gate and up rows land where the epilogue looks for them, and each clamp acts on its own side only."""
    from poptransformer_b200 import ops
    ff, limit = 13, 1.5
    gate, up = np.zeros((ff, 8), np.float32), np.zeros((ff, 8), np.float32)
    gate[:, 0], up[:, 1] = 1.0, 1.0
    gate[:, 2], up[:, 3] = 0.01 * np.arange(ff), 0.02 * np.arange(ff)
    xs = np.array([[g, u, 1, 1, 0, 0, 0, 0] for g in (-9.0, -1.0, 1.0, 9.0) for u in (-9.0, -1.0, 1.0, 9.0)], np.float32)
    want = ref.clamped_glu(xs.astype(np.float64) @ gate.T, xs.astype(np.float64) @ up.T, limit)
    lin = ops.DenseLinear(ops.glu_rows(as_type(gate, F32, cuda), as_type(up, F32, cuda), 16), F32, limit=limit)
    out = torch.empty((len(xs), 16), device=cuda)
    lin(as_type(xs, F32, cuda), out, len(xs), 16, epilogue=ops.EPI_GLU)
    assert np.abs(out[:, :ff].cpu().numpy() - want).max() < 1e-5 and not out[:, ff:].any()


# ------------------------------------------------------------------------------------------ router
@pytest.mark.parametrize("tokens,experts,top,tile", [(1, 5, 5, 0), (3, 33, 4, 0), (7, 64, 8, 0), (9, 6, 2, 16), (40, 33, 4, 16), (300, 12, 3, 64), (1500, 7, 1, 128),
                                                     (50, 100, 40, 64), (20, 3, 3, 32), (1901, 11, 5, 64)])
def test_router(cuda, tokens, experts, top, tile):
    from poptransformer_b200 import ops
    r = np.random.default_rng(4)
    z = r.permuted(np.tile(np.arange(experts) * 0.37, (tokens, 1)), axis=1).astype(np.float32)    # no two logits of a token are close
    if experts > 3:
        z[0, 2] = z[0, 3] = z[0].max() + 1                     # equals: the lower index first
    idx, wt = ref.choose(z.astype(np.float64), top)
    expert, pair_row = (torch.full((tokens, top), -5, dtype=torch.int32, device=cuda) for _ in range(2))
    weight = torch.empty((tokens, top), device=cuda)
    kw, tiles = {}, 0
    h = bf16(r.standard_normal((tokens, 24)))
    if tile:
        tiles = ops.moe_max_tiles(tokens, experts, top, tile)
        tile_expert, tile_rows, row_token = (torch.full((n,), -5, dtype=torch.int32, device=cuda) for n in (tiles, tiles, tiles * tile))
        gathered = torch.full((tiles * tile, 24), -7.0, dtype=BF16, device=cuda)
        kw = dict(tile=tile, pair_row=pair_row, tile_expert=tile_expert, tile_rows=tile_rows, row_token=row_token,
                  counts=torch.full((experts,), -5, dtype=torch.int32, device=cuda) if tokens % 2 else None, h=as_type(h, BF16, cuda), h_ld=24, gathered=gathered)
    ops.moe_route(as_type(z, F32, cuda), tokens, experts, top, expert, weight, **kw)
    assert np.array_equal(expert.cpu().numpy(), idx) and np.abs(weight.cpu().numpy() - wt).max() < 1e-6
    if not tile:
        return
    rows, te, rt, g = (t.float().cpu().numpy() for t in (pair_row, tile_expert, row_token, gathered))
    rows, te, rt = rows.astype(int), te.astype(int), rt.astype(int)
    assert len(set(rows.ravel())) == tokens * top and rows.min() >= 0 and rows.max() < tiles * tile
    assert np.array_equal(te[rows // tile], idx)                                    # every pair lies in a tile of its expert
    assert np.array_equal(rt[rows], np.repeat(np.arange(tokens)[:, None], top, 1))
    assert (rt >= 0).sum() == tokens * top and ((rt == -1) | (rt >= 0)).all()
    used = -(-np.bincount(idx.ravel(), minlength=experts) // tile)
    assert np.array_equal(np.bincount(te[te >= 0], minlength=experts), used) and (te[used.sum():] == -1).all()
    assert np.array_equal(tile_rows.cpu().numpy(), (rt.reshape(tiles, tile) >= 0).sum(1))
    assert all((np.diff(np.sort(rows[idx == e])) == 1).sum() >= (idx == e).sum() - used[e] and (np.diff(rows[idx == e]) > 0).all() for e in range(experts))   # in order
    assert np.array_equal(g, np.where(rt[:, None] >= 0, h[np.maximum(rt, 0)], -7))


# ------------------------------------------------------------------------------------------ attention
ROT = [  # heads, kv heads, dim, rotated dims, scaling
    (4, 2, 32, 32, (4.0, 1.0, 4.0, 64)), (6, 1, 40, 24, None), (16, 2, 128, 128, (8.0, 2.0, 8.0, 512)), (5, 5, 20, 6, (2.0, 1.0, 3.0, 32)), (2, 1, 64, 0, None),
    (3, 1, 160, 64, None), (24, 2, 72, 72, None), (8, 8, 16, 2, (4.0, 1.0, 4.0, 64))]


def rope_table(n, dims, base, scaling, dev):
    from poptransformer_b200.padetar import rope_frequencies
    if not dims:
        return None, np.zeros(0)
    sc = dict(zip(("factor", "low", "high", "original"), scaling)) if scaling else None
    a = np.arange(n)[:, None] * rope_frequencies(dims, base, sc)
    return as_type(np.stack([np.cos(a), np.sin(a)], -1), F32, dev), ref.frequencies(dims, base, sc)


@pytest.mark.parametrize("dtype,plain", [(F32, True), (BF16, True), (BF16, False)])
@pytest.mark.parametrize("H,G,D,dims,scaling", ROT)
def test_attention_with_norm_and_rotation(cuda, dtype, plain, H, G, D, dims, scaling):
    """The values are the keys as they come; three sequences of unequal length in portions (down to two tokens) and single tokens."""
    r = np.random.default_rng(5)
    lens, eps, scale = [215, 70, 134], 1e-2, 2.5 * D ** -0.5
    qn, kn = 1 + 0.3 * r.standard_normal(D), 1 + 0.3 * r.standard_normal(D)
    table, freq = rope_table(256, dims, 100.0, scaling, cuda)
    q, k = ([bf16(r.standard_normal((n, h, D))) for n in lens] for h in (H, G))
    att = PagedAttention(cuda, dtype, 3, G, D, D, 256)
    kw = dict(q_norm=as_type(qn, F32, cuda), k_norm=as_type(kn, F32, cuda), eps=eps, rope=table, rope_dims=dims, out_scale=0.6, pad_cols=16)
    got, at, slots = [[] for _ in lens], [0, 0, 0], [2, 0, 1]
    for take in ([1, 2, 1], [63, 1, 64], [3, 2, 1], [100, 33, 60], [2, 2, 2], [1, 1, 1], [1, 1, 1], [10, 24, 1], [1, 1, 1], [33, 3, 2]):
        cut = lambda t: np.concatenate([t[i][at[i]:at[i] + n] for i, n in enumerate(take)])
        o = att(cut(q), cut(k), None, take, at, slots, scale, 0, 0, None, plain, **kw)
        for i, part in enumerate(np.split(o, np.cumsum(take)[:-1])):
            got[i].append(part)
            at[i] += take[i]
    assert at == lens
    for i in range(3):
        qr, kr = (ref.rotate(ref.rms(t[i].astype(np.float64), eps) * n, freq) for t, n in ((q, qn), (k, kn)))
        want = 0.6 * ref.causal_attention(qr, kr, k[i].astype(np.float64), scale)
        err = np.abs(np.concatenate(got[i]) - want).max(1)
        assert err.max() < (2e-5 if dtype == F32 else 4e-2), (i, int(err.argmax()), float(err.max()))
        assert rel(np.concatenate(got[i]), want) < (2e-6 if dtype == F32 else 8e-3)


@pytest.mark.parametrize("dtype,plain", [(F32, True), (BF16, True), (BF16, False)])
def test_one_far_key(cuda, dtype, plain):
    """One key stands out for the queries of every later token (the same direction, no rotation in its dimensions) and carries a value
    of its own: every query from that key on must find it, and none before, in prompts and in decoding, at page borders too."""
    n, H, G, D = 200, 2, 1, 32
    special = [0, 1, 62, 63, 64, 65, 127, 128, 129, 198]
    r = np.random.default_rng(6)
    B = len(special)
    q, k = bf16(0.02 * r.standard_normal((B, n, H, D))), bf16(0.3 * r.standard_normal((B, n, G, D)))
    q[..., 31] = 1.0
    for b, j in enumerate(special):
        k[b, j] = 0.0
        k[b, j, :, 31] = 4.0
    table, freq = rope_table(n, 16, 100.0, None, cuda)
    one = np.ones(D)
    rot = lambda x: ref.rotate(ref.rms(x.astype(np.float64), 1e-6), freq)
    want = np.stack([ref.causal_attention(rot(q[b]), rot(k[b]), k[b].astype(np.float64), 1.0) for b in range(B)])
    seen = np.arange(n)[None] >= np.array(special)[:, None]
    assert ((want[:, :, 31] > 3) == seen).all()
    kw = dict(q_norm=as_type(one, F32, cuda), k_norm=as_type(one, F32, cuda), eps=1e-6, rope=table, rope_dims=16)
    att = PagedAttention(cuda, dtype, B, G, D, D, 256)
    flat = lambda t, a, b: t[:, a:b].reshape(B * (b - a), *t.shape[2:])
    split = n - 75
    got = [att(flat(q, 0, split), flat(k, 0, split), None, [split] * B, [0] * B, range(B), 1.0, 0, 0, None, plain, **kw).reshape(B, split, -1)]
    for i in range(split, n):
        got.append(att(flat(q, i, i + 1), flat(k, i, i + 1), None, [1] * B, [i] * B, range(B), 1.0, 0, 0, None, plain, **kw).reshape(B, 1, -1))
    got = np.concatenate(got, 1)
    wrong = np.argwhere((got[:, :, 31] > 3) != seen)
    assert not len(wrong), [(special[b], int(i)) for b, i in wrong[:5]]
    assert np.abs(got - want).max() < (1e-4 if dtype == F32 else 5e-2)


# ------------------------------------------------------------------------------------------ matrix memory
MEM_SHAPES = [  # heads, key width, value width, gate cap
    (4, 16, 24, 10.0), (2, 64, 32, 15.0), (3, 24, 40, 3.0), (1, 128, 160, 12.0), (2, 256, 64, 15.0), (3, 19, 33, 8.0), (2, 8, 8, 1.0), (1, 40, 100, 20.0), (2, 320, 16, 5.0)]


class MemorySite:
    """One matrix-memory call site: its state, and the oracle's view of the same."""

    def __init__(self, dev, dt, n_slots, heads, dim, vdim, cap, seed=7):
        from poptransformer_b200 import ops
        L = ops._lib.lib()
        self.ops, self.dev, self.dt, self.H, self.N, self.P, self.cap = ops, dev, dt, heads, dim, vdim, cap
        self.norm = 1 + 0.3 * np.random.default_rng(seed).standard_normal(heads * vdim)
        self.w = SimpleNamespace(heads=heads, dim=dim, vdim=vdim, cap=cap, eps=1e-4, norm_w=as_type(self.norm, F32, dev))
        # whatever an earlier sequence left must not matter
        self.state, self.nm = (torch.full((n_slots, L.pt_mlstm_state_floats(heads, dim, vdim, k)), float("nan"), device=dev) for k in (0, 1))
        self.ws = torch.zeros(L.pt_mlstm_workspace_bytes(4096, n_slots, heads, dim, vdim), dtype=torch.uint8, device=dev)
        self.width = heads * (2 * dim + 2 * vdim)

    def inputs(self, n, seed, spread=1.0):
        r = np.random.default_rng(seed)
        g = np.concatenate([r.uniform(-1, 1, (n, self.H)) * self.cap * spread, r.uniform(-1, 2, (n, self.H)) * self.cap * spread], 1)
        return bf16(r.standard_normal((n, self.width))), g.astype(np.float32)

    def __call__(self, x, gates, lens, starts, slots, plain):
        ops, dev, T = self.ops, self.dev, x.shape[0]
        lead, ld = 8, ops.pad_to(self.width, 8) + 8
        buf = torch.zeros((T, ld), dtype=self.dt, device=dev)
        buf[:, lead:lead + self.width] = as_type(x, self.dt, dev)
        cols, inner = lead + np.cumsum([0, self.H * self.N, self.H * self.N, self.H * self.P]), self.H * self.P
        out_ld, first = ops.pad_to(inner, 64) + 16, 8
        out = torch.full((T, out_ld), float("nan"), dtype=self.dt, device=dev)
        self.ws[1 << 18:] = 255
        ops.mlstm(view_of(lens, starts, slots, dev), buf, ld, cols.tolist(), as_type(gates, F32, dev), 2 * self.H, out.view(-1)[first:], out_ld, self.w, self.state, self.nm,
                  torch.empty((T, inner), device=dev), self.ws, out_scale=0.5, out_cols=out_ld - 16, plain=plain)
        assert not out[:, first + inner:out_ld - 8].any() and out[:, :first].isnan().all() and out[:, out_ld - 8:].isnan().all()
        return out[:, first:first + inner].float().cpu().numpy()

    def split(self, x):
        q, k, v, g = np.split(x.astype(np.float64), np.cumsum([self.H * self.N, self.H * self.N, self.H * self.P]), axis=1)
        T = len(x)
        return q.reshape(T, self.H, self.N) * self.N ** -0.5, k.reshape(T, self.H, self.N), v.reshape(T, self.H, self.P), g

    def oracle(self, x, gates):
        q, k, v, g = self.split(x)
        z = gates.astype(np.float64)
        o = ref.matrix_memory(q, k, v, *ref.memory_gates(z[:, :self.H], z[:, self.H:], self.cap))
        return 0.5 * ref.rms(o, 1e-4).reshape(len(x), -1) * self.norm * ref.sigmoid(g)

    def run(self, x, gates, takes, slots, plain):
        """Sequences in portions; the outputs of each."""
        got, at = [[] for _ in x], [0] * len(x)
        for take in takes:
            cut = lambda t: np.concatenate([t[i][at[i]:at[i] + n] for i, n in enumerate(take)])
            o = self(cut(x), cut(gates), take, at, slots, plain)
            for i, part in enumerate(np.split(o, np.cumsum(take)[:-1])):
                got[i].append(part)
                at[i] += take[i]
        assert at == [len(t) for t in x]
        return [np.concatenate(g) for g in got]


@pytest.mark.parametrize("dtype,plain", [(F32, True), (BF16, True), (BF16, False)])
@pytest.mark.parametrize("heads,dim,vdim,cap", MEM_SHAPES)
def test_matrix_memory(cuda, dtype, plain, heads, dim, vdim, cap):
    """Unequal sequences in portions (single tokens, two tokens, around the chunk of 64, long), state carried over."""
    site = MemorySite(cuda, dtype, 4, heads, dim, vdim, cap)
    lens = [205, 75, 136]
    x, g = zip(*(site.inputs(n, 8 + i) for i, n in enumerate(lens)))
    takes = ([1, 1, 2], [1, 1, 1], [1, 1, 1], [63, 2, 65], [64, 2, 1], [66, 3, 60], [1, 1, 1], [1, 60, 1], [7, 4, 4])
    for i, got in enumerate(site.run(x, g, takes, [3, 0, 1], plain)):
        want = site.oracle(x[i], g[i])
        per_token = np.sqrt(((got - want) ** 2).mean(1)) / np.sqrt((want ** 2).mean())
        assert rel(got, want) < (2e-5 if dtype == F32 else 8e-3), i
        assert per_token.max() < (3e-4 if dtype == F32 else 6e-2), (i, int(per_token.argmax()))


@pytest.mark.parametrize("dtype,plain", [(F32, True), (BF16, True), (BF16, False)])
def test_memory_of_one_early_token(cuda, dtype, plain):
    """A token whose input gate is wide open while all others' are shut, under forget gates that hardly forget: every later query finds
    its value (200 tokens on, across chunks, portions and decoding), and a token with a shut forget gate wipes it."""
    H, N, P, cap, n = 2, 32, 24, 15.0, 260
    for at, wipe in ((0, None), (5, None), (63, None), (64, 190), (65, 127), (70, 128)):
        site = MemorySite(cuda, dtype, 1, H, N, P, cap)
        x, g = site.inputs(n, 20 + at)
        g[:, :H], g[:, H:] = -4 * cap, 4 * cap
        g[at, :H] = 1.5
        if wipe is not None:
            g[wipe, H:] = -4 * cap
        cols = np.cumsum([H * N, H * N, H * P])
        x[:, :H * N] = 1.0                                                 # every query the same, and the key of the one token along it
        x[:, cols[0]:cols[1]] = bf16(0.05 * np.random.default_rng(1).standard_normal((n, H * N)))
        x[at, cols[0]:cols[1]] = 1.0
        x[at, cols[1]:cols[2]] = np.where(np.arange(H * P) % 2, 3.0, -3.0)
        x[:, cols[2]:] = 8.0
        want = site.oracle(x, g)
        sign = want / (0.5 * site.norm) * np.where(np.arange(H * P) % 2, 1, -1)
        held = slice(at, n if wipe is None else wipe)
        assert (sign[held] > 0.8).all() and (wipe is None or not (sign[wipe + 1:] > 0.8).all(1).any())
        got = site.run([x], [g], [[100], [2], [77], [64]] + [[1]] * 17, [0], plain)[0]
        per_token = np.sqrt(((got - want) ** 2).mean(1)) / np.sqrt((want ** 2).mean())
        assert per_token[held].max() < (1e-4 if dtype == F32 else 2e-2), (at, int(per_token[held].argmax()) + at)
        if wipe is not None:
            assert per_token[wipe:].max() < (3e-3 if dtype == F32 else 0.1), (at, int(per_token[wipe:].argmax()) + wipe)


@pytest.mark.parametrize("dtype,plain", [(F32, True), (BF16, False)])
def test_memory_denominator(cuda, dtype, plain):
    """Both sides of max(|n . q|, exp(-m)), and the constant behind it: with large gates it weighs as much as the sum itself."""
    H, N, P, n = 2, 16, 16, 150
    for cap, zi, qs, side in ((15.0, 60.0, 1e-5, "constant"), (6.0, 4.0, 4.0, "sum"), (8.0, -60.0, 0.3, "floor")):
        site = MemorySite(cuda, dtype, 1, H, N, P, cap)
        x, g = site.inputs(n, 30)
        x[:, :H * N] = bf16(x[:, :H * N] * qs)
        g[:, :H] = zi
        q, k, v, _ = site.split(x)
        li, lf = ref.memory_gates(g[:, :H].astype(np.float64), g[:, H:].astype(np.float64), cap)
        site.w.eps = 1e-12                    # (the per-head norm would hide a common factor of the denominator otherwise)
        o = ref.matrix_memory(q, k, v, li, lf)
        want = 0.5 * o.reshape(n, -1)
        # the outputs before the norm: undo it by handing the kernel's own o over
        y = torch.empty((n, H * P), device=cuda)
        a = site.ops
        buf = torch.zeros((n, a.pad_to(site.width, 8)), dtype=dtype, device=cuda)
        buf[:, :site.width] = as_type(x, dtype, cuda)
        out = torch.empty((n, 64), dtype=dtype, device=cuda)
        cols = np.cumsum([0, H * N, H * N, H * P]).tolist()
        a.mlstm(view_of([n], [0], [0], cuda), buf, buf.shape[1], cols, as_type(g, F32, cuda), 2 * H, out, 64, site.w, site.state, site.nm, y, site.ws, plain=plain)
        assert rel(0.5 * y.cpu().numpy(), want) < (2e-5 if dtype == F32 else 5e-3), side
        for t in (n - 1,):                    # the last token once more as a decode step, from the state before it
            a.mlstm(view_of([t], [0], [0], cuda), buf, buf.shape[1], cols, as_type(g, F32, cuda), 2 * H, out, 64, site.w, site.state, site.nm, y, site.ws, plain=plain)
            a.mlstm(view_of([1], [t], [0], cuda), buf[t:].contiguous(), buf.shape[1], cols, as_type(g[t:], F32, cuda), 2 * H, out, 64, site.w, site.state, site.nm, y, site.ws,
                    plain=plain)
            assert rel(0.5 * y[:1].cpu().numpy(), want[t:]) < (2e-5 if dtype == F32 else 5e-3), side


# ------------------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_model_prompts_portions_and_decoding(cuda, name, dtype):
    cfg = CONFIGS[name]
    w = weights(cfg, seed=11)
    n = 150
    tokens = prompt(n, cfg["vocab"])
    sums = []
    want = ref.PadetarOracle(cfg, w).forward(tokens, sums)
    dec = decoder(cfg, w, 3, 192, dtype)
    dec.rows_prompt = dec._row_buffers(n)
    for r in (dec.rows_prompt, dec.rows_decode):     # nothing may depend on what the buffers held (padding rows of the experts' tiles, padded columns)
        for t in vars(r).values():
            if torch.is_tensor(t) and t.is_floating_point():
                t.fill_(float("nan"))
    for plain in (False, True):
        dec.plain = plain
        got_sums, s = [], dec.open()
        whole = dec.extend([(s, tokens, list(range(n)))], layer_sums=got_sums).cpu().numpy()
        dec.close(s)
        assert len(got_sums) == len(sums)
        for i, (a, b) in enumerate(zip(got_sums, sums)):
            assert rel(a.cpu(), b) < TOL[dtype], f"after layer {i}"
        assert rel(whole, want) < TOL[dtype]
        for cuts in ([1] * n, [2] * (n // 2), [64, 64, 22], [63, 2, 65, 20], [100] + [1] * 50):
            got = run_cut(dec, tokens, cuts)
            per = np.sqrt(((got - whole) ** 2).mean(1)) / np.sqrt((whole ** 2).mean())
            # (a token whose sublayer output nearly cancels before its norm amplifies the bf16 roundings of its inputs)
            assert per.max() < (1e-4 if dtype == "float32" else 0.3), (cuts[:4], int(per.argmax()), float(per.max()))
            assert np.sort(per)[-4] < (1e-4 if dtype == "float32" else 4e-2), (cuts[:4], np.argsort(per)[-4:])
            assert rel(got, want) < TOL[dtype]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_unequal_batch_against_each_alone(cuda, dtype):
    cfg = CONFIGS["mixed"]
    w = weights(cfg, seed=12)
    lens = [1, 97, 2, 40, 64, 130]
    toks = [prompt(n + 12, cfg["vocab"], i) for i, n in enumerate(lens)]
    alone = decoder(cfg, w, 1, 256, dtype)
    want = [run_cut(alone, t, [n, *[1] * 12]) for t, n in zip(toks, lens)]
    dec = decoder(cfg, w, len(lens), 256, dtype)
    dec.PROMPT_TOKENS = 100                       # the prompt batch takes several passes
    seqs = [dec.open() for _ in lens]
    got = [[g] for g in np.split(dec.extend([(s, t[:n], list(range(n))) for s, t, n in zip(seqs, toks, lens)]).cpu().numpy(), np.cumsum(lens)[:-1])]
    live = list(range(len(lens)))
    for step in range(12):
        if step in (4, 8):                        # some end earlier; the rest go on in another order
            dec.close(seqs[live.pop(1)])
            live = live[::-1]
        o = dec.extend([(seqs[i], toks[i][lens[i] + step:lens[i] + step + 1], [0]) for i in live]).cpu().numpy()
        for k, i in enumerate(live):
            got[i].append(o[k:k + 1])
    for g, t in zip(got, want):
        g = np.concatenate(g)
        assert rel(g, t[:len(g)]) < TOL[dtype]


def test_more_rows_than_the_skinny_kernels_take(cuda):
    cfg = CONFIGS["wide-heads"]
    w = weights(cfg, seed=13)
    B = 45
    toks = [prompt(20, cfg["vocab"], i) for i in range(B)]
    picked = (0, 17, 31, 32, 44)
    want = np.stack([ref.PadetarOracle(cfg, w).forward(toks[b])[18:] for b in picked])
    for dtype in ("float32", "bfloat16"):
        dec = decoder(cfg, w, B, 64, dtype)
        seqs = [dec.open() for _ in range(B)]
        dec.extend([(s, t[:18], []) for s, t in zip(seqs, toks)])
        got = np.stack([dec.extend([(s, t[i:i + 1], [0]) for s, t in zip(seqs, toks)]).cpu().numpy() for i in (18, 19)], 1)
        assert rel(got[list(picked)], want) < 1.5 * TOL[dtype]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_slots_and_pages_are_used_again(cuda, dtype):
    """A pool that only fits one batch at a time; before every batch all caches and states are poisoned."""
    cfg = CONFIGS["mixed"]
    w = weights(cfg, seed=14)
    fresh = decoder(cfg, w, 1, 192, dtype)
    dec = decoder(cfg, w, 3, 192, dtype, n_pages=5)
    for rnd, lens in enumerate([[120, 60], [10, 64, 65], [190], [3, 130], [1, 1, 1]]):
        for t in [c.pool for c in dec.caches.values()] + list(dec.states.values()) + list(dec.norms.values()):
            t.fill_(float("nan"))
        toks = [prompt(n + 2, cfg["vocab"], 10 * rnd + i) for i, n in enumerate(lens)]
        seqs = [dec.open() for _ in lens]
        got = dec.extend([(s, t[:-2], [n - 1]) for s, t, n in zip(seqs, toks, lens)]).cpu().numpy()
        more = [dec.extend([(s, t[n + k:n + k + 1], [0]) for s, t, n in zip(seqs, toks, lens)]).cpu().numpy() for k in range(2)]
        for i, s in enumerate(seqs):
            want = run_cut(fresh, toks[i], [lens[i], 1, 1])
            assert rel(np.stack([got[i], more[0][i], more[1][i]]), want[lens[i] - 1:]) < (1e-5 if dtype == "float32" else 2e-2)
            dec.close(s)
    assert dec.slots.free_pages == 5 and dec.slots.free_slots == 3


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(cuda, dtype):
    cfg = CONFIGS["mixed"]
    w = weights(cfg, seed=15)
    tokens = prompt(340, cfg["vocab"])
    dec = decoder(cfg, w, 1, 384, dtype)
    got = run_cut(dec, tokens, [9] + [1] * 331)
    want = ref.PadetarOracle(cfg, w).forward(tokens)
    assert rel(got, want) < TOL[dtype]
    assert rel(got[-20:], want[-20:]) < TOL[dtype]


def test_first_tokens(cuda):
    """Prompts of 1 .. 9 tokens."""
    cfg = config([layer(), layer(rot=0, cap=2.0)], width=64)
    w = weights(cfg, seed=16)
    orc = ref.PadetarOracle(cfg, w)
    for dtype in ("float32", "bfloat16"):
        dec = decoder(cfg, w, 9, 64, dtype)
        toks = [prompt(n, cfg["vocab"], n) for n in range(1, 10)]
        seqs = [dec.open() for _ in toks]
        got = dec.extend([(s, t, list(range(len(t)))) for s, t in zip(seqs, toks)]).cpu().numpy()
        assert rel(got, np.concatenate([orc.forward(t) for t in toks])) < TOL[dtype]


def test_missing_parts_would_show(cuda):
    """The comparison above is sharp: an oracle with one part changed is far from the kernels."""
    cfg = CONFIGS["mixed"]
    w = weights(cfg, seed=22)
    tokens = prompt(140, cfg["vocab"])
    dec = decoder(cfg, w, 1, 192, "bfloat16")
    s = dec.open()
    got = dec.extend([(s, tokens, list(range(140)))]).cpu().numpy()
    assert rel(got, ref.PadetarOracle(cfg, w).forward(tokens)) < TOL["bfloat16"]

    def changed(edit_cfg=None, edit_w=None):
        c, v = json.loads(json.dumps(cfg)), dict(w)
        for f, x in ((edit_cfg, c), (edit_w, v)):
            if f:
                f(x)
        return rel(got, ref.PadetarOracle(c, v).forward(tokens))

    mix = lambda c, i: c["layers"][i]["mixer"]
    edits = [dict(edit_cfg=lambda c: mix(c, 0)["left"]["rot"].update(base=2e4)), dict(edit_cfg=lambda c: mix(c, 0)["left"]["rot"].pop("scaling")),
             dict(edit_cfg=lambda c: mix(c, 1)["left"]["rot"].update(dims=22)), dict(edit_cfg=lambda c: mix(c, 0)["right"].update(gate_cap=6.0)),
             dict(edit_cfg=lambda c: mix(c, 0).update(left_scale=0.8)), dict(edit_cfg=lambda c: c["layers"][0]["mlp"]["expert"].update(limit=0.4)),
             dict(edit_cfg=lambda c: c["layers"][0]["mlp"]["shared"].update(limit=0.9)), dict(edit_cfg=lambda c: c["layers"][0]["mlp"]["router"].update(top=1)),
             dict(edit_w=lambda v: v.update({"l0.mix.right.f.b": v["l0.mix.right.f.b"] - 1})), dict(edit_w=lambda v: v.update({"l0.mix.left.k.b": 0 * v["l0.mix.left.k.b"]})),
             dict(edit_w=lambda v: v.update({"l2.side.norm": 0 * v["l2.side.norm"]}))]
    assert [i for i, e in enumerate(edits) if changed(**e) < 1.4 * TOL["bfloat16"]] == []


# ------------------------------------------------------------------------------------------ the decode loop
@pytest.mark.parametrize("dtype,tol", [("float32", 1e-4), ("bfloat16", 8e-2)])
def test_greedy_generation(cuda, dtype, tol):
    cfg = CONFIGS["mixed"]
    w = weights(cfg, seed=17)
    orc = ref.PadetarOracle(cfg, w)
    max_len, lens = 80, [3, 20, 9]
    dec = decoder(cfg, w, 3, max_len, dtype, pad_id=-1)
    ids = np.full((3, max_len), -1, np.int32)
    for b, n in enumerate(lens):
        ids[b, :n] = prompt(n, cfg["vocab"], b)
    eager = dec.run(ids, max_loop=max_len - 1)["Loop:0"]
    assert all((eager[b, :n] == ids[b, :n]).all() for b, n in enumerate(lens)) and (eager >= 0).all()
    assert greedy_ok(orc, eager, lens, tol) > 0.9
    dec.capture()
    assert np.array_equal(dec.run(ids, max_loop=max_len - 1)["Loop:0"], eager)          # one CUDA graph per step, state of the run before left behind
    pre = dec.run(ids, max_loop=max_len - 1, prefill=True)["Loop:0"]
    assert greedy_ok(orc, pre, lens, tol) > 0.9
    # sequences of their own on the same decoder, then the loop again
    s = dec.open()
    dec.extend([(s, ids[1, :20], [])])
    dec.close(s)
    assert np.array_equal(dec.run(ids, max_loop=max_len - 1)["Loop:0"], eager)


def test_prefill_in_portions_and_early_stop(cuda):
    cfg = CONFIGS["mixed"]
    w = weights(cfg, seed=18)
    ids = np.full((2, 120), -1, np.int32)
    for b in range(2):
        ids[b, :90] = prompt(90, cfg["vocab"], b)
    dec = decoder(cfg, w, 2, 120, "float32", pad_id=-1)
    want = dec.run(ids, max_loop=119)["Loop:0"]
    dec.reset(ids)
    assert dec.prefill(chunk=33) == 89
    for _ in range(89, 119):
        dec.step()
    assert np.array_equal(dec.ids.cpu().numpy(), want)
    eos = int(want[0, 95])                                   # row 0 stops there; row 1 wherever it produces the same id, if it does
    stop = decoder(cfg, w, 2, 120, "float32", pad_id=-1, eos_id=eos, early_stop=True)
    slow, fast = stop.run(ids, max_loop=119), stop.run(ids, max_loop=119, prefill=True)
    assert np.array_equal(slow["Loop:0"], fast["Loop:0"]) and np.array_equal(slow["Loop:1"], fast["Loop:1"])


def test_streams_share_weights(cuda):
    from poptransformer_b200.loop import MultiStreamLoop
    cfg = CONFIGS["mixed"]
    dec = decoder(cfg, weights(cfg, seed=19), 1, 40, "bfloat16", pad_id=-1)
    reqs = []
    for i in range(5):
        ids = np.full((1, 40), -1, np.int32)
        ids[0, :4 + i] = prompt(4 + i, cfg["vocab"], i)
        reqs.append(ids)
    want = [dec.run(r, max_loop=39)["Loop:0"] for r in reqs]
    got = MultiStreamLoop(dec, 3).run(reqs, max_loop=39)
    assert all(np.array_equal(g["Loop:0"], x) for g, x in zip(got, want))


# ------------------------------------------------------------------------------------------ programs
def test_trace_replay_program(cuda, tmp_path):
    cfg = CONFIGS["mixed"]
    w = weights(cfg, seed=20)
    model, out = tmp_path / "model", tmp_path / "out"
    model.mkdir(); out.mkdir()
    write_model(str(model), cfg, w)
    toks = {"a": prompt(70, cfg["vocab"], 1), "b": prompt(5, cfg["vocab"], 2), "c": prompt(66, cfg["vocab"], 3)}
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks["a"][:68].tolist(), "want": [0, 67]}, {"id": "b", "tokens": toks["b"][:3].tolist(), "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": [int(toks["b"][3])], "want": []}, {"id": "a", "tokens": [int(toks["a"][68])], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": [int(toks["a"][69])], "want": [0]}, {"id": "b", "tokens": [int(toks["b"][4])], "want": [0]}], "end": ["a", "b"]},
             {"step": 3, "entries": [{"id": k, "tokens": toks["c"][:n].tolist(), "want": [n - 1]} for k, n in (("c", 66), ("d", 2), ("e", 9))], "end": ["c", "d", "e"]}]
    orc = {k: ref.PadetarOracle(cfg, w).forward(t) for k, t in toks.items()}
    want = {0: orc["a"][[0, 67]], 2: np.stack([orc["a"][69], orc["b"][4]]), 3: orc["c"][[65, 1, 8]]}
    for dtype in ("float32", "bfloat16"):
        p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(model), "--dtype", dtype, "--out", str(out), "--max-tokens", "80"],
                           input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
        assert p.returncode == 0, p.stderr[-2000:]
        assert [ln for ln in p.stdout.splitlines() if ln.startswith("done")] == [f"done {i}" for i in range(4)]
        assert sorted(os.listdir(out)) == ["0.f32", "2.f32", "3.f32"]
        for k, exp in want.items():
            got = np.fromfile(out / f"{k}.f32", "<f4").reshape(exp.shape)
            assert rel(got, exp) < TOL[dtype]
            os.unlink(out / f"{k}.f32")


def test_generate_command(cuda, tmp_path):
    cfg = CONFIGS["no-side"]
    w = weights(cfg, seed=21)
    write_model(str(tmp_path), cfg, w)
    a, b = prompt(6, cfg["vocab"], 1).tolist(), prompt(3, cfg["vocab"], 2).tolist()
    cmd = [sys.executable, "-m", "poptransformer_b200", "generate", "--model", str(tmp_path), "--prompt", ",".join(map(str, a)), "--prompt", ",".join(map(str, b)),
           "--new", "10", "--dtype", "float32", "--prefill"]
    p = subprocess.run(cmd, capture_output=True, text=True, timeout=300, cwd=ROOT)
    assert p.returncode == 0, p.stderr[-2000:]
    rows = [json.loads(ln)["ids"] for ln in p.stdout.splitlines()]
    assert [len(r) for r in rows] == [16, 16] and rows[0][:6] == a and rows[1][:3] == b
    assert greedy_ok(ref.PadetarOracle(cfg, w), np.array(rows), [6, 3], 1e-4) == 1.0
