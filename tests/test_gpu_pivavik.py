"""Pivavik on the GPU against the plain restatement (oracle/pivavik_np.py): every mechanism alone, then whole models in prompts, portions,
batches and decoding, with slots and pages that are used again, and greedy generation through the decode loop."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from oracle import pivavik_np as ref
from latent_util import LatentSite
from pivavik_util import CONFIGS, attention, config, decoder, dense, latent, moe, weights
from seq_util import PagedAttention, as_type, bf16, greedy_ok, i32, prompt, rel, run_cut, write_model

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = {"float32": 2e-5, "bfloat16": 2.5e-2}       # rms of the difference over the rms of the logits, whole model
F32, BF16 = torch.float32, torch.bfloat16


# ------------------------------------------------------------------------------------------ residual stream
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("width", [33, 96, 2052])
def test_norm_before_a_layer(cuda, dtype, width):
    """The residual step that adds as it is and normalises what is read next, the embedding with a norm, and a second copy of the stream."""
    from poptransformer_b200 import ops
    r = np.random.default_rng(1)
    rows, vocab, top, eps = 6, 11, 3, 1e-3
    ld, tol = 2 * width + 9, 1e-6 if dtype == F32 else 4e-3
    f = lambda a: as_type(a, F32, cuda)
    back = lambda t: t.float().cpu().numpy()
    table, ids = bf16(r.standard_normal((vocab, width))), r.integers(0, vocab, (rows, 4))
    nw, fw = 1 + 0.3 * r.standard_normal(width), 1 + 0.3 * r.standard_normal(width)
    x = torch.full((rows, width), float("nan"), device=cuda)
    pos = torch.full((rows,), -1, dtype=torch.int32, device=cuda)
    # the embedding: its norm, then beside each other the stream and its copy with zeros behind it
    both = torch.full((rows, ld), -7.0, dtype=dtype, device=cuda)
    flat = both.view(-1)
    ops.post_norm(rows, width, eps, dtype, x_out=x, h=both, h_ld=ld, h_cols=width, copy=flat[width:], copy_ld=ld, copy_cols=width + 4, table=as_type(table, dtype, cuda), ids=i32(ids, cuda),
                  ids_ld=4, step=i32([2], cuda), pos_out=pos, norm_w=f(nw))
    want = ref.rms(table[ids[:, 2]].astype(np.float64), eps) * nw
    assert rel(x.cpu(), want) < 1e-6 and rel(back(both[:, :width]), want) < tol and rel(back(both[:, width:2 * width]), want) < tol and (pos == 2).all()
    assert not both[:, 2 * width:2 * width + 4].any() and (both[:, 2 * width + 4:] == -7).all()
    h = torch.full((rows, width + 3), float("nan"), dtype=dtype, device=cuda)
    ops.post_norm(rows, width, eps, dtype, x_out=x, h=h, h_ld=width + 3, table=as_type(table, dtype, cuda), ids=i32(ids, cuda), ids_ld=4, norm_w=f(nw), final_w=f(fw))
    want = ref.rms(ref.rms(table[ids[:, 0]].astype(np.float64), eps) * nw, eps) * fw
    assert rel(back(h[:, :width]), want) < tol and not h[:, width:].any()
    # residual steps: a dense output, experts' outputs with and without weights
    X, y = (r.standard_normal((rows, width)).astype(np.float32) for _ in range(2))
    py, pw = r.standard_normal((20, width)).astype(np.float32), r.uniform(0, 1, (rows, top)).astype(np.float32)
    where = r.permutation(20)[:rows * top].reshape(rows, top)
    for weighted in (True, False):
        N = X.astype(np.float64) + y + np.einsum("tk,tkw->tw", pw if weighted else np.ones_like(pw), py[where])
        kw = dict(y=f(y), y_ld=width, pair_y=f(py), pair_ld=width, top=top, pair_w=f(pw) if weighted else None, pair_row=i32(where, cuda))
        x.copy_(f(X))
        ops.post_norm(rows, width, eps, dtype, x_in=x, x_out=x, h=h, h_ld=width + 3, final_w=f(fw), **kw)
        assert rel(x.cpu(), N) < 1e-6 and rel(back(h[:, :width]), ref.rms(N, eps) * fw) < tol
        x.copy_(f(X))
        both.fill_(-7)
        ops.post_norm(rows, width, eps, dtype, x_in=x, x_out=x, h=both, h_ld=ld, h_cols=width, **kw)         # the stream itself, for a product that mixes it
        assert rel(x.cpu(), N) < 1e-6 and rel(back(both[:, :width]), N) < tol and (both[:, width:] == -7).all()
    ops.post_norm(3, width, eps, dtype, x_in=f(X), h=h, h_ld=width + 3, final_w=f(fw), row_index=i32([4, 1, 4], cuda))       # nothing is added
    assert rel(back(h[:3, :width]), (ref.rms(X.astype(np.float64), eps) * fw)[[4, 1, 4]]) < tol


# ------------------------------------------------------------------------------------------ linears
def unzip(v):
    v = v.reshape(len(v), -1, 2, 8)
    return v[:, :, 0].reshape(len(v), -1), v[:, :, 1].reshape(len(v), -1)


@pytest.mark.parametrize("rows", [1, 5, 8, 33, 70, 257])
@pytest.mark.parametrize("n,split,k", [(64, None, 40), (160, None, 96), (167, 128, 328), (96, None, 2048), (261, 256, 1100)])
def test_linear_epilogues(cuda, rows, n, split, k):
    """Gated units and the softcap, with a bias, a factor on every row and outputs that leave in fp32 behind them; all three kernels."""
    from poptransformer_b200 import ops
    r = np.random.default_rng(2)
    L = ops._lib.lib()
    x, w, b = bf16(r.standard_normal((rows, k))), bf16(r.standard_normal((n, k)) * k ** -0.5), r.standard_normal(n).astype(np.float32)
    s = r.uniform(0.2, 3.0, rows).astype(np.float32)
    flag = torch.zeros(1, dtype=torch.int32, device=cuda)
    ws = dict(linear_ws=torch.zeros(L.pt_linear_workspace_bytes(min(rows, 32), n, 32), dtype=torch.uint8, device=cuda),
              gemm_ws=torch.zeros(L.pt_gemm_workspace_bytes(rows, n, 8), dtype=torch.uint8, device=cuda), error_flag=flag)
    cut = n if split is None else split
    cases = [("silu", ops.EPI_GLU, ops.GLU_SILU, cut // 2, lambda v: ref.gated_unit(ref.silu, *unzip(v))),
             ("gelu", ops.EPI_GLU, ops.GLU_GELU, cut // 2, lambda v: ref.gated_unit(ref.gelu_tanh, *unzip(v))),
             ("softcap", ops.EPI_SOFTCAP, ops.GLU_CLAMPED, cut, lambda v: ref.cap(v, 1.3)), ("store", ops.EPI_STORE, ops.GLU_CLAMPED, cut, lambda v: v)]
    for dt in (F32, BF16):
        for name, epi, glu, feats, f in cases:
            for scaled in (False, True):
                lin = ops.DenseLinear(as_type(w, dt, cuda), dt, bias=as_type(b, F32, cuda), split=split, limit=1.3, glu=glu)
                factor = as_type(s, F32, cuda)
                if scaled:
                    plain_ext = lin._ext

                    def scaled_ext(*a):
                        e = plain_ext(*a)
                        e.row_scale = factor.data_ptr()
                        return e
                    lin._ext = scaled_ext
                sums = (s[:, None] if scaled else 1.0) * (x.astype(np.float64) @ w.T) + b
                xp = torch.zeros((rows, lin.ld), dtype=dt, device=cuda)
                xp[:, :k] = as_type(x, dt, cuda)
                out2 = torch.full((rows, n - cut + 3), -7.0, device=cuda)
                for odt in {dt, F32}:
                    out = torch.full((rows, feats + 5), -7.0, dtype=odt, device=cuda)
                    lin(xp, out, rows, feats + 5, epilogue=epi, out2=out2, out2_ld=n - cut + 3, **ws)
                    assert rel(out[:, :feats].float().cpu(), f(sums[:, :cut])) < (5e-6 if odt == F32 else 6e-3), (dt, odt, name, scaled)
                    assert (out[:, feats:] == -7).all()
                    if split is not None:
                        assert rel(out2[:, :n - cut].cpu(), sums[:, cut:]) < 5e-6 and (out2[:, n - cut:] == -7).all(), (dt, name)
    other = as_type(-b, F32, cuda)         # a bias in place of the linear's own
    out = torch.empty((rows, n), device=cuda)
    lin = ops.DenseLinear(as_type(w, BF16, cuda), BF16)
    xp = torch.zeros((rows, lin.ld), dtype=BF16, device=cuda)
    xp[:, :k] = as_type(x, BF16, cuda)
    lin(xp, out, rows, n, bias=other, **ws)
    assert rel(out.cpu(), x.astype(np.float64) @ w.T - b) < 5e-6 and int(flag.item()) == 0


@pytest.mark.parametrize("n,k", [(48, 40), (272, 96), (128, 1344)])
@pytest.mark.parametrize("tile", [1, 16, 32, 64, 128])
def test_grouped_linear_with_weighed_inputs(cuda, tile, n, k):
    from poptransformer_b200 import ops
    r = np.random.default_rng(3)
    G, L = 5, ops._lib.lib()
    w = [bf16(r.standard_normal((n, k)) * k ** -0.5) for _ in range(G)]
    group_of = np.array([3, 0, 4, 3, 1, 3, 2] if tile == 1 else [3, 0, -1, 3, 1, -1, 2, -1])
    rows = len(group_of) * tile
    s = r.uniform(0.1, 2.0, rows).astype(np.float32)
    for dt in (F32, BF16):
        if dt == F32 and tile != 64:
            continue
        lin = ops.GroupedLinear([as_type(m, dt, cuda) for m in w], dt, glu=ops.GLU_SILU)
        for x_div in (1, 3) if tile == 1 else (1,):
            x = bf16(r.standard_normal((-(-rows // x_div), k)))
            xp = torch.zeros((len(x), lin.ld), dtype=dt, device=cuda)
            xp[:, :k] = as_type(x, dt, cuda)
            flag = torch.zeros(1, dtype=torch.int32, device=cuda)
            ws = dict(linear_ws=torch.zeros(L.pt_linear_workspace_bytes(rows, n, 4), dtype=torch.uint8, device=cuda),
                      gemm_ws=torch.zeros(L.pt_gemm_workspace_bytes(rows, n, 8), dtype=torch.uint8, device=cuda), error_flag=flag)
            for odt in {dt, F32}:
                out = torch.full((rows, n // 2 + 1), -7.0, dtype=odt, device=cuda)
                lin(xp, out, rows, n // 2 + 1, tile, i32(group_of, cuda), x_div=x_div, epilogue=ops.EPI_GLU, row_scale=as_type(s, F32, cuda), **ws)
                got = out.float().cpu().numpy()
                for t, g in enumerate(group_of):
                    at = np.arange(t * tile, (t + 1) * tile)
                    if g < 0:
                        assert (got[at] == -7).all()
                        continue
                    v = (s[at, None] * x[at // x_div].astype(np.float64)) @ w[g].T
                    assert rel(got[at, :n // 2], ref.gated_unit(ref.silu, *unzip(v))) < (5e-6 if odt == F32 else 6e-3) and (got[at, n // 2:] == -7).all()
            assert int(flag.item()) == 0


@pytest.mark.parametrize("tokens,experts,top,tile", [(1, 5, 5, 0), (3, 33, 4, 0), (9, 6, 2, 16), (300, 12, 3, 64), (1500, 7, 1, 128), (1901, 11, 5, 64)])
def test_router_with_sigmoid_scores(cuda, tokens, experts, top, tile):
    from poptransformer_b200 import ops
    r = np.random.default_rng(4)
    z = r.permuted(np.tile((np.arange(experts) - experts / 2) * 0.37, (tokens, 1)), axis=1).astype(np.float32)
    idx, score = ref.choose(z.astype(np.float64), top)
    expert, pair_row = (torch.full((tokens, top), -5, dtype=torch.int32, device=cuda) for _ in range(2))
    weight = torch.full((tokens, top), float("nan"), device=cuda)
    kw, row_weight = {}, None
    if tile:
        rows = tile * ops.moe_max_tiles(tokens, experts, top, tile)
        buf = lambda: torch.full((rows,), -5, dtype=torch.int32, device=cuda)
        row_weight, row_token = torch.full((rows,), -1.0, device=cuda), buf()
        kw = dict(tile=tile, pair_row=pair_row, tile_expert=buf(), tile_rows=buf(), row_token=row_token, counts=buf(), row_weight=row_weight)
    ops.moe_route(as_type(z, F32, cuda), tokens, experts, top, expert, weight, score=ops.MOE_SIGMOID, **kw)
    assert np.array_equal(expert.cpu().numpy(), idx) and rel(weight.cpu(), score) < 1e-6
    if tile:      # every placed row has its pair's weight, the padding none
        got = np.full(len(row_weight), -1.0)
        got[pair_row.cpu().numpy()] = weight.cpu().numpy()
        assert np.array_equal(row_weight.cpu().numpy(), got.astype(np.float32)) and ((row_token.cpu().numpy() < 0) == (got < 0)).all()


# ------------------------------------------------------------------------------------------ windowed attention
KINDS = [(F32, True), (BF16, True), (BF16, False)]


def gate_rows(g, dt, dev):
    """A gate tensor with some columns in front, and how window_attn is told about it."""
    buf = torch.zeros((len(g), g.shape[1] + 8), dtype=dt, device=dev)
    buf[:, 8:] = as_type(g, dt, dev)
    return dict(gate=buf.view(-1)[8:], gate_ld=buf.shape[1])


@pytest.mark.parametrize("dtype,plain", KINDS)
@pytest.mark.parametrize("H,G,D,V,window,cap,per_head", [(4, 2, 32, 64, 70, 2.0, False), (3, 1, 128, 96, 128, 5.0, False), (2, 2, 40, 24, 1, 1.0, True), (12, 1, 64, 32, 65, 0.0, False),
                                                         (5, 5, 14, 9, 33, 3.0, False), (6, 2, 96, 128, 0, 8.0, True), (4, 4, 64, 64, 300, 50.0, False),
                                                         (2, 1, 160, 136, 100, 4.0, False)])
def test_attention_with_softcap_and_gate(cuda, dtype, plain, H, G, D, V, window, cap, per_head):
    """Three sequences of unequal length in portions (down to two tokens) and single tokens."""
    r = np.random.default_rng(5)
    lens, scale = [215, 70, 134], 3.0 * D ** -0.5
    q, k, v, g = ([bf16(r.standard_normal((n, *shape))) for n in lens] for shape in ((H, D), (G, D), (G, V), (H if per_head else H * V,)))
    att = PagedAttention(cuda, dtype, 3, G, D, V, 256)
    got, at, slots = [[] for _ in lens], [0, 0, 0], [2, 0, 1]
    for take in ([1, 2, 1], [63, 1, 64], [3, 2, 1], [100, 33, 60], [2, 2, 2], [1, 1, 1], [1, 1, 1], [10, 24, 1], [1, 1, 1], [33, 3, 2]):
        cut = lambda t: np.concatenate([t[i][at[i]:at[i] + n] for i, n in enumerate(take)])
        o = att(cut(q), cut(k), cut(v), take, at, slots, scale, window, 0, None, plain, softcap=cap, gate_per_head=per_head, pad_cols=16, **gate_rows(cut(g), dtype, cuda))
        for i, part in enumerate(np.split(o, np.cumsum(take)[:-1])):
            got[i].append(part)
            at[i] += take[i]
    assert at == lens
    for i, n in enumerate(lens):
        f = lambda t: t[i].astype(np.float64)
        gate = ref.sigmoid(f(g))
        want = (ref.masked_attention(f(q), f(k), f(v), scale, window, cap) * (gate[:, :, None] if per_head else gate.reshape(n, H, V))).reshape(n, -1)
        err = np.abs(np.concatenate(got[i]) - want).max(1)
        assert err.max() < (2e-5 if dtype == F32 else 4e-2), (i, int(err.argmax()), float(err.max()))
        assert rel(np.concatenate(got[i]), want) < (2e-6 if dtype == F32 else 8e-3)


@pytest.mark.parametrize("dtype,plain", KINDS)
@pytest.mark.parametrize("window", [1, 2, 63, 64, 65, 100, 128])
def test_one_key_in_and_out_of_the_window(cuda, dtype, plain, window):
    """One key stands out for every query and carries a value of its own: just the queries from it to window - 1 tokens on may see it, in
    prompts, portions and decoding, at page borders too.  The softcap leaves it on top."""
    n, H, G, D = 260, 2, 1, 32
    special = [0, 1, 62, 63, 64, 65, 127, 128, 129, 198]
    r = np.random.default_rng(6)
    B = len(special)
    q, k, v = bf16(0.02 * r.standard_normal((B, n, H, D))), bf16(0.3 * r.standard_normal((B, n, G, D))), bf16(0.1 * r.standard_normal((B, n, G, D)))
    q[..., 31] = 1.0
    for b, j in enumerate(special):
        k[b, j, :, 31] = 40.0
        v[b, j] = 5.0
    want = np.stack([ref.masked_attention(*(t[b].astype(np.float64) for t in (q, k, v)), 1.0, window, 12.0).reshape(n, -1) for b in range(B)])
    at = np.array(special)[:, None]
    seen = (np.arange(n) >= at) & (np.arange(n) < at + window)
    assert ((want.min(2) > 3) == seen).all()
    att = PagedAttention(cuda, dtype, B, G, D, D, 320)
    flat = lambda t, a, b: t[:, a:b].reshape(B * (b - a), *t.shape[2:])
    got, a = [], 0
    for m in [100, 2, 58] + [1] * 100:
        got.append(att(flat(q, a, a + m), flat(k, a, a + m), flat(v, a, a + m), [m] * B, [a] * B, range(B), 1.0, window, 0, None, plain, softcap=12.0).reshape(B, m, -1))
        a += m
    got = np.concatenate(got, 1)
    wrong = np.argwhere((got.min(2) > 3) != seen)
    assert not len(wrong), [(special[b], int(i)) for b, i in wrong[:5]]
    assert np.abs(got - want).max() < (1e-4 if dtype == F32 else 5e-2)


# ------------------------------------------------------------------------------------------ latent attention
LATENTS = [  # heads, plain key width, rotated width, value width, rank, query rank
    (4, 24, 16, 32, 48, 40), (20, 128, 64, 128, 512, 96), (3, 16, 8, 8, 136, 72), (33, 64, 32, 64, 256, 300), (16, 32, 64, 40, 320, 16), (3, 13, 6, 11, 21, 17), (2, 200, 48, 120, 72, 8),
    (1, 8, 200, 16, 16, 24), (40, 16, 8, 24, 64, 64), (2, 24, 16, 32, 520, 24), (3, 40, 32, 136, 64, 48), (17, 264, 16, 16, 96, 32)]


@pytest.mark.parametrize("dtype,plain", KINDS)
@pytest.mark.parametrize("shape", LATENTS)
def test_latent_attention(cuda, dtype, plain, shape):
    """Three sequences of unequal length in portions (down to two tokens) and single tokens."""
    site = LatentSite(cuda, dtype, 3, *shape, 256)
    lens = [215, 70, 134]
    x, q = zip(*(site.inputs(n, 8 + i) for i, n in enumerate(lens)))
    takes = ([1, 2, 1], [63, 1, 64], [3, 2, 1], [100, 33, 60], [2, 2, 2], [1, 1, 1], [1, 1, 1], [10, 24, 1], [1, 1, 1], [33, 3, 2])
    for i, got in enumerate(site.run(x, q, takes, [2, 0, 1], plain)):
        want = site.oracle(x[i], q[i])
        err = np.abs(got - want).max(1)
        assert err.max() < (5e-5 if dtype == F32 else 6e-2), (i, int(err.argmax()), float(err.max()))
        assert rel(got, want) < (3e-6 if dtype == F32 else 1.2e-2)


@pytest.mark.parametrize("dtype,plain", KINDS)
def test_one_far_latent(cuda, dtype, plain):
    """One position's latent points where every query looks, and carries a value of its own: every query from it on must find it, and
    none before, across pages, portions and decoding."""
    n, H, D, R, V, rank = 230, 3, 8, 8, 16, 64
    special = [0, 1, 62, 63, 64, 65, 127, 128, 129, 198]
    B = len(special)
    site = LatentSite(cuda, dtype, B, H, D, R, V, rank, 16, 256, scale=1.0)
    site.kn[:] = 1.0
    site.uk[:] = 0.0
    site.uk[:, 0, 0], site.uv[:] = 1.0, 0.0
    site.uv[:, :, 0] = 1.0
    site.w.kv_norm.fill_(1.0)
    site.w.w_k, site.w.w_v = as_type(site.uk.transpose(0, 2, 1), site.dt, cuda), as_type(site.uv, site.dt, cuda)
    site.up = site.ops.DenseLinear(as_type(np.concatenate([site.uk.reshape(-1, rank), site.uv.reshape(-1, rank)]), site.dt, cuda), site.dt)
    xs, qs = [], []
    for b, j in enumerate(special):
        x, q = site.inputs(n, 40 + b)
        x[:, 16], x[:, -H:] = 0.0, 8.0                       # (the first latent dimension; open gates)
        x[j, 16:16 + rank] = 0.0
        x[j, 16] = 9.0
        x[:, 16 + rank:16 + rank + R] *= 0.1
        q[..., 0] = 2.0
        xs.append(x), qs.append(q)
    want = [site.oracle(x, q) for x, q in zip(xs, qs)]
    seen = np.arange(n)[None] >= np.array(special)[:, None]
    assert all(((w.min(1) > 5) == s).all() for w, s in zip(want, seen))
    got = site.run(xs, qs, [[100] * B, [2] * B, [57] * B] + [[1] * B] * 71, list(range(B)), plain)
    wrong = np.argwhere((np.stack([g.min(1) for g in got]) > 5) != seen)
    assert not len(wrong), [(special[b], int(i)) for b, i in wrong[:5]]
    assert max(np.abs(g - w).max() for g, w in zip(got, want)) < (1e-4 if dtype == F32 else 8e-2)


@pytest.mark.parametrize("plain", [True, False])
def test_many_decoding_rows(cuda, plain):
    """More sequences than SMs (no runs of pages), more than the 16 tokens of a tile, and positions from 0 to several pages."""
    site = LatentSite(cuda, BF16, 170, 18, 32, 16, 32, 128, 32, 330)
    r = np.random.default_rng(9)
    for B in (170, 35, 3):
        lens = [int(v) for v in r.integers(1, 300, B)]
        lens[:3] = [1, 64, 65]
        x, q = zip(*(site.inputs(n, 60 + i) for i, n in enumerate(lens)))
        site.cache.pool.fill_(float("nan"))
        if max(lens) > 1:
            head = [i for i, n in enumerate(lens) if n > 1]
            site(np.concatenate([x[i][:-1] for i in head]), np.concatenate([q[i][:-1] for i in head]), [lens[i] - 1 for i in head], [0] * len(head), head, plain, check_cq=False)
        got = site(np.stack([t[-1] for t in x]), np.stack([t[-1] for t in q]), [1] * B, [n - 1 for n in lens], range(B), plain)
        for i in list(range(0, B, 9)) + [0, 1, 2]:
            assert rel(got[i], site.oracle(x[i], q[i])[-1]) < 2e-2, (B, i, lens[i])


# ------------------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_model_prompts_portions_and_decoding(cuda, name, dtype):
    cfg = CONFIGS[name]
    w = weights(cfg, seed=11)
    n = 150
    tokens = prompt(n, cfg["vocab"])
    sums = []
    want = ref.PivavikOracle(cfg, w).forward(tokens, sums)
    dec = decoder(cfg, w, 3, 192, dtype)
    dec.rows_prompt = dec._row_buffers(n)
    for r in (dec.rows_prompt, dec.rows_decode):     # nothing may depend on what the buffers held (padding rows of the experts' tiles, padded columns)
        for t in vars(r).values():
            if torch.is_tensor(t) and t.is_floating_point():
                t.fill_(float("nan"))
    for plain in (False, True):
        dec.plain = plain
        if plain:
            dec.rows_prompt = None
        got_sums, s = [], dec.open()
        whole = dec.extend([(s, tokens, list(range(n)))], layer_sums=got_sums).cpu().numpy()
        dec.close(s)
        assert len(got_sums) == len(sums)
        for i, (a, b) in enumerate(zip(got_sums, sums)):
            assert rel(a.cpu(), b) < TOL[dtype], f"after run {i}"
        assert rel(whole, want) < TOL[dtype]
        for cuts in ([1] * n, [2] * (n // 2), [64, 64, 22], [63, 2, 65, 20], [100] + [1] * 50):
            got = run_cut(dec, tokens, cuts)
            per = np.sqrt(((got - whole) ** 2).mean(1)) / np.sqrt((whole ** 2).mean())
            assert per.max() < (1e-4 if dtype == "float32" else 6e-2), (cuts[:4], int(per.argmax()), float(per.max()))
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


def test_mixed_batches(cuda):
    """First tokens, portions and single tokens of different sequences in one batch."""
    cfg = CONFIGS["wide-heads"]
    w = weights(cfg, seed=23)
    toks = [prompt(90, cfg["vocab"], i) for i in range(3)]
    orc = [ref.PivavikOracle(cfg, w).forward(t) for t in toks]
    for dtype in ("float32", "bfloat16"):
        dec = decoder(cfg, w, 3, 128, dtype)
        seqs, at, got = [dec.open() for _ in toks], [0, 0, 0], [[], [], []]
        for take in ([66, 0, 1], [1, 30, 2], [0, 1, 1], [1, 1, 60], [1, 1, 1], [20, 1, 0], [1, 56, 25]):
            o = dec.extend([(s, t[a:a + n], list(range(n))) for s, t, a, n in zip(seqs, toks, at, take) if n]).cpu().numpy()
            for i, n in enumerate(take):
                got[i].append(o[sum(take[:i]):sum(take[:i]) + n])
                at[i] += n
        assert at == [90, 90, 90]
        for g, want in zip(got, orc):
            assert rel(np.concatenate(g), want) < TOL[dtype]


def test_more_rows_than_the_skinny_kernels_take(cuda):
    cfg = CONFIGS["wide-heads"]
    w = weights(cfg, seed=13)
    B = 45
    toks = [prompt(20, cfg["vocab"], i) for i in range(B)]
    picked = (0, 17, 31, 32, 44)
    want = np.stack([ref.PivavikOracle(cfg, w).forward(toks[b])[18:] for b in picked])
    for dtype in ("float32", "bfloat16"):
        dec = decoder(cfg, w, B, 64, dtype)
        seqs = [dec.open() for _ in range(B)]
        dec.extend([(s, t[:18], []) for s, t in zip(seqs, toks)])
        got = np.stack([dec.extend([(s, t[i:i + 1], [0]) for s, t in zip(seqs, toks)]).cpu().numpy() for i in (18, 19)], 1)
        assert rel(got[list(picked)], want) < 1.5 * TOL[dtype]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_slots_and_pages_are_used_again(cuda, dtype):
    """A pool that only fits one batch at a time; before every batch all caches are poisoned."""
    cfg = CONFIGS["mixed"]
    w = weights(cfg, seed=14)
    fresh = decoder(cfg, w, 1, 192, dtype)
    dec = decoder(cfg, w, 3, 192, dtype, n_pages=5)
    assert len(dec.caches) == len(dec.runs) == 9           # every pass of the loop has caches of its own
    for rnd, lens in enumerate([[120, 60], [10, 64, 65], [190], [3, 130], [1, 1, 1]]):
        for c in dec.caches.values():
            c.pool.fill_(float("nan"))
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
    want = ref.PivavikOracle(cfg, w).forward(tokens)
    assert rel(got, want) < TOL[dtype]
    assert rel(got[-20:], want[-20:]) < TOL[dtype]


def test_first_tokens(cuda):
    """Prompts of 1 .. 9 tokens."""
    cfg = config([latent(mlp=dense()), attention(window=4, mlp=moe())], width=64, loop=(0, 1, 2))
    w = weights(cfg, seed=16)
    orc = ref.PivavikOracle(cfg, w)
    for dtype in ("float32", "bfloat16"):
        dec = decoder(cfg, w, 9, 64, dtype)
        toks = [prompt(n, cfg["vocab"], n) for n in range(1, 10)]
        seqs = [dec.open() for _ in toks]
        got = dec.extend([(s, t, list(range(len(t)))) for s, t in zip(seqs, toks)]).cpu().numpy()
        assert rel(got, np.concatenate([orc.forward(t) for t in toks])) < TOL[dtype]


def test_pages_of_another_size(cuda):
    cfg = CONFIGS["mixed"]
    w = weights(cfg, seed=24)
    tokens = prompt(70, cfg["vocab"])
    want = ref.PivavikOracle(cfg, w).forward(tokens)
    for dtype in ("float32", "bfloat16"):
        assert rel(run_cut(decoder(cfg, w, 1, 96, dtype, page_size=24), tokens, [50] + [1] * 10 + [10]), want) < TOL[dtype]


def test_missing_parts_would_show(cuda):
    """The comparison above is sharp: an oracle with one part changed is far from the kernels."""
    cfg = CONFIGS["mixed"]
    w = weights(cfg, seed=22)
    tokens = prompt(140, cfg["vocab"])
    dec = decoder(cfg, w, 1, 192, "bfloat16")
    s = dec.open()
    got = dec.extend([(s, tokens, list(range(140)))]).cpu().numpy()
    right = rel(got, ref.PivavikOracle(cfg, w).forward(tokens))
    assert right < TOL["bfloat16"]

    def changed(edit_cfg=None, edit_w=None):
        c, v = json.loads(json.dumps(cfg)), dict(w)
        for f, x in ((edit_cfg, c), (edit_w, v)):
            if f:
                f(x)
        return rel(got, ref.PivavikOracle(c, v).forward(tokens))

    mix = lambda c, i: c["layers"][i]["mixer"]
    zero = lambda k: dict(edit_w=lambda v: v.update({k: 0 * v[k]}))
    edits = [dict(edit_cfg=lambda c: mix(c, 0)["rot"].update(base=2e3)), dict(edit_cfg=lambda c: mix(c, 1).update(softcap=1.0)), dict(edit_cfg=lambda c: mix(c, 3).update(softcap=0.0)),
             dict(edit_cfg=lambda c: mix(c, 1)["mask"].update(size=38)), dict(edit_cfg=lambda c: mix(c, 2).update(scale=1.2 * mix(c, 2)["scale"])),
             dict(edit_cfg=lambda c: c.update(logit_softcap=5.0)), dict(edit_cfg=lambda c: c["loop"].update(times=2)), dict(edit_cfg=lambda c: c["layers"][1]["mlp"]["router"].update(top=1)),
             zero("l0.mix.g"), zero("l1.mix.g"), zero("l1.mix.q.b"), zero("l1.mix.v.b"), zero("l0.mlp.up.b"), zero("l0.mlp.down.b"), zero("loop.step"), zero("embed.norm"), zero("final.norm"),
             zero("l4.norm1"), dict(edit_w=lambda v: v.update({"l2.mix.dkv.norm": 0 * v["l2.mix.dkv.norm"] + 1})), dict(edit_w=lambda v: v.update({"l0.mix.dq.norm": 0 * v["l0.mix.dq.norm"] + 1}))]
    far = [changed(**e) for e in edits]
    assert [(i, d, right) for i, d in enumerate(far) if d < max(TOL["bfloat16"], 2.5 * right)] == []


# ------------------------------------------------------------------------------------------ the decode loop
@pytest.mark.parametrize("dtype,tol", [("float32", 1e-4), ("bfloat16", 8e-2)])
def test_greedy_generation(cuda, dtype, tol):
    cfg = CONFIGS["mixed"]
    w = weights(cfg, seed=17)
    orc = ref.PivavikOracle(cfg, w)
    max_len, lens = 80, [3, 20, 9]
    dec = decoder(cfg, w, 3, max_len, dtype, pad_id=-1)
    ids = np.full((3, max_len), -1, np.int32)
    for b, n in enumerate(lens):
        ids[b, :n] = prompt(n, cfg["vocab"], b)
    eager = dec.run(ids, max_loop=max_len - 1)["Loop:0"]
    assert all((eager[b, :n] == ids[b, :n]).all() for b, n in enumerate(lens)) and (eager >= 0).all()
    assert greedy_ok(orc, eager, lens, tol) > 0.9
    dec.capture()
    assert np.array_equal(dec.run(ids, max_loop=max_len - 1)["Loop:0"], eager)          # one CUDA graph per step, caches of the run before left behind
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
    eos = int(next(t for t in want[0, 92:] if t not in ids))         # row 0 stops there; row 1 wherever it produces the same id, if it does
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
    orc = {k: ref.PivavikOracle(cfg, w).forward(t) for k, t in toks.items()}
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
    cfg = CONFIGS["plain-order"]
    w = weights(cfg, seed=21)
    write_model(str(tmp_path), cfg, w)
    a, b = prompt(6, cfg["vocab"], 1).tolist(), prompt(3, cfg["vocab"], 2).tolist()
    cmd = [sys.executable, "-m", "poptransformer_b200", "generate", "--model", str(tmp_path), "--prompt", ",".join(map(str, a)), "--prompt", ",".join(map(str, b)),
           "--new", "10", "--dtype", "float32", "--prefill"]
    p = subprocess.run(cmd, capture_output=True, text=True, timeout=300, cwd=ROOT)
    assert p.returncode == 0, p.stderr[-2000:]
    rows = [json.loads(ln)["ids"] for ln in p.stdout.splitlines()]
    assert [len(r) for r in rows] == [16, 16] and rows[0][:6] == a and rows[1][:3] == b
    assert greedy_ok(ref.PivavikOracle(cfg, w), np.array(rows), [6, 3], 1e-4) == 1.0
