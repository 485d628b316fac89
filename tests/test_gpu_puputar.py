"""Puputar on the GPU against the plain restatement (oracle/puputar_np.py): every mechanism alone, then whole models in prompts, portions,
batches and decoding, with slots and pages that are used again, and greedy generation through the decode loop."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from latent_util import LatentSite
from oracle import puputar_np as ref
from puputar_util import CONFIGS, config, decoder, dense, latent, latent2, moe, weights
from seq_util import as_type, bf16, greedy_ok, i32, prompt, rel, run_cut, tensors, view_of, write_model

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = {"float32": 2e-5, "bfloat16": 2.5e-2}       # rms of the difference over the rms of the logits, whole model
F32, BF16 = torch.float32, torch.bfloat16
back = lambda t: t.float().cpu().numpy()


# ------------------------------------------------------------------------------------------ residual stream
class ShiftSite:
    """The residual step in front of one layer, called on portions of several sequences as a decoder calls it."""

    def __init__(self, dev, dt, W, G, slots, seed=0):
        r = np.random.default_rng(seed)
        self.dev, self.dt, self.W, self.G, self.eps, self.ld = dev, dt, W, G, 1e-3, W + 5 if W % 4 else W + 8
        self.w1, self.w2, self.mix, self.we = (m + 0.3 * r.standard_normal(W) for m in (1, 1, 0.5, 1))
        self.state = torch.full((slots, W), float("nan"), device=dev)       # position 0 reads none of it

    def common(self, n):
        f = lambda a: as_type(a, F32, self.dev)
        nan = lambda w, dt: torch.full((n, w), float("nan"), dtype=dt, device=self.dev)
        return dict(w1=f(self.w1), shift=f(self.mix), w2=f(self.w2), h1=nan(self.ld, self.dt), h2=nan(self.ld, self.dt), h1_ld=self.ld, h2_ld=self.ld, x_out=nan(self.W, F32))

    def __call__(self, lens, starts, slots, **kw):
        from poptransformer_b200 import ops
        n, single = sum(lens), max(lens) == 1
        out = self.common(n)
        after = self.state if single else torch.full((len(lens), self.W), float("nan"), device=self.dev)
        ops.shift_norm(view_of(lens, starts, slots, self.dev), n, self.W, self.G, self.eps, self.dt, state_in=self.state, state_out=after, state_by_seq=not single, **out, **kw)
        if not single:
            self.state[list(slots)] = after
        assert not out["h1"][:, self.W:].any() and not out["h2"][:, self.W:].any()
        return [back(out[k][:, :self.W]) for k in ("x_out", "h1", "h2")]

    def want(self, x):
        """x: the stream of one sequence from its first token on."""
        a = ref.group_norm(x, self.w1, self.eps, self.G)
        return x, ref.token_shift(a, self.mix), ref.group_norm(x, self.w2, self.eps, self.G)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("W,G", [(33, 3), (96, 4), (96, 1), (50, 50), (2048, 8), (260, 13), (128, 1), (384, 3), (768, 3), (4096, 1), (4224, 33)])
def test_residual_step_with_token_shift(cuda, dtype, W, G):
    """Three sequences in portions (down to two tokens) and single tokens: dense outputs, experts' outputs with weights, and experts that
    give the feed-forward's input back."""
    r = np.random.default_rng(1)
    tol, lens, top = 1e-6 if dtype == F32 else 4e-3, [215, 70, 134], 3
    X, Y, S = ([r.standard_normal((n, W)).astype(np.float32) for n in lens] for _ in range(3))
    S = [bf16(s) for s in S]
    PW, PY = [r.uniform(0.1, 1, (n, top)).astype(np.float32) for n in lens], [bf16(r.standard_normal((n, top, W))) for n in lens]
    own = [r.integers(0, 3, (n, top)) == 0 for n in lens]                         # pairs that chose an identity expert
    site, at, slots, got = ShiftSite(cuda, dtype, W, G, 4), [0, 0, 0], [3, 0, 1], [[], [], []]
    takes = ([1, 2, 1], [63, 1, 64], [3, 2, 1], [100, 33, 60], [2, 2, 2], [1, 1, 1], [1, 1, 1], [10, 24, 1], [1, 1, 1], [33, 3, 2])
    for k, take in enumerate(takes):
        cut = lambda t: np.concatenate([t[i][at[i]:at[i] + n] for i, n in enumerate(take)])
        n = sum(take)
        pw, py, self_, mine = cut(PW), cut(PY), cut(S), cut(own)
        rows = r.permutation(n * top + 7)[:n * top].reshape(n, top)               # where the router put the pairs' rows
        where = np.where(mine, -1, rows)
        edt = dtype if k % 2 else F32
        pair_y, self_t = torch.full((n * top + 7, W), float("nan"), dtype=edt, device=cuda), torch.full((n, site.ld), float("nan"), dtype=dtype, device=cuda)
        pair_y[i32(rows, cuda).long().view(-1)] = as_type(py.reshape(-1, W), edt, cuda)
        pair_y[i32(rows[mine], cuda).long()] = float("nan")                       # no row of theirs may be read
        self_t[:, :W] = as_type(self_, dtype, cuda)
        o = site(take, at, slots, x_in=as_type(cut(X), F32, cuda), y=as_type(cut(Y), F32, cuda), y_ld=W, pair_y=pair_y, pair_ld=W, top=top, pair_w=as_type(pw, F32, cuda),
                 pair_row=i32(where, cuda), self_rows=self_t, self_ld=site.ld)
        for i, part in enumerate(zip(*(np.split(a, np.cumsum(take)[:-1]) for a in o))):
            got[i].append(part)
            at[i] += take[i]
    assert at == lens
    for i in range(3):
        f = lambda t: t[i].astype(np.float64)
        x = f(X) + f(Y) + np.einsum("tk,tkw->tw", f(PW), np.where(own[i][:, :, None], f(S)[:, None], f(PY)))
        for g, want, t in zip((np.concatenate(p) for p in zip(*got[i])), site.want(x), (1e-6, tol, tol)):
            per = np.sqrt(((g - want) ** 2).mean(1)) / np.sqrt((want ** 2).mean())
            assert per.max() < 3 * t, (i, int(per.argmax()), float(per.max()))
    assert site.state[2].isnan().all()                                            # a slot that no sequence had


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("W,G", [(64, 2), (256, 2)])
@pytest.mark.parametrize("rows", [3, 700, 1300])
def test_residual_step_over_many_rows(cuda, dtype, rows, W, G):
    """Runs of one row per block and more, with sequences that begin and end anywhere in them, and an embedding start."""
    r = np.random.default_rng(2)
    vocab = 31
    lens = []
    while sum(lens) < rows:
        lens.append(int(min(r.integers(1, 12), rows - sum(lens))))
    site, n = ShiftSite(cuda, dtype, W, G, len(lens)), sum(lens)
    table, ids = bf16(r.standard_normal((vocab, W))), r.integers(0, vocab, n)
    x, y = r.standard_normal((n, W)).astype(np.float32), r.standard_normal((n, W)).astype(np.float32)
    before = r.standard_normal((len(lens), W)).astype(np.float32)
    for start, mode in ((0, "table"), (0, "stream"), (9, "table"), (9, "stream")):
        site.state.copy_(as_type(before, F32, cuda))
        if mode == "table":
            got = site(lens, [start] * len(lens), range(len(lens)), table=as_type(table, dtype, cuda), ids=i32(ids, cuda), embed_w=as_type(site.we, F32, cuda))
            xs = ref.group_norm(table[ids].astype(np.float64), site.we, site.eps, G)
        else:
            got = site(lens, [start] * len(lens), range(len(lens)), x_in=as_type(x, F32, cuda), y=as_type(y, F32, cuda), y_ld=W)
            xs = x.astype(np.float64) + y
        a = ref.group_norm(xs, site.w1, site.eps, G)
        first = np.cumsum([0] + lens[:-1])
        above = np.concatenate([a[:1], a[:-1]])
        above[first] = before if start else 0.0
        for g, w, t in zip(got, (xs, a + (above - a) * site.mix, ref.group_norm(xs, site.w2, site.eps, G)), (1e-6, *[1e-6 if dtype == F32 else 4e-3] * 2)):
            assert rel(g, w) < t, (start, mode)
        assert rel(site.state.cpu(), a[first + np.array(lens) - 1]) < 1e-6


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("W,G", [(96, 4), (512, 2)])
def test_residual_step_of_the_decode_loop_and_the_end(cuda, dtype, W, G):
    """One token per row from an id container at a position that is read on the device; and the norm in front of the output layer."""
    from poptransformer_b200 import ops
    r = np.random.default_rng(3)
    B, vocab = 5, 17
    site, tol = ShiftSite(cuda, dtype, W, G, B), 1e-6 if dtype == F32 else 4e-3
    table, ids = bf16(r.standard_normal((vocab, W))), r.integers(0, vocab, (B, 4))
    pos, step, rows = torch.full((B,), 77, dtype=torch.int32, device=cuda), i32([0], cuda), i32(np.arange(B + 1), cuda)
    view = ops.batch_view(B, B, rows, pos, rows, rows)
    xs = ref.group_norm(table[ids].astype(np.float64).reshape(-1, W), site.we, site.eps, G).reshape(B, 4, W)
    for t in range(4):
        step.fill_(t)
        out = site.common(B)
        ops.shift_norm(view, B, W, G, site.eps, dtype, state_in=site.state, state_out=site.state, table=as_type(table, dtype, cuda), ids=i32(ids, cuda), ids_ld=4, step=step, pos_out=pos,
                       embed_w=as_type(site.we, F32, cuda), **out)
        want = np.stack([[w[t] for w in site.want(x)] for x in xs], 1)
        assert rel(back(out["x_out"]), want[0]) < 1e-6 and rel(back(out["h1"][:, :W]), want[1]) < tol and rel(back(out["h2"][:, :W]), want[2]) < tol and (pos == t).all()
    (x, y), pick = (r.standard_normal((B, W)).astype(np.float32) for _ in range(2)), [3, 0, 3]
    h = torch.full((3, site.ld), float("nan"), dtype=dtype, device=cuda)
    ops.shift_norm(None, 3, W, G, site.eps, dtype, x_in=as_type(x, F32, cuda), y=as_type(y, F32, cuda), y_ld=W, w2=as_type(site.w2, F32, cuda), h2=h, h2_ld=site.ld, row_index=i32(pick, cuda))
    assert rel(back(h[:, :W]), ref.group_norm((x.astype(np.float64) + y)[pick], site.w2, site.eps, G)) < tol and not h[:, W:].any()


def test_residual_step_refuses(cuda):
    from poptransformer_b200 import PtError, ops
    site = ShiftSite(cuda, F32, 32, 2, 2)
    x, view = torch.zeros((3, 32), device=cuda), view_of([2, 1], [0, 0], [0, 1], cuda)
    kw = {**site.common(3), "x_out": x}
    with pytest.raises(PtError, match="other buffers"):
        ops.shift_norm(view, 3, 32, 2, 1e-3, F32, x_in=x, state_in=site.state, state_out=torch.empty_like(site.state), **kw)
    with pytest.raises(PtError, match="other buffers"):
        ops.shift_norm(view, 3, 32, 2, 1e-3, F32, x_in=torch.zeros_like(x), state_in=site.state, state_out=site.state, **kw)
    with pytest.raises(PtError, match="groups"):
        ops.shift_norm(None, 3, 32, 3, 1e-3, F32, x_in=x, x_out=x)


# ------------------------------------------------------------------------------------------ linears
@pytest.mark.parametrize("rows", [1, 5, 8, 33, 70, 257])
@pytest.mark.parametrize("n,split,k", [(64, None, 40), (167, 128, 328), (96, None, 2048), (261, 256, 1100)])
def test_xielu_epilogue(cuda, rows, n, split, k):
    """All three kernels, with k-slices and without, outputs behind the split without the unit, sums from far below to far above zero."""
    from poptransformer_b200 import ops
    r = np.random.default_rng(4)
    L = ops._lib.lib()
    x, w, b = bf16(r.standard_normal((rows, k))), bf16(r.standard_normal((n, k)) * k ** -0.5 * r.choice([0.03, 1, 6], (n, 1))), 0.2 * r.standard_normal(n).astype(np.float32)
    b[:4] = [120, -120, 0, 1e-3]                                   # exp(120) overflows, and must not show
    flag = torch.zeros(1, dtype=torch.int32, device=cuda)
    ws = dict(linear_ws=torch.zeros(L.pt_linear_workspace_bytes(min(rows, 32), n, 32), dtype=torch.uint8, device=cuda),
              gemm_ws=torch.zeros(L.pt_gemm_workspace_bytes(rows, n, 8), dtype=torch.uint8, device=cuda), error_flag=flag)
    cut, p, q = n if split is None else split, 0.4, -1.3
    sums = x.astype(np.float64) @ w.T + b
    want = ref.xielu(sums[:, :cut], p, q)
    for dt in (F32, BF16):
        lin = ops.DenseLinear(as_type(w, dt, cuda), dt, bias=as_type(b, F32, cuda), split=split, xielu=(float(ref.softplus(p)), float(0.5 + ref.softplus(q))))
        xp = torch.zeros((rows, lin.ld), dtype=dt, device=cuda)
        xp[:, :k] = as_type(x, dt, cuda)
        out2 = torch.full((rows, n - cut + 3), -7.0, device=cuda)
        for odt in {dt, F32}:
            out = torch.full((rows, cut + 5), -7.0, dtype=odt, device=cuda)
            lin(xp, out, rows, cut + 5, epilogue=ops.EPI_XIELU, out2=out2, out2_ld=n - cut + 3, **ws)
            got = back(out[:, :cut])
            small = np.abs(want) < 50
            assert rel(got[small], want[small]) < (5e-6 if odt == F32 else 6e-3) and np.allclose(got[~small], want[~small], rtol=1e-5 if odt == F32 else 1e-2), (dt, odt)
            assert (out[:, cut:] == -7).all()
            if split is not None:
                assert rel(out2[:, :n - cut].cpu(), sums[:, cut:]) < 5e-6 and (out2[:, n - cut:] == -7).all(), dt
    assert int(flag.item()) == 0


@pytest.mark.parametrize("n,k", [(48, 40), (272, 96), (128, 1344)])
@pytest.mark.parametrize("tile", [1, 16, 64, 128])
def test_grouped_linear_with_rows_of_no_expert(cuda, tile, n, k):
    """relu^2 experts; tiles that belong to none leave their output as it is."""
    from poptransformer_b200 import ops
    r = np.random.default_rng(5)
    G, L = 5, ops._lib.lib()
    w = [bf16(r.standard_normal((n, k)) * k ** -0.5) for _ in range(G)]
    group_of = np.array([3, 0, -1, 3, 1, -1, 2, -1])
    rows = len(group_of) * tile
    for dt in (F32, BF16):
        if dt == F32 and tile != 64:
            continue
        lin = ops.GroupedLinear([as_type(m, dt, cuda) for m in w], dt)
        for x_div in (1, 2) if tile == 1 else (1,):
            x = bf16(r.standard_normal((-(-rows // x_div), k)))
            xp = torch.zeros((len(x), lin.ld), dtype=dt, device=cuda)
            xp[:, :k] = as_type(x, dt, cuda)
            flag = torch.zeros(1, dtype=torch.int32, device=cuda)
            ws = dict(linear_ws=torch.zeros(L.pt_linear_workspace_bytes(rows, n, 4), dtype=torch.uint8, device=cuda),
                      gemm_ws=torch.zeros(L.pt_gemm_workspace_bytes(rows, n, 8), dtype=torch.uint8, device=cuda), error_flag=flag)
            for odt in {dt, F32}:
                for _ in range(2):                                 # the arrival counters of k-slices are left at zero
                    out = torch.full((rows, n + 1), -7.0, dtype=odt, device=cuda)
                    lin(xp, out, rows, n + 1, tile, i32(group_of, cuda), x_div=x_div, epilogue=ops.EPI_RELU2, **ws)
                    got = back(out)
                    for t, g in enumerate(group_of):
                        at = np.arange(t * tile, (t + 1) * tile)
                        if g < 0:
                            assert (got[at] == -7).all()
                        else:
                            assert rel(got[at, :n], ref.relu2(x[at // x_div].astype(np.float64) @ w[g].T)) < (5e-6 if odt == F32 else 6e-3) and (got[at, n:] == -7).all()
            assert int(flag.item()) == 0


# ------------------------------------------------------------------------------------------ router
@pytest.mark.parametrize("tokens,experts,identity,count,keep,top,tile", [
    (1, 5, 0, 1, 1, 5, 0), (3, 33, 3, 4, 2, 4, 0), (7, 6, 2, 4, 3, 2, 0), (9, 6, 2, 2, 1, 2, 16), (300, 12, 4, 8, 4, 3, 64), (1500, 7, 1, 4, 4, 1, 128), (1901, 11, 5, 4, 2, 5, 64),
    (40, 1, 3, 1, 1, 2, 16), (5, 90, 6, 48, 20, 40, 0), (64, 1000, 24, 32, 3, 7, 32)])
def test_router_with_corrections_and_groups(cuda, tokens, experts, identity, count, keep, top, tile):
    from poptransformer_b200 import ops
    r = np.random.default_rng(6)
    n = experts + identity
    z, corr = (2.0 * r.standard_normal((tokens, n))).astype(np.float32), (0.5 * r.standard_normal(n) - 0.4).astype(np.float32)     # (most corrected scores are negative)
    idx, wt = ref.choose(z.astype(np.float64), corr.astype(np.float64), top, count, keep)
    for correction in (corr, None):
        if correction is None:
            idx, wt = ref.choose(z.astype(np.float64), 0.0, top, count, keep)
        expert, pair_row = (torch.full((tokens, top), -5, dtype=torch.int32, device=cuda) for _ in range(2))
        weight, kw = torch.full((tokens, top), float("nan"), device=cuda), {}
        h = bf16(r.standard_normal((tokens, 24)))
        if tile:
            rows = tile * ops.moe_max_tiles(tokens, experts, top, tile)
            buf = lambda: torch.full((rows,), -5, dtype=torch.int32, device=cuda)
            gathered, row_token = torch.full((rows, 24), -3.0, dtype=BF16, device=cuda), buf()
            kw = dict(tile=tile, tile_expert=buf(), tile_rows=buf(), row_token=row_token, counts=buf(), h=as_type(h, BF16, cuda), h_ld=24, gathered=gathered)
        ops.moe_route(as_type(z, F32, cuda), tokens, experts, top, expert, weight, pair_row=pair_row, score=ops.MOE_SOFTMAX_ALL,
                      correction=None if correction is None else as_type(correction, F32, cuda), groups=count, keep=keep, identity=identity, **kw)
        e, rows_of = expert.cpu().numpy(), pair_row.cpu().numpy()
        assert np.array_equal(e, np.where(idx < experts, idx, -1)) and rel(weight.cpu(), wt) < 2e-6
        assert ((rows_of < 0) == (idx >= experts)).all()
        placed = idx < experts
        if not tile:
            assert np.array_equal(rows_of[placed], np.arange(tokens * top).reshape(tokens, top)[placed])
            continue
        at, token = rows_of[placed], np.nonzero(placed)[0]
        assert len(set(at.tolist())) == len(at) and np.array_equal(row_token.cpu().numpy()[at], token)
        assert np.array_equal(kw["tile_expert"].cpu().numpy()[at // tile], idx[placed]) and np.array_equal(back(gathered)[at], h[token])
        assert (row_token >= 0).sum().item() == placed.sum()
        used = np.where(kw["tile_expert"].cpu().numpy()[:rows // tile] < 0, 0, kw["tile_rows"].cpu().numpy()[:rows // tile])
        assert used.sum() == placed.sum() and (at % tile < used[at // tile]).all()


def test_router_takes_the_first_of_equals(cuda):
    from poptransformer_b200 import ops
    z = torch.zeros((2, 8), device=cuda)
    z[1, 6:] = 1.0
    expert, weight = torch.zeros((2, 3), dtype=torch.int32, device=cuda), torch.zeros((2, 3), device=cuda)
    ops.moe_route(z, 2, 8, 3, expert, weight, score=ops.MOE_SOFTMAX_ALL, groups=4, keep=2)
    assert expert.tolist() == [[0, 1, 2], [6, 7, 0]] and torch.allclose(weight[0], torch.full((3,), 1 / 3, device=cuda))


# ------------------------------------------------------------------------------------------ latent attention
KINDS = [(F32, True), (BF16, True), (BF16, False)]
SHAPES = [(4, 24, 16, 32, 48, 40), (20, 128, 64, 128, 512, 96), (33, 64, 32, 64, 256, 300), (3, 13, 6, 11, 21, 17), (2, 200, 48, 120, 72, 8), (17, 264, 16, 16, 96, 32)]


@pytest.mark.parametrize("dtype,plain", KINDS)
@pytest.mark.parametrize("shape", SHAPES)
def test_gate_per_output_and_latents_of_another_layer(cuda, dtype, plain, shape):
    """Two sites over one cache, of which the second appends nothing: three sequences of unequal length in portions and single tokens."""
    site = LatentSite(cuda, dtype, 3, *shape, 256, per_value=True)
    H, D, R, V, rank, q_rank = shape
    reader = LatentSite(cuda, dtype, 3, H + 2, D, R, V, rank, q_rank + 8, 256, seed=1, per_value=H % 2 == 0, of=site)
    lens = [135, 70, 134]
    x, q = zip(*(site.inputs(n, 8 + i) for i, n in enumerate(lens)))
    rx, rq = zip(*(reader.inputs(n, 28 + i) for i, n in enumerate(lens)))
    takes, slots, at, got = ([1, 2, 1], [63, 1, 64], [3, 2, 1], [20, 33, 60], [2, 2, 2], [1, 1, 1], [1, 1, 1], [10, 24, 1], [1, 1, 1], [33, 3, 2]), [2, 0, 1], [0, 0, 0], [[[], []] for _ in lens]
    for take in takes:
        cut = lambda t: np.concatenate([t[i][at[i]:at[i] + n] for i, n in enumerate(take)])
        for k, o in enumerate((site(cut(x), cut(q), take, at, slots, plain), reader(cut(rx), cut(rq), take, at, slots, plain))):
            for i, part in enumerate(np.split(o, np.cumsum(take)[:-1])):
                got[i][k].append(part)
        at = [a + n for a, n in zip(at, take)]
    assert at == lens
    for i in range(3):
        for k, want in enumerate((site.oracle(x[i], q[i]), reader.oracle(rx[i], rq[i], x[i]))):
            g = np.concatenate(got[i][k])
            err = np.abs(g - want).max(1)
            assert err.max() < (5e-5 if dtype == F32 else 6e-2), (i, k, int(err.argmax()), float(err.max()))
            assert rel(g, want) < (3e-6 if dtype == F32 else 1.2e-2)


@pytest.mark.parametrize("dtype,plain", KINDS)
def test_one_far_latent_through_a_reading_layer(cuda, dtype, plain):
    """One position's latent points where every query of the reading layer looks, and carries a value of its own: every query from it on must
    find it, and none before, across pages, portions and decoding."""
    n, H, D, R, V, rank = 230, 3, 8, 8, 16, 64
    special = [0, 1, 62, 63, 64, 65, 127, 128, 129, 198]
    B = len(special)
    site = LatentSite(cuda, dtype, B, H, D, R, V, rank, 16, 256, scale=1.0)
    site.kn[:] = 1.0
    site.w.kv_norm.fill_(1.0)
    reader = LatentSite(cuda, dtype, B, H, D, R, V, rank, 16, 256, scale=1.0, per_value=True, of=site)
    reader.uk[:], reader.uv[:] = 0.0, 0.0
    reader.uk[:, 0, 0], reader.uv[:, :, 0] = 1.0, 1.0
    reader.w.w_k, reader.w.w_v = as_type(reader.uk.transpose(0, 2, 1), dtype, cuda), as_type(reader.uv, dtype, cuda)
    reader.up = reader.ops.DenseLinear(as_type(np.concatenate([reader.uk.reshape(-1, rank), reader.uv.reshape(-1, rank)]), dtype, cuda), dtype)
    xs, qs, rxs, rqs = [], [], [], []
    for b, j in enumerate(special):
        x, q = site.inputs(n, 40 + b)
        rx, rq = reader.inputs(n, 80 + b)
        x[:, 16] = 0.0                                         # (the first latent dimension)
        x[j, 16:16 + rank] = 0.0
        x[j, 16] = 9.0
        x[:, 16 + rank:16 + rank + R] *= 0.1
        rx[:, -H * V:], rq[..., 0] = 8.0, 2.0                  # (open gates)
        xs.append(x), qs.append(q), rxs.append(rx), rqs.append(rq)
    want = np.stack([reader.oracle(rx, rq, x) for x, rx, rq in zip(xs, rxs, rqs)])
    seen = np.arange(n)[None] >= np.array(special)[:, None]
    assert ((want.min(2) > 5) == seen).all()
    got, at = [], 0
    for m in [100, 2, 57] + [1] * 71:
        cut = lambda t: np.concatenate([v[at:at + m] for v in t])
        site(cut(xs), cut(qs), [m] * B, [at] * B, range(B), plain)
        got.append(reader(cut(rxs), cut(rqs), [m] * B, [at] * B, range(B), plain).reshape(B, m, -1))
        at += m
    got = np.concatenate(got, 1)
    wrong = np.argwhere((got.min(2) > 5) != seen)
    assert not len(wrong), [(special[b], int(i)) for b, i in wrong[:5]]
    assert np.abs(got - want).max() < (1e-4 if dtype == F32 else 8e-2)


@pytest.mark.parametrize("plain", [True, False])
def test_many_decoding_rows_with_a_gate_per_output(cuda, plain):
    """More sequences than SMs, more than the 16 tokens of a tile, and positions from 0 to several pages."""
    site = LatentSite(cuda, BF16, 170, 18, 32, 16, 32, 128, 32, 330, per_value=True)
    r = np.random.default_rng(9)
    for B in (170, 35):
        lens = [int(v) for v in r.integers(1, 300, B)]
        lens[:3] = [1, 64, 65]
        x, q = zip(*(site.inputs(n, 60 + i) for i, n in enumerate(lens)))
        site.cache.pool.fill_(float("nan"))
        head = [i for i, n in enumerate(lens) if n > 1]
        site(np.concatenate([x[i][:-1] for i in head]), np.concatenate([q[i][:-1] for i in head]), [lens[i] - 1 for i in head], [0] * len(head), head, plain, check_cq=False)
        got = site(np.stack([t[-1] for t in x]), np.stack([t[-1] for t in q]), [1] * B, [n - 1 for n in lens], range(B), plain)
        for i in list(range(0, B, 9)) + [0, 1, 2]:
            assert rel(got[i], site.oracle(x[i], q[i])[-1]) < 2e-2, (B, i, lens[i])


# ------------------------------------------------------------------------------------------ whole models
def poison(dec, n):
    """Nothing may depend on what buffers and states held (padding rows of the experts' tiles, padded columns, a slot's last sequence)."""
    dec.rows_prompt = dec._row_buffers(n)
    for r in (dec.rows_prompt, dec.rows_decode):
        for t in [v for x in vars(r).values() for v in (x if isinstance(x, list) else [x])]:
            if torch.is_tensor(t) and t.is_floating_point():
                t.fill_(float("nan"))
    for c in dec.caches.values():
        c.pool.fill_(float("nan"))
    dec.shift_state.fill_(float("nan"))
    dec.shift_next.fill_(float("nan"))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_model_prompts_portions_and_decoding(cuda, name, dtype):
    cfg = CONFIGS[name]
    w = weights(cfg, seed=11)
    n = 150
    tokens = prompt(n, cfg["vocab"])
    sums = []
    want = ref.PuputarOracle(cfg, w).forward(tokens, sums)
    dec = decoder(cfg, w, 3, 192, dtype)
    poison(dec, n)
    for plain in (False, True):
        dec.plain = plain
        if plain:
            dec.rows_prompt = None
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
            assert per.max() < (1e-4 if dtype == "float32" else 6e-2), (cuts[:4], int(per.argmax()), float(per.max()))
            assert rel(got, want) < TOL[dtype]


def test_caches_belong_to_the_layers_that_fill_them(cuda):
    dec = decoder(CONFIGS["mixed"], weights(CONFIGS["mixed"], seed=11), 2, 64)
    assert dec.caches[2] is dec.caches[0] and dec.caches[3] is dec.caches[0] and len({id(c) for c in dec.caches.values()}) == 3


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
    orc = [ref.PuputarOracle(cfg, w).forward(t) for t in toks]
    for dtype in ("float32", "bfloat16"):
        dec = decoder(cfg, w, 3, 128, dtype)
        poison(dec, 90)
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
    want = np.stack([ref.PuputarOracle(cfg, w).forward(toks[b])[18:] for b in picked])
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
        if rnd % 2 == 0:                          # (else: the states that the batch before left)
            poison(dec, 200)
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
    want = ref.PuputarOracle(cfg, w).forward(tokens)
    assert rel(got, want) < TOL[dtype]
    assert rel(got[-20:], want[-20:]) < TOL[dtype]


def test_first_tokens(cuda):
    """Prompts of 1 .. 9 tokens, with a shift that takes all of the token before."""
    cfg = config([latent(mlp=dense()), latent2(kv_from=0, mlp=moe())], width=64)
    w = weights(cfg, seed=16)
    w["l0.shift"][:] = 1.0
    orc = ref.PuputarOracle(cfg, w)
    for dtype in ("float32", "bfloat16"):
        dec = decoder(cfg, w, 9, 64, dtype)
        poison(dec, 64)
        toks = [prompt(n, cfg["vocab"], n) for n in range(1, 10)]
        seqs = [dec.open() for _ in toks]
        got = dec.extend([(s, t, list(range(len(t)))) for s, t in zip(seqs, toks)]).cpu().numpy()
        assert rel(got, np.concatenate([orc.forward(t) for t in toks])) < TOL[dtype]


def test_pages_of_another_size(cuda):
    cfg = CONFIGS["mixed"]
    w = weights(cfg, seed=24)
    tokens = prompt(70, cfg["vocab"])
    want = ref.PuputarOracle(cfg, w).forward(tokens)
    for dtype in ("float32", "bfloat16"):
        assert rel(run_cut(decoder(cfg, w, 1, 96, dtype, page_size=24), tokens, [50] + [1] * 10 + [10]), want) < TOL[dtype]


def test_a_far_token_decides(cuda):
    """In a whole model: one token's latent outweighs all others for every later query of the layer that reads another's cache; replacing
    that token far back changes what comes out as much as in the oracle."""
    cfg = config([latent2(heads=4, kv_rank=64, dim=16), latent2(heads=2, kv_rank=64, dim=16, kv_from=0, mlp=dense())], width=64, groups=2)
    w = weights(cfg, seed=25)
    w["l1.mix.uk"], w["l1.mix.uq"] = bf16(6 * w["l1.mix.uk"]), bf16(3 * w["l1.mix.uq"])       # scores of the reading layer far apart
    orc = ref.PuputarOracle(cfg, w)
    tokens = prompt(300, cfg["vocab"], 3)
    for at in (0, 1, 63, 64, 130):
        other = tokens.copy()
        other[at] = (other[at] + 1) % cfg["vocab"]
        change = orc.forward(other) - orc.forward(tokens)
        for dtype, tol in (("float32", 1e-3), ("bfloat16", 0.5)):
            dec = decoder(cfg, w, 1, 320, dtype)
            got = run_cut(dec, other, [200] + [1] * 100) - run_cut(dec, tokens, [200] + [1] * 100)
            assert np.abs(got[:at]).max(initial=0) < (1e-4 if dtype == "float32" else 5e-2)
            assert rel(got, change) < tol, (at, dtype)


def test_missing_parts_would_show(cuda):
    """The comparison above is sharp: an oracle with one part changed is far from the kernels."""
    cfg = CONFIGS["mixed"]
    w = weights(cfg, seed=22)
    tokens = prompt(140, cfg["vocab"])
    dec = decoder(cfg, w, 1, 192, "float32")
    s = dec.open()
    got = dec.extend([(s, tokens, list(range(140)))]).cpu().numpy()
    right = rel(got, ref.PuputarOracle(cfg, w).forward(tokens))
    assert right < TOL["float32"]

    def changed(edit_cfg=None, edit_w=None):
        c, v = json.loads(json.dumps(cfg)), dict(w)
        for f, x in ((edit_cfg, c), (edit_w, v)):
            if f:
                f(x)
        return rel(got, ref.PuputarOracle(c, v).forward(tokens))

    mix = lambda c, i: c["layers"][i]["mixer"]
    router = lambda c, i: c["layers"][i]["mlp"]["router"]
    zero = lambda k: dict(edit_w=lambda v: v.update({k: 0 * v[k]}))
    one = lambda k: dict(edit_w=lambda v: v.update({k: 0 * v[k] + 1}))
    edits = [dict(edit_cfg=lambda c: mix(c, 0)["rot"].update(base=2e3)), dict(edit_cfg=lambda c: mix(c, 2)["rot"].update(base=2e3)), dict(edit_cfg=lambda c: mix(c, 2).update(scale=1.2 * mix(c, 2)["scale"])),
             dict(edit_cfg=lambda c: mix(c, 3).update(scale=0.8 * mix(c, 3)["scale"])), dict(edit_cfg=lambda c: c["norm"].update(groups=2)), dict(edit_cfg=lambda c: c["norm"].update(eps=1e-2)),
             dict(edit_cfg=lambda c: router(c, 0).update(top=1)), dict(edit_cfg=lambda c: router(c, 0)["groups"].update(keep=2)), dict(edit_cfg=lambda c: router(c, 3)["groups"].update(keep=1)),
             dict(edit_cfg=lambda c: router(c, 3)["groups"].update(count=6)), zero("l0.mlp.correction"), zero("l3.mlp.correction"), zero("l0.mix.g"), zero("l1.mix.g"), zero("l4.mix.g"),
             zero("l0.shift"), zero("l4.shift"), zero("l1.mlp.act"), zero("l1.mlp.up.b"), zero("l2.mlp.down.b"), one("embed.norm"), one("final.norm"), one("l0.norm1"), one("l3.norm2"), one("l0.mix.dkv.norm"),
             one("l2.mix.dq.norm")]
    far = [changed(**e) for e in edits]
    assert [(i, d, right) for i, d in enumerate(far) if d < 50 * TOL["float32"]] == []


# ------------------------------------------------------------------------------------------ the decode loop
@pytest.mark.parametrize("dtype,tol", [("float32", 1e-4), ("bfloat16", 8e-2)])
def test_greedy_generation(cuda, dtype, tol):
    cfg = CONFIGS["mixed"]
    w = weights(cfg, seed=17)
    orc = ref.PuputarOracle(cfg, w)
    max_len, lens = 80, [3, 20, 9]
    dec = decoder(cfg, w, 3, max_len, dtype, pad_id=-1)
    ids = np.full((3, max_len), -1, np.int32)
    for b, n in enumerate(lens):
        ids[b, :n] = prompt(n, cfg["vocab"], b)
    eager = dec.run(ids, max_loop=max_len - 1)["Loop:0"]
    assert all((eager[b, :n] == ids[b, :n]).all() for b, n in enumerate(lens)) and (eager >= 0).all()
    assert greedy_ok(orc, eager, lens, tol) > 0.9
    dec.capture()
    assert np.array_equal(dec.run(ids, max_loop=max_len - 1)["Loop:0"], eager)          # one CUDA graph per step, caches and states of the run before left behind
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


def test_missing_or_misshapen_tensors_are_named(cuda):
    from poptransformer_b200 import PtError, registry
    cfg = CONFIGS["mixed"]
    sd = tensors(weights(cfg, seed=20))
    for key in ("l2.shift", "l0.mlp.correction", "l1.mlp.act", "head"):
        with pytest.raises(PtError, match=key):
            registry.build_decoder(cfg, {k: v for k, v in sd.items() if k != key}, 1, 16)
        with pytest.raises(PtError, match=key):
            registry.build_decoder(cfg, {**sd, key: sd[key][1:]}, 1, 16)


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
    orc = {k: ref.PuputarOracle(cfg, w).forward(t) for k, t in toks.items()}
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
    cfg = CONFIGS["one-group"]
    w = weights(cfg, seed=21)
    write_model(str(tmp_path), cfg, w)
    a, b = prompt(6, cfg["vocab"], 1).tolist(), prompt(3, cfg["vocab"], 2).tolist()
    cmd = [sys.executable, "-m", "poptransformer_b200", "generate", "--model", str(tmp_path), "--prompt", ",".join(map(str, a)), "--prompt", ",".join(map(str, b)),
           "--new", "10", "--dtype", "float32", "--prefill"]
    p = subprocess.run(cmd, capture_output=True, text=True, timeout=300, cwd=ROOT)
    assert p.returncode == 0, p.stderr[-2000:]
    rows = [json.loads(ln)["ids"] for ln in p.stdout.splitlines()]
    assert [len(r) for r in rows] == [16, 16] and rows[0][:6] == a and rows[1][:3] == b
    assert greedy_ok(ref.PuputarOracle(cfg, w), np.array(rows), [6, 3], 1e-4) == 1.0
