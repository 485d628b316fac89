"""Sabisun on the GPU against the plain restatement (oracle/sabisun_np.py): every mechanism alone, then whole models in prompts,
portions, batches and decoding, with slots and pages that are used again, and greedy generation through the decode loop."""
import json
import os
import subprocess
import sys
from types import SimpleNamespace

import numpy as np
import pytest
import torch

from oracle import sabisun_np as ref
from sabisun_util import CONFIGS, attn, config, decoder, mamba, weights
from seq_util import PagedAttention, as_type, bf16, greedy_ok, i32, prompt, rel, run_cut, view_of, write_model

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = {"float32": 2e-5, "bfloat16": 2e-2}       # rms of the difference over the rms of the logits, whole model


# ------------------------------------------------------------------------------------------ mechanisms
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("streams,width", [(1, 40), (2, 96), (3, 64), (4, 33), (5, 72), (7, 30)])
def test_hyper_connections(cuda, dtype, streams, width):
    from poptransformer_b200 import ops
    r = np.random.default_rng(1)
    rows, vocab, ld, eps, mult = 6, 11, width + 8, 1e-4, 0.6
    table = bf16(r.standard_normal((vocab, width)))
    ids = r.integers(0, vocab, rows)
    w_in, w_in2, w_out, mix, nw = (r.standard_normal(s).astype(np.float32) for s in (streams, streams, streams, (streams, streams), width))
    y = r.standard_normal((rows, width)).astype(np.float32)
    f = lambda a: torch.from_numpy(np.ascontiguousarray(a)).to(cuda)
    xs = torch.full((rows, streams, width), float("nan"), device=cuda)
    h = torch.full((rows, ld), float("nan"), dtype=dtype, device=cuda)
    ops.hyper(xs, rows, eps, norm_w=f(nw), h=h, h_ld=ld, w_in=f(w_in), table=as_type(table, dtype, cuda), ids=i32(ids, cuda))
    X = np.repeat(table[ids][None], streams, 0).astype(np.float64)
    tol = 1e-5 if dtype == torch.float32 else 6e-3
    assert np.array_equal(xs.cpu().numpy(), X.transpose(1, 0, 2).astype(np.float32))
    assert rel(h[:, :width].float().cpu(), ref.rms(ref.stream_read(X, w_in), eps) * nw) < tol
    assert not h[:, width:].any()
    # write, next read, and the sum
    sums = torch.empty((rows, width), device=cuda)
    X = r.standard_normal((streams, rows, width))
    xs.copy_(f(X.transpose(1, 0, 2).astype(np.float32)))
    ops.hyper(xs, rows, eps, norm_w=f(nw), h=h, h_ld=ld, w_in=f(w_in2), y=f(y), y_ld=width, mix=f(mix), w_out=f(w_out), mult=mult, sum_out=sums)
    N = ref.stream_write(X, y, mix, w_out, mult)
    assert rel(xs.cpu(), N.transpose(1, 0, 2)) < 1e-6 and rel(sums.cpu(), N.sum(0)) < 1e-6
    assert rel(h[:, :width].float().cpu(), ref.rms(ref.stream_read(N, w_in2), eps) * nw) < tol
    # the end of the model on chosen rows: the sum is normalised, the streams stay as they are
    pick, before = [4, 1], xs.clone()
    ops.hyper(xs, 2, eps, norm_w=f(nw), h=h, h_ld=ld, y=f(y), y_ld=width, mix=f(mix), w_out=f(w_out), mult=mult, row_index=i32(pick, cuda))
    M = ref.stream_write(N, y, mix, w_out, mult).sum(0)[pick]
    assert rel(h[:2, :width].float().cpu(), ref.rms(M, eps) * nw) < tol and torch.equal(before, xs)


@pytest.mark.parametrize("m,n,k", [(1, 5, 7), (3, 64, 16), (70, 130, 33), (129, 65, 200)])
def test_true_fp32_product(cuda, m, n, k):
    from poptransformer_b200 import ops
    r = np.random.default_rng(2)
    x, w = r.standard_normal((m, k)).astype(np.float32), r.standard_normal((n, k)).astype(np.float32)
    lin = ops.DenseLinear(as_type(w, torch.float32, cuda), torch.float32)
    for epi, f in ((ops.EPI_STORE, lambda v: v), (ops.EPI_RELU2, lambda v: np.maximum(v, 0) ** 2)):
        out = torch.full((m, n + 3), -7.0, device=cuda)
        lin(as_type(x, torch.float32, cuda), out, m, n + 3, epilogue=epi, alpha=0.3)
        assert rel(out[:, :n].cpu(), f(0.3 * (x.astype(np.float64) @ w.T))) < 1e-6
        assert (out[:, n:] == -7).all()


@pytest.mark.parametrize("rows", [1, 5, 7, 8, 16, 17, 31, 70, 257, 600])
@pytest.mark.parametrize("n,k", [(24, 40), (200, 64), (513, 328), (128, 2048)])
def test_bf16_linear(cuda, rows, n, k):
    """Skinny-matmul kernel for few rows, tcgen05 GEMM beyond; k that is no multiple of a block, n that is no multiple of a tile."""
    from poptransformer_b200 import ops
    r = np.random.default_rng(3)
    x, w = bf16(r.standard_normal((rows, k))), bf16(r.standard_normal((n, k)) * k ** -0.5)
    want = 0.7 * (x.astype(np.float64) @ w.T)
    flag = torch.zeros(1, dtype=torch.int32, device=cuda)
    L = ops._lib.lib()
    lws = torch.zeros(L.pt_linear_workspace_bytes(min(rows, 32), n, 32), dtype=torch.uint8, device=cuda)
    gws = torch.zeros(L.pt_gemm_workspace_bytes(rows, n, 8), dtype=torch.uint8, device=cuda)
    lin = ops.DenseLinear(as_type(w, torch.bfloat16, cuda), torch.bfloat16)
    xp = torch.zeros((rows, lin.ld), dtype=torch.bfloat16, device=cuda)
    xp[:, :k] = as_type(x, torch.bfloat16, cuda)
    for dt, tol in ((torch.float32, 1e-5), (torch.bfloat16, 4e-3)):
        for epi, f in ((ops.EPI_STORE, lambda v: v), (ops.EPI_RELU2, lambda v: np.maximum(v, 0) ** 2)):
            out = torch.full((rows, n + 8), -7.0, dtype=dt, device=cuda)
            lin(xp, out, rows, n + 8, epilogue=epi, alpha=0.7, linear_ws=lws, gemm_ws=gws, error_flag=flag)
            assert rel(out[:, :n].float().cpu(), f(want)) < tol, (dt, epi)
            assert (out[:, n:] == -7).all()
    if rows <= 32:      # the skinny kernel also where the decoder prefers the GEMM
        out = torch.empty((rows, n), device=cuda)
        ops.linear(xp, lin.skinny, out, workspace=lws, alpha=0.7)
        assert rel(out.cpu(), want) < 1e-5
    assert int(flag.item()) == 0


ATTN_SHAPES = [  # heads, kv heads, dim, vdim, window, keep_first, sink
    (4, 2, 32, 32, 24, 5, True), (4, 4, 64, 32, 64, 64, True), (6, 2, 16, 40, 65, 1, True), (16, 1, 128, 128, 130, 70, False), (8, 8, 40, 64, 0, 0, True),
    (24, 2, 64, 128, 63, 0, True), (3, 3, 24, 8, 1, 3, False), (2, 1, 96, 96, 0, 0, False), (5, 5, 20, 12, 17, 2, True), (10, 2, 160, 48, 100, 10, True)]


@pytest.mark.parametrize("dtype,plain", [(torch.float32, True), (torch.bfloat16, True), (torch.bfloat16, False)])
@pytest.mark.parametrize("H,G,D,V,window,keep,with_sink", ATTN_SHAPES)
def test_window_attention(cuda, dtype, plain, H, G, D, V, window, keep, with_sink):
    """Three sequences of unequal length: first portions of a prompt, later portions (down to two tokens), then single tokens."""
    r = np.random.default_rng(4)
    lens = [215, 70, 134]
    sink = 2 * r.standard_normal(H) if with_sink else None
    q, k, v = ([bf16(r.standard_normal((n, h, d))) for n in lens] for h, d in ((H, D), (G, D), (G, V)))
    scale = 2.0 * D ** -0.5
    att = PagedAttention(cuda, dtype, 3, G, D, V, 256)
    got = [[] for _ in lens]
    at = [0, 0, 0]
    slots = [2, 0, 1]
    for take in ([64, 2, 65], [3, 2, 1], [100, 33, 60], [2, 2, 2], [1, 1, 1], [1, 1, 1], [10, 24, 1], [1, 1, 1], [33, 4, 2]):
        cut = lambda t: np.concatenate([t[i][at[i]:at[i] + n] for i, n in enumerate(take)])
        o = att(cut(q), cut(k), cut(v), take, at, slots, scale, window, keep, sink, plain)
        for i, part in enumerate(np.split(o, np.cumsum(take)[:-1])):
            got[i].append(part)
            at[i] += take[i]
    assert at == lens
    for i, n in enumerate(lens):
        want = ref.attention(q[i].astype(np.float64), k[i].astype(np.float64), v[i].astype(np.float64), scale, ref.visible(n, window or None, keep), sink)
        err = np.abs(np.concatenate(got[i]) - want).max(1)
        assert err.max() < (2e-5 if dtype == torch.float32 else 2.5e-2), (i, int(err.argmax()), float(err.max()))


@pytest.mark.parametrize("dtype,plain", [(torch.float32, True), (torch.bfloat16, True), (torch.bfloat16, False)])
@pytest.mark.parametrize("window,keep", [(1, 0), (24, 5), (64, 64), (65, 63), (63, 65), (130, 1), (0, 0)])
def test_single_keys_at_every_edge(cuda, dtype, plain, window, keep):
    """One key per sequence matches every query strongly and carries a value of its own, so each query's output says whether it saw
    that key: keys around the kept tokens, page borders and window edges, for every query, in prompts and in decoding."""
    n, H, G, D, V = 200, 2, 1, 32, 32
    special = sorted({0, 1, 62, 63, 64, 65, 127, 128, 129, n - 2, *(max(0, keep + d) for d in (-1, 0, 1))})
    r = np.random.default_rng(5)
    B = len(special)
    q = np.zeros((B, n, H, D)); q[..., 0] = 8.0
    k = bf16(0.1 * r.standard_normal((B, n, G, D)))
    v = bf16(0.1 * r.standard_normal((B, n, G, V)))
    for b, j in enumerate(special):
        k[b, j, :, 0], v[b, j] = 8.0, 4.0
    want = [ref.attention(q[b], k[b].astype(np.float64), v[b].astype(np.float64), 0.3, ref.visible(n, window or None, keep), None) for b in range(B)]
    seen = np.array([[ref.visible(n, window or None, keep)[i, j] for i in range(n)] for j in special])
    assert seen.any(1).all() and ((np.array(want)[:, :, 0] > 3) == seen).all()          # the construction shows what it should
    split = n - 75
    att = PagedAttention(cuda, dtype, B, G, D, V, 256)
    flat = lambda t, a, b: t[:, a:b].reshape(B * (b - a), *t.shape[2:])
    got = [att(flat(q, 0, split), flat(k, 0, split), flat(v, 0, split), [split] * B, [0] * B, range(B), 0.3, window, keep, None, plain).reshape(B, split, -1)]
    for i in range(split, n):
        got.append(att(flat(q, i, i + 1), flat(k, i, i + 1), flat(v, i, i + 1), [1] * B, [i] * B, range(B), 0.3, window, keep, None, plain).reshape(B, 1, -1))
    got = np.concatenate(got, 1)
    wrong = np.argwhere((got[:, :, 0] > 3) != seen)
    assert not len(wrong), [(special[b], int(i)) for b, i in wrong[:5]]
    assert np.abs(got - np.array(want)).max() < (1e-4 if dtype == torch.float32 else 4e-2)


@pytest.mark.parametrize("plain", [True, False])
def test_attention_over_another_layers_cache(cuda, plain):
    """Queries only: the keys are those an earlier call left, under another mask and scale; also for the newest token."""
    r = np.random.default_rng(6)
    n, H, G, D, V = 150, 4, 2, 32, 64
    k, v = bf16(r.standard_normal((n, G, D))), bf16(r.standard_normal((n, G, V)))
    q = [bf16(r.standard_normal((n, H, D))) for _ in range(2)]
    att = PagedAttention(cuda, torch.bfloat16, 1, G, D, V, 192)
    for a, b in ((0, 120), (120, 121), (121, 149), (149, 150)):
        att(q[0][a:b], k[a:b], v[a:b], [b - a], [a], [0], 0.2, 20, 3, None, plain)
        o = att(q[1][a:b], None, None, [b - a], [a], [0], 0.4, 90, 9, None, plain)
        want = ref.attention(q[1].astype(np.float64), k.astype(np.float64), v.astype(np.float64), 0.4, ref.visible(n, 90, 9), None)[a:b]
        assert np.abs(o - want).max() < 2.5e-2


SSM_SHAPES = [  # heads, vdim, state, groups, taps, norm_groups
    (4, 16, 24, 2, 4, 1), (2, 32, 64, 1, 3, 2), (3, 8, 16, 3, 2, 3), (4, 64, 128, 2, 4, 8), (2, 40, 200, 2, 5, 1), (3, 33, 19, 1, 1, 9), (6, 24, 256, 3, 4, 2),
    (1, 8, 8, 1, 7, 4)]


class SsmSite:
    """One state-space call site: its weights, its state, and the oracle's view of the same."""

    def __init__(self, dev, dt, n_slots, heads, vdim, state, groups, taps, norm_groups, seed=7):
        r = np.random.default_rng(seed)
        self.dev, self.dt, self.inner, self.C = dev, dt, heads * vdim, heads * vdim + 2 * groups * state
        w = SimpleNamespace(heads=heads, vdim=vdim, state=state, groups=groups, taps=taps, norm_groups=norm_groups, eps=1e-5)
        w.conv_w, w.conv_b = r.standard_normal((self.C, taps)) * 0.6, 0.2 * r.standard_normal(self.C)
        w.dt_bias, w.A_log, w.D = r.uniform(-4, 1, heads), r.uniform(-3, 4, heads), r.standard_normal(heads)
        w.norm_w = 1 + 0.2 * r.standard_normal(self.inner)
        self.np = SimpleNamespace(**vars(w))
        for n in ("conv_w", "conv_b", "dt_bias", "A_log", "D", "norm_w"):
            setattr(w, n, as_type(getattr(w, n), torch.float32, dev))
        self.w = w
        # whatever an earlier sequence left must not matter
        self.ring = torch.full((n_slots, taps, self.C), float("nan"), dtype=dt, device=dev)
        self.state = torch.full((n_slots, heads, state, vdim), float("nan"), device=dev)
        self.width = self.inner + self.C + heads

    def __call__(self, zx, lens, starts, slots, plain):
        from poptransformer_b200 import ops
        T, dev = zx.shape[0], self.dev
        ld, out_ld = ops.pad_to(self.width, 8), ops.pad_to(self.inner, 64)
        buf = torch.zeros((T, ld), dtype=self.dt, device=dev)
        buf[:, :self.width] = as_type(zx, self.dt, dev)
        out = torch.full((T, out_ld), float("nan"), dtype=self.dt, device=dev)
        n = ops._lib.lib().pt_ssm_workspace_bytes(T, len(lens), self.w.heads, self.w.vdim, self.w.state)
        ops.ssm(view_of(lens, starts, slots, dev), buf, ld, out, out_ld, self.w, self.ring, self.state, torch.empty((T, self.inner), device=dev),
                torch.empty((T, self.C), dtype=self.dt, device=dev), torch.empty((T, self.w.heads), device=dev),
                torch.full((n,), 255, dtype=torch.uint8, device=dev), plain=plain)
        assert not out[:, self.inner:].any()
        return out[:, :self.inner].float().cpu().numpy()

    def oracle(self, zx):
        w, T = self.np, zx.shape[0]
        z, xbc, dt = np.split(zx.astype(np.float64), [self.inner, self.inner + self.C], axis=1)
        x, B, C = np.split(ref.silu(ref.causal_conv(xbc, w.conv_w, w.conv_b)), [self.inner, self.inner + w.groups * w.state], axis=1)
        y = ref.ssm_scan(x.reshape(T, w.heads, w.vdim), B.reshape(T, w.groups, w.state), C.reshape(T, w.groups, w.state), ref.softplus(dt + w.dt_bias), w.A_log, w.D)
        return ref.gated_group_norm(y.reshape(T, -1), z, w.norm_w, w.norm_groups, w.eps)


@pytest.mark.parametrize("dtype,plain", [(torch.float32, True), (torch.bfloat16, True), (torch.bfloat16, False)])
@pytest.mark.parametrize("heads,vdim,state,groups,taps,norm_groups", SSM_SHAPES)
def test_state_space_layer(cuda, dtype, plain, heads, vdim, state, groups, taps, norm_groups):
    """Unequal sequences in portions (single tokens, two tokens, around the chunk of 64, long), state and convolution carried over."""
    r = np.random.default_rng(8)
    lens = [205, 75, 136]
    site = SsmSite(cuda, dtype, 4, heads, vdim, state, groups, taps, norm_groups)
    zx = [bf16(r.standard_normal((n, site.width))) for n in lens]
    got, at, slots = [[] for _ in lens], [0, 0, 0], [3, 0, 1]
    for take in ([1, 1, 2], [1, 1, 1], [1, 1, 1], [63, 2, 65], [64, 2, 1], [66, 3, 60], [1, 1, 1], [1, 60, 1], [7, 4, 4]):
        o = site(np.concatenate([zx[i][at[i]:at[i] + n] for i, n in enumerate(take)]), take, at, slots, plain)
        for i, part in enumerate(np.split(o, np.cumsum(take)[:-1])):
            got[i].append(part)
            at[i] += take[i]
    assert at == lens
    for i in range(3):
        want, g = site.oracle(zx[i]), np.concatenate(got[i])
        assert rel(g, want) < (2e-5 if dtype == torch.float32 else 3e-2)
        per_token = np.sqrt(((g - want) ** 2).mean(1)) / np.sqrt((want ** 2).mean())
        # (a token whose gated row nearly cancels amplifies the bf16 roundings of its x, B and C)
        assert per_token.max() < (2e-4 if dtype == torch.float32 else 0.2) and np.median(per_token) < 1e-2, int(per_token.argmax())


def test_decay_survives_long_running_sums(cuda):
    """A few tokens with huge steps drive a chunk's running log decay to minus tens of thousands; the tokens after them decay
    slowly and must still see each other exactly as without the chunk."""
    site = SsmSite(cuda, torch.bfloat16, 2, 2, 16, 64, 1, 2, 1)
    site.np.A_log[:] = [5.0, 4.0]
    site.np.dt_bias[:] = 0.0
    site.w.A_log, site.w.dt_bias = as_type(site.np.A_log, torch.float32, cuda), as_type(site.np.dt_bias, torch.float32, cuda)
    r = np.random.default_rng(9)
    zx = bf16(r.standard_normal((192, site.width)))
    zx[:, -2:] = bf16(np.where(np.arange(192) % 64 < 40, 6.0, -7.5))[:, None]
    exact = SsmSite(cuda, torch.float32, 2, 2, 16, 64, 1, 2, 1)
    exact.w = site.w
    a = site(zx, [192], [0], [0], False)
    b = exact(zx, [192], [0], [0], True)
    tail = [t for t in range(192) if t % 64 >= 40]
    assert rel(b, site.oracle(zx)) < 1e-4
    assert rel(a[tail], b[tail]) < 8e-3


# ------------------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_model_prompts_portions_and_decoding(cuda, name, dtype):
    cfg = CONFIGS[name]
    w = weights(cfg, seed=11)
    n = 150
    tokens = prompt(n, cfg["vocab"])
    sums = []
    want = ref.SabisunOracle(cfg, w).forward(tokens, sums)
    dec = decoder(cfg, w, 3, 192, dtype)
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
        assert rel(g, t[:len(g)]) < (2e-5 if dtype == "float32" else 2e-2)


def test_more_rows_than_the_skinny_kernels_take(cuda):
    cfg = CONFIGS["wide-heads"]
    w = weights(cfg, seed=13)
    B = 45
    toks = [prompt(20, cfg["vocab"], i) for i in range(B)]
    picked = (0, 17, 31, 32, 44)
    want = np.stack([ref.SabisunOracle(cfg, w).forward(toks[b])[18:] for b in picked])
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
        for t in [c.pool for c in dec.caches.values()] + list(dec.rings.values()) + list(dec.states.values()):
            t.fill_(float("nan"))
        toks = [prompt(n + 2, cfg["vocab"], 10 * rnd + i) for i, n in enumerate(lens)]
        seqs = [dec.open() for _ in lens]
        got = dec.extend([(s, t[:-2], [n - 1]) for s, t, n in zip(seqs, toks, lens)]).cpu().numpy()
        more = [dec.extend([(s, t[n + k:n + k + 1], [0]) for s, t, n in zip(seqs, toks, lens)]).cpu().numpy() for k in range(2)]
        for i, s in enumerate(seqs):
            want = run_cut(fresh, toks[i], [lens[i], 1, 1])
            assert rel(np.stack([got[i], more[0][i], more[1][i]]), want[lens[i] - 1:]) < (1e-5 if dtype == "float32" else 1e-2)
            dec.close(s)
    assert dec.slots.free_pages == 5 and dec.slots.free_slots == 3


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(cuda, dtype):
    cfg = CONFIGS["attention-first"]
    w = weights(cfg, seed=15)
    tokens = prompt(340, cfg["vocab"])
    dec = decoder(cfg, w, 1, 384, dtype)
    got = run_cut(dec, tokens, [9] + [1] * 331)
    want = ref.SabisunOracle(cfg, w).forward(tokens)
    assert rel(got, want) < TOL[dtype]
    assert rel(got[-20:], want[-20:]) < TOL[dtype]


def test_first_tokens(cuda):
    """Prompts of 1 .. 9 tokens: shorter than the convolution, the window and the kept tokens."""
    cfg = config([mamba(conv=6), attn(size=4, keep_first=3)], streams=3, width=64)
    w = weights(cfg, seed=16)
    orc = ref.SabisunOracle(cfg, w)
    for dtype in ("float32", "bfloat16"):
        dec = decoder(cfg, w, 9, 64, dtype)
        toks = [prompt(n, cfg["vocab"], n) for n in range(1, 10)]
        seqs = [dec.open() for _ in toks]
        got = dec.extend([(s, t, list(range(len(t)))) for s, t in zip(seqs, toks)]).cpu().numpy()
        assert rel(got, np.concatenate([orc.forward(t) for t in toks])) < TOL[dtype]


# ------------------------------------------------------------------------------------------ the decode loop
@pytest.mark.parametrize("dtype,tol", [("float32", 1e-4), ("bfloat16", 8e-2)])
def test_greedy_generation(cuda, dtype, tol):
    cfg = CONFIGS["mixed"]
    w = weights(cfg, seed=17)
    orc = ref.SabisunOracle(cfg, w)
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


def test_errors(cuda):
    from poptransformer_b200 import PtError
    cfg = CONFIGS["mixed"]
    dec = decoder(cfg, weights(cfg), 1, 32, "bfloat16")
    s = dec.open()
    with pytest.raises(PtError, match="slots"):
        dec.open()
    with pytest.raises(PtError, match="max_len"):
        dec.extend([(s, prompt(33, cfg["vocab"]), [])])
    with pytest.raises(PtError, match="vocabulary"):
        dec.extend([(s, [cfg["vocab"]], [])])
    with pytest.raises(PtError, match="wanted"):
        dec.extend([(s, [1], [1])])
    assert dec.extend([(s, [1, 2], [1])]).shape == (1, cfg["vocab"])       # the refused calls left nothing behind


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
    orc = {k: ref.SabisunOracle(cfg, w).forward(t) for k, t in toks.items()}
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
    cfg = CONFIGS["one-stream"]
    w = weights(cfg, seed=21)
    write_model(str(tmp_path), cfg, w)
    a, b = prompt(6, cfg["vocab"], 1).tolist(), prompt(3, cfg["vocab"], 2).tolist()
    cmd = [sys.executable, "-m", "poptransformer_b200", "generate", "--model", str(tmp_path), "--prompt", ",".join(map(str, a)), "--prompt", ",".join(map(str, b)),
           "--new", "10", "--dtype", "float32", "--prefill"]
    p = subprocess.run(cmd, capture_output=True, text=True, timeout=300, cwd=ROOT)
    assert p.returncode == 0, p.stderr[-2000:]
    rows = [json.loads(ln)["ids"] for ln in p.stdout.splitlines()]
    assert [len(r) for r in rows] == [16, 16] and rows[0][:6] == a and rows[1][:3] == b
    assert greedy_ok(ref.SabisunOracle(cfg, w), np.array(rows), [6, 3], 1e-4) == 1.0
