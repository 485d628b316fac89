"""Host side of the Pivavik decoder, without a GPU: configuration, registry, order of the layers, and the oracle's own consistency (its
mechanisms against a second formulation)."""
import json

import numpy as np
import pytest

from oracle import pivavik_np as ref
from pivavik_util import CODE, CONFIGS, attention, config, dense, gaps, latent, moe, router_order, weights


def test_configuration_reads_every_layer():
    from poptransformer_b200.pivavik import PivavikConfig
    c = PivavikConfig(CONFIGS["mixed"], 99)
    assert (c.max_len, c.width, c.vocab, c.eps, c.logit_softcap, c.loop) == (99, 96, 150, 1e-5, 6.0, (1, 3, 3))
    assert [x.kind for x in c.layers] == ["latent_attention", "attention", "latent_attention", "attention", "latent_attention"]
    assert [(x.heads, x.dim, x.vdim) for x in c.layers] == [(4, 24, 32), (6, 32, 24), (3, 16, 8), (4, 16, 40), (4, 24, 16)]
    assert [(x.q_rank, x.rank, x.rot_dim, x.base) for x in c.layers[::2]] == [(40, 48, 16, 1e3), (24, 72, 32, 50.0), (40, 48, 16, 1e3)]
    assert [(x.kv_heads, x.window, x.softcap) for x in c.layers[1::2]] == [(2, 40, 3.0), (4, 70, 1.5)]
    assert [x.ff for x in c.layers] == [72, 0, 0, 0, 0]
    assert [x.moe and (x.moe.experts, x.moe.top, x.moe.ff) for x in c.layers] == [None, (6, 2, 40), (9, 3, 72), None, None]


@pytest.mark.parametrize("n,loop", [(4, None), (4, (0, 4, 2)), (5, (1, 3, 3)), (3, (2, 3, 1)), (2, (0, 1, 4))])
def test_order_of_the_layers(n, loop):
    from poptransformer_b200.pivavik import PivavikConfig
    cfg = config([attention() for _ in range(n)], loop=loop)
    runs = PivavikConfig(cfg, 9).runs()
    want = ref.layer_runs(n, cfg["loop"])
    assert [i for i, _ in runs] == [i for i, _ in want]
    # a pass begins where its first layer runs
    assert [t for _, t in runs] == [t if t is not None and i == loop[0] else None for i, t in want]
    if loop == (1, 3, 3):
        assert runs == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (1, 2), (2, None), (3, None), (4, None)]


def edited(lay, **kw):
    lay = json.loads(json.dumps(lay))
    for path, v in kw.items():
        d = lay
        *way, last = path.split("__")
        for k in way:
            d = d[k]
        d[last] = v
    return config([lay])


@pytest.mark.parametrize("bad,match", [
    (config([attention(heads=3, kv_heads=2)]), "heads"), (config([attention(mlp=moe(top=7))]), "experts"), (config([latent(rot=7)]), "rotated"),
    (edited(latent(), mixer__rot__dims=8), "rotated"), (edited(latent(), type="mamba2"), "unknown mixer"), (edited(attention(mlp=dense()), mlp__kind="sparse"), "unknown feed-forward"),
    (config([attention()], loop=(0, 2, 2)), "loop"), (config([attention()], loop=(1, 1, 2)), "loop"), (config([attention()], loop=(0, 1, 0)), "loop")])
def test_configuration_refuses(bad, match):
    from poptransformer_b200 import PtError
    from poptransformer_b200.pivavik import PivavikConfig
    with pytest.raises(PtError, match=match):
        PivavikConfig(bad, 16)


def test_registry():
    from poptransformer_b200 import registry
    assert registry.architecture({"architecture": "Pivavik"}) == "Pivavik" and registry.dtypes({"architecture": "Pivavik"}) == ("bfloat16", "float32")


def test_oracle_rotation():
    """A pair turns like a complex number, and the score of two rotated vectors depends on their distance only."""
    r = np.random.default_rng(0)
    x = r.standard_normal((7, 2, 6))
    y, f = ref.rotate(x, 50.0), 50.0 ** (-np.arange(3) / 3)
    z = (x[..., :3] + 1j * x[..., 3:]) * np.exp(1j * np.arange(7)[:, None, None] * f)
    assert np.allclose(y[..., :3], z.real) and np.allclose(y[..., 3:], z.imag)
    same = ref.rotate(np.repeat(x[:1], 9, 0), 50.0)[:, 0]
    assert np.allclose(same[5] @ same[3], same[8] @ same[6])


@pytest.mark.parametrize("window,cap", [(0, 0.0), (1, 0.0), (3, 2.0), (50, 0.5)])
def test_oracle_attention(window, cap):
    r = np.random.default_rng(1)
    q, k, v = r.standard_normal((6, 4, 3)), r.standard_normal((6, 2, 3)), r.standard_normal((6, 2, 5))
    o = ref.masked_attention(q, k, v, 0.7, window, cap)
    for i in range(6):
        for h in range(4):
            js = [j for j in range(i + 1) if not window or i - j < window]
            s = np.array([0.7 * q[i, h] @ k[j, h // 2] for j in js])
            if cap:
                s = cap * np.tanh(s / cap)
            e = np.exp(s) / np.exp(s).sum()
            assert np.allclose(o[i, h], sum(a * v[j, h // 2] for a, j in zip(e, js)))


def test_oracle_latent_attention_in_the_latents_space():
    """The same from queries taken into the latent's space and values expanded after the sum."""
    cfg = config([latent(heads=3, dim=5, rot=4, vdim=6, kv_rank=7, q_rank=8)], width=20)
    w = weights(cfg, seed=3)
    o = ref.PivavikOracle(cfg, w)
    m, p = cfg["layers"][0]["mixer"], "l0.mix."
    h = np.random.default_rng(2).standard_normal((9, 20))
    cq = ref.rms(h @ w[p + "dq"].T, 1e-5) * w[p + "dq.norm"]
    q = (cq @ w[p + "uq"].T).reshape(9, 3, 9)
    down = h @ w[p + "dkv"].T
    c, kr = ref.rms(down[:, :7], 1e-5) * w[p + "dkv.norm"], ref.rotate(down[:, None, 7:], 1e3)[:, 0]
    qr, out = ref.rotate(q[..., 5:], 1e3), np.zeros((9, 3, 6))
    for head in range(3):
        qc = q[:, head, :5] @ w[p + "uk"][head * 5:head * 5 + 5]
        s = np.where(np.tril(np.ones((9, 9), bool)), (qc @ c.T + qr[:, head] @ kr.T) * m["scale"], -np.inf)
        e = np.exp(s - s.max(1, keepdims=True))
        out[:, head] = e / e.sum(1, keepdims=True) @ c @ w[p + "uv"][head * 6:head * 6 + 6].T / (1 + np.exp(-h @ w[p + "g"][head]))[:, None]
    assert np.allclose(o.latent_attention(p, m, h), out.reshape(9, -1) @ w[p + "o"].T)


def test_oracle_units():
    assert np.allclose(ref.silu(np.array([0.0, 2.0, -800.0])), [0, 2 / (1 + np.exp(-2.0)), 0]) and abs(ref.gelu_tanh(1.0) - 0.841192) < 1e-6
    assert np.allclose(ref.cap(np.array([1e-3, 50.0]), 5.0), [1e-3, 5.0], rtol=1e-4) and ref.cap(3.0, None) == 3.0
    idx, s = ref.choose(np.array([[1.0, 3.0, 3.0, 0.0]]), 3)
    assert idx.tolist() == [[1, 2, 0]] and np.allclose(s, 1 / (1 + np.exp([[-3.0, -3.0, -1.0]])))
    cfg = config([attention(mlp=moe(4, 2, 5))], width=20)
    w = weights(cfg, seed=5)
    h = np.random.default_rng(3).standard_normal((1, 20))
    z = (h @ w["l0.mlp.router"].T)[0]
    want = 0
    for e in np.argsort(-z)[:2]:
        x = h[0] / (1 + np.exp(-z[e]))
        want = want + w[f"l0.mlp.e{e}.down"] @ (ref.silu(w[f"l0.mlp.e{e}.gate"] @ x) * (w[f"l0.mlp.e{e}.up"] @ x))
    assert np.allclose(ref.PivavikOracle(cfg, w).experts("l0.mlp.", cfg["layers"][0]["mlp"], h)[0], want)


def test_test_models_have_no_close_choice():
    """No sublayer writes the dimensions that the routers read, so every choice depends on the token alone, with a gap."""
    for cfg in CONFIGS.values():
        w = weights(cfg, seed=11)
        assert gaps(cfg, w).min() > 0.03
        orc, tokens, sums = ref.PivavikOracle(cfg, w), np.arange(40), []
        orc.forward(tokens, sums)
        x0 = ref.zero_centred_norm(orc.w["embed"][tokens], orc.w["embed.norm"], cfg["norm"]["eps"])
        assert all(np.allclose(x[:, :CODE], x0[:, :CODE]) for x in sums)
        for i, z in router_order(cfg, w).items():
            assert not w[f"l{i}.mlp.router"][:, CODE:].any() and z.shape == (cfg["vocab"], cfg["layers"][i]["mlp"]["router"]["experts"])
