"""Host side of the Puputar decoder, without a GPU: configuration, registry, and the oracle's own consistency (its mechanisms against a
second formulation)."""
import json

import numpy as np
import pytest

from oracle import puputar_np as ref
from puputar_util import CONFIGS, code_of, config, dense, gaps, latent, latent2, moe, weights


def test_configuration_reads_every_layer():
    from poptransformer_b200.puputar import PuputarConfig
    c = PuputarConfig(CONFIGS["mixed"], 99)
    assert (c.max_len, c.width, c.vocab, c.eps, c.groups) == (99, 96, 150, 1e-5, 4)
    assert [x.kind[-2:] for x in c.layers] == ["_2", "on", "_2", "on", "_2"]
    assert [(x.heads, x.dim, x.vdim) for x in c.layers] == [(3, 24, 40), (5, 16, 8), (2, 40, 24), (3, 24, 40), (7, 8, 16)]
    assert [(x.q_rank, x.rank, x.rot_dim, x.base) for x in c.layers] == [(32, 56, 16, 1e3), (24, 72, 32, 50.0), (48, 56, 16, 1e3), (32, 56, 16, 1e3), (32, 56, 16, 20.0)]
    assert [x.kv_from for x in c.layers] == [None, None, 0, 0, None] and [x.ff for x in c.layers] == [0, 72, 40, 0, 0]
    assert [x.moe and (x.moe.experts, x.moe.identity, x.moe.groups, x.moe.keep, x.moe.top, x.moe.ff) for x in c.layers] == [(7, 1, 2, 1, 2, 40), None, None, (10, 2, 4, 2, 3, 72), None]


def test_router_without_groups_or_identity_experts():
    from poptransformer_b200.puputar import PuputarConfig
    lay = latent(mlp=moe())
    for k in ("groups", "identity"):
        del lay["mlp"]["router"][k]
    m = PuputarConfig(config([lay]), 9).layers[0].moe
    assert (m.identity, m.groups, m.keep) == (0, 1, 1)


def edited(lay, **kw):
    lay = json.loads(json.dumps(lay))
    for path, v in kw.items():
        d = lay
        *way, last = path.split("__")
        for k in way:
            d = d[k]
        d[last] = v
    return config([latent(), lay])


@pytest.mark.parametrize("bad,match", [
    (config([latent()], width=90), "groups"), (config([latent(rot=7)]), "rotated"), (edited(latent(), mixer__rot__dims=8), "rotated"), (edited(latent(), type="attention"), "unknown mixer"),
    (edited(latent(mlp=dense()), mlp__kind="sparse"), "unknown feed-forward"), (config([latent(mlp=moe(count=3))]), "groups of 8"), (config([latent(mlp=moe(keep=3))]), "groups"),
    (config([latent(mlp=moe(top=5))]), "the 4 experts"), (config([latent(mlp=moe(experts=0, identity=2))]), "groups"), (config([latent(kv_from=0)]), "caches nothing"),
    (config([latent(), latent2(kv_from=0), latent2(kv_from=1)]), "caches nothing"), (config([latent(), latent2(kv_from=0, kv_rank=64)]), "another shape"),
    (config([latent(), latent2(kv_from=0, base=2e3)]), "rotation"), (config([latent(), latent2(kv_from=0, rot=8)]), "another shape")])
def test_configuration_refuses(bad, match):
    from poptransformer_b200 import PtError
    from poptransformer_b200.puputar import PuputarConfig
    with pytest.raises(PtError, match=match):
        PuputarConfig(bad, 16)


def test_registry():
    from poptransformer_b200 import registry
    assert registry.architecture({"architecture": "Puputar"}) == "Puputar" and registry.dtypes({"architecture": "Puputar"}) == ("bfloat16", "float32")


def test_random_weights_have_every_tensor():
    """The weights that benchmarks draw carry the names and shapes that the tests' models have."""
    from poptransformer_b200 import synth
    for cfg in CONFIGS.values():
        sd = synth.puputar_state_dict(cfg)
        assert {k: tuple(v.shape) for k, v in sd.items()} == {k: v.shape for k, v in weights(cfg).items()}


# ------------------------------------------------------------------------------------------ the oracle
def test_oracle_group_norm():
    r = np.random.default_rng(0)
    x, w = r.standard_normal((3, 12)), r.standard_normal(12)
    y = ref.group_norm(x, w, 0.1, 3)
    for t in range(3):
        for g in range(3):
            part = x[t, 4 * g:4 * g + 4]
            assert np.allclose(y[t, 4 * g:4 * g + 4], part / np.sqrt((part ** 2).sum() / 4 + 0.1) * w[4 * g:4 * g + 4])
    assert np.allclose(ref.group_norm(x, w, 0.1, 1), ref.rms(x, 0.1) * w)


def test_oracle_token_shift():
    h, mix = np.array([[1.0, 2.0, 3.0], [4.0, 5.0, 6.0], [7.0, 8.0, 9.0]]), np.array([0.0, 1.0, 0.25])
    assert np.allclose(ref.token_shift(h, mix), [[1, 0, 2.25], [4, 2, 5.25], [7, 5, 8.25]])


def test_oracle_rotation():
    """A pair of neighbours turns like a complex number, and the score of two rotated vectors depends on their distance only."""
    r = np.random.default_rng(1)
    x = r.standard_normal((7, 2, 6))
    y, f = ref.rotate_pairs(x, 50.0), 50.0 ** (-np.arange(3) / 3)
    z = (x[..., 0::2] + 1j * x[..., 1::2]) * np.exp(1j * np.arange(7)[:, None, None] * f)
    assert np.allclose(y[..., 0::2], z.real) and np.allclose(y[..., 1::2], z.imag)
    same = ref.rotate_pairs(np.repeat(x[:1], 9, 0), 50.0)[:, 0]
    assert np.allclose(same[5] @ same[3], same[8] @ same[6])


def test_oracle_units():
    p, q = 0.3, -0.7
    z = np.array([-800.0, -2.0, -1e-4, 0.0, 1e-4, 3.0])
    want = [(np.log1p(np.exp(p)) * v * v if v > 0 else (0.5 + np.log1p(np.exp(q))) * (np.exp(v) - 1 - v)) + v / 2 for v in z]
    assert np.allclose(ref.xielu(z, p, q), want, atol=1e-15) and np.allclose(ref.relu2(np.array([-3.0, 0.5])), [0, 0.25])


def test_oracle_choice():
    z, corr = np.array([[0.0, 1.0, 2.0, 3.0, -1.0, 0.5]]), np.array([0.0, 0.9, 0.0, -1.0, -0.5, 0.0])
    s = np.exp(z[0]) / np.exp(z[0]).sum()
    # groups (0, 1), (2, 3), (4, 5): the first leads by its correction, then the second; of these, 1 and 2 and 0
    idx, wt = ref.choose(z, corr, 3, 3, 2)
    assert idx.tolist() == [[1, 2, 0]] and np.allclose(wt, s[[1, 2, 0]] / s[[1, 2, 0]].sum())
    assert (s + corr)[3] < 0 and ref.choose(z, corr, 4, 3, 2)[0].tolist() == [[1, 2, 0, 3]]      # a negative score in the group beats one outside
    assert ref.choose(z, 0 * corr, 2, 1, 1)[0].tolist() == [[3, 2]]


def test_oracle_experts():
    cfg = config([latent(mlp=moe(3, 1, 2, 1, 2, 5))], width=20)
    w = weights(cfg, seed=5)
    h = np.random.default_rng(3).standard_normal((9, 20))
    z = h @ w["l0.mlp.router"].T
    idx, wt = ref.choose(z, w["l0.mlp.correction"], 2, 2, 1)
    want = np.zeros_like(h)
    for t in range(9):
        for e, a in zip(idx[t], wt[t]):
            want[t] += a * (h[t] if e == 3 else w[f"l0.mlp.e{e}.down"] @ np.maximum(w[f"l0.mlp.e{e}.up"] @ h[t], 0) ** 2)
    assert np.allclose(ref.PuputarOracle(cfg, w).experts("l0.mlp.", cfg["layers"][0]["mlp"], h), want)


@pytest.mark.parametrize("kind", ["latent_attention", "latent_attention_2"])
def test_oracle_latent_attention_in_the_latents_space(kind):
    """The same from queries taken into the latent's space and values expanded after the sum."""
    cfg = config([latent(kind, heads=3, dim=5, rot=4, vdim=6, kv_rank=7, q_rank=8)], width=20)
    w = weights(cfg, seed=3)
    o = ref.PuputarOracle(cfg, w)
    m, p = cfg["layers"][0]["mixer"], "l0.mix."
    h = np.random.default_rng(2).standard_normal((9, 20))
    cq = ref.rms(h @ w[p + "dq"].T, 1e-5) * w[p + "dq.norm"]
    q = (cq @ w[p + "uq"].T).reshape(9, 3, 9)
    down = h @ w[p + "dkv"].T
    c, kr = ref.rms(down[:, :7], 1e-5) * w[p + "dkv.norm"], ref.rotate_pairs(down[:, None, 7:], 1e3)[:, 0]
    qr, out = ref.rotate_pairs(q[..., 5:], 1e3), np.zeros((9, 3, 6))
    gate = 1 / (1 + np.exp(-h @ w[p + "g"].T))
    for head in range(3):
        qc = q[:, head, :5] @ w[p + "uk"][head * 5:head * 5 + 5]
        s = np.where(np.tril(np.ones((9, 9), bool)), (qc @ c.T + qr[:, head] @ kr.T) * m["scale"], -np.inf)
        e = np.exp(s - s.max(1, keepdims=True))
        out[:, head] = e / e.sum(1, keepdims=True) @ c @ w[p + "uv"][head * 6:head * 6 + 6].T * (gate[:, head, None] if kind == "latent_attention" else gate[:, head * 6:head * 6 + 6])
    assert np.allclose(o.mixer(0, h, {}), out.reshape(9, -1) @ w[p + "o"].T)


def test_oracle_reads_another_layers_latents():
    cfg = config([latent2(), latent2(heads=2, vdim=8, kv_from=0)])
    w = weights(cfg, seed=4)
    h = np.random.default_rng(4).standard_normal((2, 6, 96))
    caches = {}
    o = ref.PuputarOracle(cfg, w)
    o.mixer(0, h[0], caches)
    got = o.mixer(1, h[1], caches)
    twin = {**w, "l1.mix.dkv": w["l0.mix.dkv"], "l1.mix.dkv.norm": w["l0.mix.dkv.norm"]}     # a layer that is shown the same latents as its own
    own = ref.PuputarOracle(config([latent2(), latent2(heads=2, vdim=8)]), twin)
    assert not np.allclose(got, own.mixer(1, h[1], {}))
    p, m = "l1.mix.", cfg["layers"][1]["mixer"]
    heads = own.latent_attention(p, m, h[1], own.latents("l0.mix.", m, h[0])).reshape(6, -1)
    assert np.allclose(got, heads * ref.sigmoid(h[1] @ w[p + "g"].T) @ w[p + "o"].T) and list(caches) == [0]


def test_test_models_have_no_close_choice():
    """No sublayer turns the dimensions that the routers read, so every choice depends on the token alone, with a gap."""
    for cfg in CONFIGS.values():
        w = weights(cfg, seed=11)
        assert gaps(cfg, w).min() > 1.0
        orc, tokens, sums, n = ref.PuputarOracle(cfg, w), np.arange(40), [], code_of(cfg)
        orc.forward(tokens, sums)
        x0 = orc.norm("embed.norm", orc.w["embed"][tokens])
        assert all(np.allclose(ref.rms(x[:, :n], 0), ref.rms(x0[:, :n], 0)) for x in sums)
        for i, lay in enumerate(cfg["layers"]):
            if lay["mlp"] and lay["mlp"]["kind"] == "moe":
                assert not w[f"l{i}.mlp.router"][:, n:].any() and (cfg["norm"]["groups"] > 1 or not w[f"l{i}.mlp.correction"].any())
