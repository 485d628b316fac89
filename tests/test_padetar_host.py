"""Host side of the Padetar decoder, without a GPU: configuration, registry, frequencies, and the oracle's own consistency (its
mechanisms against a second formulation)."""
import json

import numpy as np
import pytest
import torch

from oracle import padetar_np as ref
from padetar_util import CODE, CONFIGS, config, layer, weights


def test_configuration_reads_every_layer():
    from poptransformer_b200.padetar import PadetarConfig
    c = PadetarConfig(CONFIGS["mixed"], 99)
    assert (c.max_len, c.width, c.vocab, c.side, c.eps) == (99, 96, 150, 24, 1e-5)
    assert [(x.left.heads, x.left.rot_dims, x.right.cap, x.left_scale, x.right_scale) for x in c.layers] == [(4, 32, 10.0, 0.7, 0.9), (6, 24, 4.0, 1.0, 0.6), (4, 32, 10.0, 0.7, 0.9)]
    assert [x.moe and (x.moe.experts, x.moe.top, x.moe.ff, x.moe.limit, x.moe.shared_ff, x.moe.shared_limit) for x in c.layers] == [
        (6, 2, 40, 0.9, 56, 1.3), (9, 3, 72, 0.5, 24, 2.0), None]
    assert c.layers[0].left.rot == (32, 1e4, (8.0, 1.0, 4.0, 64.0)) and c.layers[2].left.rot == (32, 1e4, None)
    assert PadetarConfig(CONFIGS["no-side"], 9).side == 0


def edited(**kw):
    c = json.loads(json.dumps(config([layer()])))
    for path, v in kw.items():
        d = c["layers"][0]
        *way, last = path.split("__")
        for k in way:
            d = d[k]
        d[last] = v
    return c


@pytest.mark.parametrize("bad,match", [
    (config([layer(heads=3, kv_heads=2)]), "heads"), (config([layer(rot=34)]), "rotated"), (config([layer(rot=7)]), "rotated"), (config([layer(top=7)]), "experts"),
    (edited(type="attention"), "unknown mixer"), (edited(mlp__kind="dense"), "unknown feed-forward"), (edited(mixer__left__vdim=16), "values are keys")])
def test_configuration_refuses(bad, match):
    from poptransformer_b200 import PtError
    from poptransformer_b200.padetar import PadetarConfig
    with pytest.raises(PtError, match=match):
        PadetarConfig(bad, 16)


def test_registry():
    from poptransformer_b200 import registry
    assert registry.architecture({"architecture": "Padetar"}) == "Padetar" and registry.dtypes({"architecture": "Padetar"}) == ("bfloat16", "float32")


@pytest.mark.parametrize("dims,base,scaling", [(56, 3e5, (5.0, 1.5, 6.0, 200)), (64, 1e4, (8.0, 2.0, 32.0, 512)), (16, 100.0, None), (2, 1e4, (3.0, 1.0, 2.0, 4))])
def test_frequencies(dims, base, scaling):
    from poptransformer_b200.padetar import rope_frequencies
    sc = dict(zip(("factor", "low", "high", "original"), scaling)) if scaling else None
    got, want = rope_frequencies(dims, base, sc), ref.frequencies(dims, base, sc)
    assert np.allclose(got, want, rtol=1e-14)
    plain = ref.frequencies(dims, base)
    if scaling and dims > 2:      # all three bands occur
        turns = scaling[3] * plain / (2 * np.pi)
        assert (want[turns > scaling[2]] == plain[turns > scaling[2]]).all() and np.allclose(want[turns < scaling[1]] * scaling[0], plain[turns < scaling[1]])
        mid = (turns > scaling[1]) & (turns < scaling[2])
        assert mid.any() and ((want < plain) & (want > plain / scaling[0]))[mid].all()


def test_gated_rows():
    from poptransformer_b200 import ops
    g, u = torch.arange(10.0)[:, None] + torch.zeros(10, 3), 100 + torch.arange(10.0)[:, None] + torch.zeros(10, 3)
    rows = ops.glu_rows(g, u, 16)[:, 0].tolist()
    assert rows == [*range(8), *range(100, 108), 8, 9, 0, 0, 0, 0, 0, 0, 108, 109, 0, 0, 0, 0, 0, 0]


def test_weight_look_ups_are_checked():
    from poptransformer_b200 import PtError
    from poptransformer_b200.sequences import Weights
    w = Weights({"a": torch.zeros(2, 3)}, "cpu", torch.float32)
    assert w.mat("a", (2, 3)).shape == (2, 3) and "a" in w and "b" not in w
    with pytest.raises(PtError, match="expected"):
        w.f32("a", (3, 2))
    with pytest.raises(PtError, match="no such tensor"):
        w.f32("b", (3,))


def test_oracle_memory_against_the_unrolled_sum():
    """o_t = sum_s exp(F_t - F_s + i_s) (k_s . q_t) v_s / (max(|the same sum with 1 for v|, 1) + 1e-6 exp(m_t)), F the running sum of f,
    m_t the largest exponent so far (at least F_t)."""
    r = np.random.default_rng(0)
    T, H, D, V = 12, 2, 4, 3
    q, k, v = r.standard_normal((T, H, D)), r.standard_normal((T, H, D)), r.standard_normal((T, H, V))
    li, lf = ref.memory_gates(r.uniform(-9, 9, (T, H)), r.uniform(-6, 9, (T, H)), 7.0)
    assert (np.abs(li) < 7).all() and (lf < 0).all()
    F = np.cumsum(lf, 0)
    want = np.zeros_like(v)
    for h in range(H):
        for t in range(T):
            e = F[t, h] - F[:t + 1, h] + li[:t + 1, h]
            m = max(F[t, h], e.max())
            c = np.exp(e) * (k[:t + 1, h] @ q[t, h])
            want[t, h] = c @ v[:t + 1, h] / (max(abs(c.sum()), 1.0) + 1e-6 * np.exp(m))
    assert np.allclose(ref.matrix_memory(q, k, v, li, lf), want)


def test_oracle_rotation_and_attention():
    r = np.random.default_rng(1)
    x = r.standard_normal((7, 2, 6))
    f = ref.frequencies(4, 50.0)
    y = ref.rotate(x, f)
    z = (x[..., :2] + 1j * x[..., 2:4]) * np.exp(1j * np.arange(7)[:, None, None] * f)
    assert np.allclose(y[..., :2], z.real) and np.allclose(y[..., 2:4], z.imag) and np.array_equal(y[..., 4:], x[..., 4:])
    q, k = r.standard_normal((5, 4, 3)), r.standard_normal((5, 2, 3))
    o = ref.causal_attention(q, k, k, 0.7).reshape(5, 4, 3)
    e = np.exp(0.7 * k[:4, 1] @ q[3, 2])
    assert np.allclose(o[3, 2], e @ k[:4, 1] / e.sum()) and np.allclose(o[0, 3], k[0, 1])


def test_oracle_choice_and_units():
    z = np.array([[1.0, 3.0, 3.0, 0.0]])
    idx, w = ref.choose(z, 3)
    assert idx.tolist() == [[1, 2, 0]] and np.allclose(w, [[1, 1, np.exp(-2.0)] / (2 + np.exp(-2.0))])
    assert np.allclose(ref.clamped_glu(np.array([9.0, -9.0]), np.array([-9.0, 9.0]), 2.0), [2 / (1 + np.exp(-3.404)) * -1, -9 / (1 + np.exp(1.702 * 9)) * 3])
    assert abs(ref.gelu_tanh(1.0) - 0.841192) < 1e-6


def test_test_models_have_no_close_choice():
    """No sublayer writes the dimensions that the routers read, so every choice depends on the token alone, with a gap."""
    for cfg in CONFIGS.values():
        w = weights(cfg, seed=11)
        for i, lay in enumerate(cfg["layers"]):
            if not lay["mlp"]:
                continue
            z = np.sort(w["embed"] @ w[f"l{i}.mlp.router"].T + w[f"l{i}.mlp.router.b"], 1)[:, ::-1]
            top = lay["mlp"]["router"]["top"]
            assert not w[f"l{i}.mlp.router"][:, CODE:].any() and not w[f"l{i}.norm1"][:CODE].any() and not w[f"l{i}.norm2"][:CODE].any()
            assert top == z.shape[1] or (z[:, top - 1] - z[:, top]).min() > 1e-4
