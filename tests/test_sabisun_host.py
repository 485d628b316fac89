"""Host side of the Sabisun decoder, without a GPU: configuration, registry, checkpoint folder, slots and pages, and the oracle's own
consistency (its mechanisms against a second formulation)."""
import json
import os
import subprocess

import numpy as np
import pytest
import torch

from oracle import sabisun_np as ref
from sabisun_util import CONFIGS, attn, config, mamba, weights
from seq_util import write_model

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def test_configuration_reads_every_layer():
    from poptransformer_b200.sabisun import SabisunConfig
    c = SabisunConfig(CONFIGS["attention-first"], 99)
    assert (c.max_len, c.width, c.streams, c.vocab, c.residual_mult) == (99, 72, 4, 101, 1.3)
    assert [lay.mixer.kind for lay in c.layers] == ["attention", "mamba2", "attention"] and [lay.ff for lay in c.layers] == [40, 0, 88]
    assert (c.layers[2].mixer.kv_from, c.layers[2].mixer.window, c.layers[2].mixer.keep_first) == (0, 33, 70)
    assert c.layers[1].mixer.proj == 2 * 80 + 2 * 72 + 2
    assert SabisunConfig(CONFIGS["one-stream"], 9).layers[0].mixer.window == 0


@pytest.mark.parametrize("bad,match", [
    (config([attn(heads=3, kv_heads=2)]), "heads"), (config([attn(), attn(kv_from=1)]), "kv_from"), (config([mamba(), attn(kv_from=0)]), "kv_from"),
    (config([attn(dim=16), attn(kv_from=0)]), "kv_from"), (config([mamba(heads=3, groups=2)]), "groups"), (config([mamba(norm_groups=5)]), "norm")])
def test_configuration_refuses(bad, match):
    from poptransformer_b200 import PtError
    from poptransformer_b200.sabisun import SabisunConfig
    with pytest.raises(PtError, match=match):
        SabisunConfig(bad, 16)


def test_registry():
    from poptransformer_b200 import PtError, registry
    assert registry.architecture({"architecture": "Sabisun"}) == "Sabisun"
    assert registry.architecture({"architectures": ["LlamaForCausalLM"]}) == "LlamaForCausalLM"
    assert registry.dtypes({"architecture": "Sabisun"}) == ("bfloat16", "float32")
    with pytest.raises(PtError, match="unknown architecture"):
        registry.architecture({"architectures": ["Other"]})
    with pytest.raises(registry.UnsupportedDtype):
        registry.build_decoder({"architectures": ["GPT2LMHeadModel"]}, {}, 1, 8, "float32")


def test_trace_replay_refuses_a_type_the_model_lacks(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps({"architectures": ["LlamaForCausalLM"]}))
    (tmp_path / "model.safetensors").write_bytes((2).to_bytes(8, "little") + b"{}")
    p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "8"],
                       input="", capture_output=True, text=True, timeout=300)
    assert p.returncode == 3, p.stderr


def test_model_folder_round_trip(tmp_path):
    from poptransformer_b200 import checkpoint
    cfg = CONFIGS["mixed"]
    w = weights(cfg, seed=3)
    write_model(str(tmp_path), cfg, w)
    got, sd = checkpoint.load_model_dir(str(tmp_path))
    assert got == cfg and set(sd) == set(w)
    assert all(sd[k].dtype == torch.bfloat16 and np.array_equal(sd[k].float().numpy(), w[k]) for k in w)


def test_safetensors_types(tmp_path):
    from poptransformer_b200 import checkpoint
    a, b, c = np.arange(6, dtype="<i4").reshape(2, 3), np.array([1.5, -2.0], "<f4"), np.array(7.0, "<f8")
    blobs = [a.tobytes(), b.tobytes(), c.tobytes()]
    at = np.concatenate([[0], np.cumsum([len(x) for x in blobs])]).tolist()
    head = {n: {"dtype": d, "shape": list(t.shape), "data_offsets": at[i:i + 2]} for i, (n, d, t) in enumerate([("a", "I32", a), ("b", "F32", b), ("c", "F64", c)])}
    head["e"] = {"dtype": "F32", "shape": [0, 4], "data_offsets": [at[3], at[3]]}
    head["__metadata__"] = {"format": "pt"}
    h = json.dumps(head).encode()
    (tmp_path / "x.safetensors").write_bytes(len(h).to_bytes(8, "little") + h + b"".join(blobs))
    sd = checkpoint.load_state_dict(str(tmp_path / "x.safetensors"))
    assert np.array_equal(sd["a"].numpy(), a) and np.array_equal(sd["b"].numpy(), b) and sd["c"].item() == 7.0 and sd["e"].shape == (0, 4)


def test_slots_and_pages():
    from poptransformer_b200 import PtError
    from poptransformer_b200.cache import SequenceSlots
    s = SequenceSlots(3, 40, page_size=8, n_pages=7, device="cpu")
    a, b = s.open(), s.open()
    assert (a, b) == (0, 1) and s.extend(a, 9) == 0 and s.extend(b, 16) == 0 and s.free_pages == 3
    assert s.extend(a, 7) == 9 and s.free_pages == 3 and s.extend(a, 1) == 16 and s.free_pages == 2
    used = s.page_table[a, :3].tolist() + s.page_table[b, :2].tolist()
    assert len(set(used)) == 5 and all(0 <= p < 7 for p in used)
    c = s.open()
    with pytest.raises(PtError, match="pages"):
        s.extend(c, 17)
    assert s.length[c] == 0 and s.free_pages == 2                # a refused call takes nothing
    with pytest.raises(PtError, match="max_len"):
        s.extend(a, 24)
    with pytest.raises(PtError, match="slots"):
        s.open()
    s.close(a)
    assert s.free_pages == 5 and s.open() == a and s.extend(a, 40) == 0 and s.free_pages == 0
    s.close_all()
    assert s.free_pages == 7 and [s.open() for _ in range(3)] == [0, 1, 2]


def test_oracle_scan_against_the_unrolled_sum():
    """The recurrence equals y_t = sum_s (C_t . B_s) exp(sum of log decays in (s, t]) dt_s x_s + D x_t."""
    r = np.random.default_rng(0)
    T, H, P, G, N = 9, 4, 3, 2, 5
    x, B, C, dt = r.standard_normal((T, H, P)), r.standard_normal((T, G, N)), r.standard_normal((T, G, N)), r.uniform(0, 1, (T, H))
    A_log, D = r.standard_normal(H), r.standard_normal(H)
    cum = np.cumsum(-np.exp(A_log) * dt, 0)
    want = np.zeros_like(x)
    for h in range(H):
        g = h // 2
        for t in range(T):
            want[t, h] = D[h] * x[t, h] + sum((C[t, g] @ B[s, g]) * np.exp(cum[t, h] - cum[s, h]) * dt[s, h] * x[s, h] for s in range(t + 1))
    assert np.allclose(ref.ssm_scan(x, B, C, dt, A_log, D), want)


def test_oracle_mask_and_sink():
    m = ref.visible(12, size=3, keep_first=2)
    assert [list(np.flatnonzero(m[i])) for i in (0, 2, 4, 5, 11)] == [[0], [0, 1, 2], [0, 1, 2, 3, 4], [0, 1, 3, 4, 5], [0, 1, 9, 10, 11]]
    assert ref.visible(5).sum() == 15
    s = np.array([[0.0, 1.0, -np.inf]])
    e = np.exp([0.0, 1.0])
    assert np.allclose(ref.sink_softmax(s, None), [[*(e / e.sum()), 0]]) and np.allclose(ref.sink_softmax(s, 2.0), [[*(e / (e.sum() + np.exp(2.0))), 0]])


def test_oracle_streams_and_conv():
    r = np.random.default_rng(1)
    xs, y, mix, out = r.standard_normal((2, 1, 3)), r.standard_normal((1, 3)), np.array([[1.0, 2.0], [3.0, 4.0]]), np.array([5.0, 6.0])
    n = ref.stream_write(xs, y, mix, out, 0.5)
    assert np.allclose(n[0], xs[0] + 3 * xs[1] + 2.5 * y) and np.allclose(n[1], 2 * xs[0] + 4 * xs[1] + 3 * y)
    assert np.allclose(ref.stream_read(xs, np.array([2.0, -1.0])), 2 * xs[0] - xs[1])
    x = np.arange(1.0, 5.0)[:, None]
    assert np.allclose(ref.causal_conv(x, np.array([[10.0, 1.0]]), np.array([0.5])).ravel(), [1.5, 12.5, 23.5, 34.5])
