"""Small Sabisun configurations and random weights for the tests."""
import numpy as np

from seq_util import bf16, tensors


def attn(heads=4, kv_heads=2, dim=32, vdim=32, scale=None, size=None, keep_first=0, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": dim ** -0.5 if scale is None else scale}
    if size is not None:
        m["mask"] = {"size": size, "keep_first": keep_first}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def mamba(heads=4, vdim=16, state=24, groups=2, conv=4, norm_groups=1):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}


def config(mixers, width=96, vocab=160, ff=128, streams=2, eps=1e-5, mult=0.9, logit_scale=0.5):
    """mixers: attn() / mamba() entries; ff: one size, or a list with None for layers without a feed-forward."""
    ffs = ff if isinstance(ff, list) else [ff] * len(mixers)
    layers = [{"type": "attention" if "kv_heads" in m else "mamba2", "mixer": m, "mlp": None if f is None else {"ff": f, "kind": "dense"}}
              for m, f in zip(mixers, ffs)]
    return {"architecture": "Sabisun", "layers": layers, "vocab": vocab, "width": width, "streams": streams, "norm": {"eps": eps}, "residual_mult": mult,
            "logit_scale": logit_scale}


def weights(cfg, seed=0, sinks=True):
    r = np.random.default_rng(seed)
    W, S = cfg["width"], cfg["streams"]
    w = {"embed": r.standard_normal((cfg["vocab"], W)), "final.norm": 1 + 0.2 * r.standard_normal(W)}
    lin = lambda o, i: r.standard_normal((o, i)) * i ** -0.5
    for i, lay in enumerate(cfg["layers"]):
        p, m = f"l{i}.", lay["mixer"]
        for q in ("1", "2") if lay["mlp"] else ("1",):
            w[p + "norm" + q] = 1 + 0.2 * r.standard_normal(W)
            w[p + f"hc{q}.in"] = 1.0 / S + 0.3 * r.standard_normal(S)
            w[p + f"hc{q}.out"] = 1 + 0.3 * r.standard_normal(S)
            w[p + f"hc{q}.mix"] = np.eye(S) * 0.8 + 0.2 * r.standard_normal((S, S))
        if lay["type"] == "attention":
            w[p + "mix.q"] = 2 * lin(m["heads"] * m["dim"], W)
            if "kv_from" not in m:
                w[p + "mix.k"], w[p + "mix.v"] = 2 * lin(m["kv_heads"] * m["dim"], W), lin(m["kv_heads"] * m["vdim"], W)
            if sinks:
                w[p + "mix.sink"] = 2 * r.standard_normal(m["heads"])
            w[p + "mix.o"] = 2 * lin(W, m["heads"] * m["vdim"])
        else:
            inner, gn = m["heads"] * m["vdim"], m["groups"] * m["state"]
            w[p + "mix.in"] = lin(2 * inner + 2 * gn + m["heads"], W)
            w[p + "mix.conv"], w[p + "mix.conv.b"] = r.standard_normal((inner + 2 * gn, m["conv"])) * 0.6, 0.2 * r.standard_normal(inner + 2 * gn)
            w[p + "mix.dt_bias"], w[p + "mix.A_log"] = r.uniform(-4, 0.5, m["heads"]), r.uniform(-1.5, 2.0, m["heads"])
            w[p + "mix.D"], w[p + "mix.norm"] = 1 + 0.2 * r.standard_normal(m["heads"]), 1 + 0.2 * r.standard_normal(inner)
            w[p + "mix.o"] = lin(W, inner)
        if lay["mlp"]:
            f = lay["mlp"]["ff"]
            w[p + "mlp.up"], w[p + "mlp.down"] = lin(f, W), lin(W, f)
    return {k: bf16(v) for k, v in w.items()}


def decoder(cfg, w, batch, max_len, dtype="float32", **kw):
    from poptransformer_b200 import registry
    return registry.build_decoder(cfg, tensors(w), batch, max_len, dtype, **kw)


# configurations that differ in every size, the order of the layers, and the optional parts
CONFIGS = {
    "mixed": config([mamba(), attn(size=24, keep_first=5), mamba(heads=6, vdim=8, state=16, groups=3, conv=3, norm_groups=4), attn(heads=8, size=24, keep_first=5,
                     kv_from=1)], streams=2),
    "attention-first": config([attn(heads=6, kv_heads=3, dim=16, vdim=24, size=10, keep_first=0), mamba(heads=2, vdim=40, state=72, groups=1, conv=2, norm_groups=2),
                               attn(heads=3, kv_heads=3, dim=16, vdim=24, size=33, keep_first=70, kv_from=0)], width=72, vocab=101, ff=[40, None, 88], streams=4, mult=1.3),
    "one-stream": config([attn(heads=5, kv_heads=1, dim=64, vdim=128), mamba(heads=3, vdim=33, state=19, groups=3, conv=5, norm_groups=3)], width=50, vocab=77, ff=36,
                         streams=1, eps=1e-3, logit_scale=2.0),
    "wide-heads": config([mamba(heads=4, vdim=64, state=128, groups=4, conv=4, norm_groups=4), attn(heads=16, kv_heads=1, dim=128, vdim=64, size=130, keep_first=66),
                          mamba(heads=2, vdim=16, state=256, groups=2, conv=1, norm_groups=1)], width=128, vocab=256, ff=192, streams=5),
}
