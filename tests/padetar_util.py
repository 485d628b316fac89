"""Small Padetar configurations and random weights for the tests."""
import numpy as np

from seq_util import bf16, tensors

CODE = 8      # leading dimensions of the residual stream that no sublayer writes: the routers of the test models read only these, so
#               that no expert choice is a close call that rounding could turn


def layer(heads=4, kv_heads=2, dim=32, rot=None, base=1e4, scaling=(8.0, 1.0, 4.0, 64), scale=None, m_heads=3, m_dim=24, m_vdim=16, cap=10.0, ls=0.7, rs=0.9, experts=6,
          top=2, ff=40, limit=0.9, shared=56, shared_limit=1.3, mlp=True):
    r = {"base": base, "dims": dim if rot is None else rot}
    if scaling:
        r["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    lay = {"type": "parallel", "mixer": {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": 2.0 * dim ** -0.5 if scale is None else scale, "rot": r},
                                         "right": {"heads": m_heads, "dim": m_dim, "vdim": m_vdim, "gate_cap": cap}, "left_scale": ls, "right_scale": rs}, "mlp": None}
    if mlp:
        lay["mlp"] = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit}}
        if shared:
            lay["mlp"]["shared"] = {"ff": shared, "limit": shared_limit}
    return lay


def config(layers, width=96, vocab=150, side=24, eps=1e-5):
    return {"architecture": "Padetar", "layers": layers, "norm": {"eps": eps}, "token_side": {"dim": side} if side else None, "vocab": vocab, "width": width}


def weights(cfg, seed=0):
    r = np.random.default_rng(seed)
    W, V = cfg["width"], cfg["vocab"]
    lin = lambda o, i, s=1.0: s * r.standard_normal((o, i)) * i ** -0.5
    vec = lambda n: 1 + 0.2 * r.standard_normal(n)
    w = {"embed": r.standard_normal((V, W)), "final.norm": vec(W), "head": lin(V, W, 2.0)}
    side = (cfg.get("token_side") or {}).get("dim", 0)
    if side:
        w["side.embed"] = r.standard_normal((V, side * len(cfg["layers"])))

    def norm(key):
        w[key] = vec(W)
        w[key][:CODE] = 0.0

    for i, lay in enumerate(cfg["layers"]):
        p, a, b, mlp = f"l{i}.", lay["mixer"]["left"], lay["mixer"]["right"], lay["mlp"]
        norm(p + "norm1")
        L, R = p + "mix.left.", p + "mix.right."
        for n, o in (("q", a["heads"] * a["dim"]), ("k", a["kv_heads"] * a["dim"])):
            w[L + n], w[L + n + ".b"], w[L + n + ".norm"] = lin(o, W), 0.3 * r.standard_normal(o), vec(a["dim"])
        w[L + "o"], w[L + "o.b"] = lin(W, a["heads"] * a["dim"]), 0.3 * r.standard_normal(W)
        H, N, P = b["heads"], b["dim"], b["vdim"]
        for n, o in (("q", H * N), ("k", H * N), ("v", H * P), ("g", H * P)):
            w[R + n] = lin(o, W)
        w[R + "o"], w[R + "norm"] = lin(W, H * P), vec(H * P)
        w[R + "i"], w[R + "i.b"], w[R + "f"], w[R + "f.b"] = lin(H, W, 2.0), r.uniform(-4, 2, H), lin(H, W), r.uniform(-1, 6, H)
        if mlp:
            norm(p + "norm2")
            M, E = p + "mlp.", mlp["router"]["experts"]
            w[M + "router"], w[M + "router.b"] = np.zeros((E, W)), 0.5 * r.standard_normal(E)
            w[M + "router"][:, :CODE] = r.standard_normal((E, CODE)) * 0.6
            for e, f in [(f"e{k}.", mlp["expert"]["ff"]) for k in range(E)] + ([("shared.", mlp["shared"]["ff"])] if mlp.get("shared") else []):
                w[M + e + "gate"], w[M + e + "up"], w[M + e + "down"] = lin(f, W), lin(f, W), lin(W, f)
        if side:
            w[p + "side.gate"], w[p + "side.proj"] = lin(side, W), lin(W, side)
            norm(p + "side.norm")
    return {k: bf16(v) for k, v in w.items()}


def decoder(cfg, w, batch, max_len, dtype="float32", **kw):
    from poptransformer_b200 import registry
    return registry.build_decoder(cfg, tensors(w), batch, max_len, dtype, **kw)


# configurations that differ in every size, in what the layers have, and in values that could be taken for granted
CONFIGS = {
    "mixed": config([layer(), layer(heads=6, kv_heads=1, dim=40, rot=24, base=500.0, m_heads=2, m_dim=64, m_vdim=40, cap=4.0, ls=1.0, rs=0.6, experts=9, top=3, ff=72,
                                    limit=0.5, shared=24, shared_limit=2.0), layer(mlp=False, scaling=None)]),
    "odd-sizes": config([layer(heads=5, kv_heads=5, dim=14, rot=6, m_heads=1, m_dim=19, m_vdim=33, experts=5, top=5, ff=13, shared=29),
                         layer(heads=3, kv_heads=1, dim=22, rot=22, m_heads=7, m_dim=5, m_vdim=3, experts=3, top=1, ff=7, shared=0)], width=50, vocab=77, side=10, eps=1e-3),
    "wide-heads": config([layer(heads=16, kv_heads=2, dim=128, rot=64, m_heads=2, m_dim=128, m_vdim=72, experts=33, top=4, ff=64, shared=128),
                          layer(heads=2, kv_heads=1, dim=64, m_heads=1, m_dim=256, m_vdim=128, experts=4, top=2, ff=192, shared=64)], width=128, vocab=256, side=64),
    "no-side": config([layer(m_dim=16, m_vdim=64, top=1, shared=0, limit=7.0), layer(dim=16, heads=4, kv_heads=4)], width=72, side=0),
}
