"""Small Puputar configurations and random weights for the tests."""
import numpy as np

from oracle import puputar_np as ref
from seq_util import bf16, tensors


def latent(kind="latent_attention", heads=3, dim=24, rot=16, vdim=40, kv_rank=56, q_rank=32, base=1e3, scale=None, kv_from=None, mlp=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "rot": {"base": base, "dims": rot},
         "scale": 2.0 * (dim + rot) ** -0.5 if scale is None else scale}
    return {"type": kind, "mlp": mlp, "mixer": m if kv_from is None else dict(m, kv_from=kv_from)}


def latent2(**kw):
    return latent("latent_attention_2", **kw)


def dense(ff=72):
    return {"kind": "dense", "ff": ff}


def moe(experts=7, identity=1, count=2, keep=1, top=2, ff=40):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "identity": identity, "groups": {"count": count, "keep": keep}, "top": top}}


def config(layers, width=96, groups=4, vocab=150, eps=1e-5):
    return {"architecture": "Puputar", "layers": layers, "norm": {"eps": eps, "groups": groups}, "vocab": vocab, "width": width}


def code_of(cfg):
    """Leading dimensions of the residual stream whose direction no sublayer changes (identity experts, which add to them, scale them): the routers of the test models read only these, and every token's
    values there are drawn until no choice is a close call that rounding could turn.  They are the first group of the norm (a router then
    sees the same at every position) or, with one group, a few (its logits then vary by a factor, and there are no corrections)."""
    return cfg["width"] // cfg["norm"]["groups"] if cfg["norm"]["groups"] > 1 else 8


def router_inputs(cfg, w):
    """Per layer with experts: logits [vocab, experts]; with one group of the norm up to a positive factor per row."""
    n, eps = code_of(cfg), cfg["norm"]["eps"]
    code = ref.rms(w["embed"][:, :n].astype(np.float64), eps) * w["embed.norm"][:n]
    return {i: ref.rms(code, eps) * w[f"l{i}.norm2"][:n] @ w[f"l{i}.mlp.router"][:, :n].T for i, lay in enumerate(cfg["layers"]) if lay["mlp"] and lay["mlp"]["kind"] == "moe"}


def gaps(cfg, w):
    """[vocab]: the smallest gap between what is chosen and what is left out, of groups and of experts, relative to the closest that the
    scores of the test models may come (so 1 is enough)."""
    out = np.full(cfg["vocab"], np.inf)
    for i, z in router_inputs(cfg, w).items():
        r = cfg["layers"][i]["mlp"]["router"]
        count, keep = r["groups"]["count"], r["groups"]["keep"]
        if cfg["norm"]["groups"] > 1:
            _, c = ref.choice_scores(z, w[f"l{i}.mlp.correction"], 1, 1)
            unit = 0.02 / z.shape[1] ** 0.5
        else:
            c, unit = z, 0.03 * np.abs(z).max(1)
        order = lambda a: np.sort(a, 1)[:, ::-1]
        per = c.reshape(len(c), count, -1)
        best = order(per.max(-1))
        if keep < count:
            out = np.minimum(out, (best[:, keep - 1] - best[:, keep]) / unit)
        kept = np.argsort(-per.max(-1), axis=1)[:, :keep]
        left = order(np.take_along_axis(per, kept[:, :, None], 1).reshape(len(c), -1))
        if r["top"] < left.shape[1]:
            out = np.minimum(out, (left[:, r["top"] - 1] - left[:, r["top"]]) / unit)
    return out


def weights(cfg, seed=0):
    r = np.random.default_rng(seed)
    W, V, code = cfg["width"], cfg["vocab"], code_of(cfg)
    lin = lambda o, i, s=1.0: s * r.standard_normal((o, i)) * i ** -0.5
    vec = lambda n, mean=1.0: mean + 0.2 * r.standard_normal(n)

    def out(i, s=1.0):
        """Rows of an output projection: the code dimensions are never written."""
        m = lin(W, i, s)
        m[:code] = 0.0
        return m

    w = {"embed": 0.5 * r.standard_normal((V, W)), "embed.norm": vec(W), "final.norm": vec(W), "head": lin(V, W)}
    for i, lay in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", lay["mixer"], lay["mlp"]
        M, H = p + "mix.", m["heads"]
        w[p + "norm1"], w[p + "shift"] = vec(W), r.uniform(-0.3, 1.0, W)
        w[M + "dq"], w[M + "dq.norm"] = lin(m["q_rank"], W), vec(m["q_rank"])
        w[M + "uq"] = lin(H * (m["dim"] + m["rot_dim"]), m["q_rank"])
        if m.get("kv_from") is None:
            w[M + "dkv"], w[M + "dkv.norm"] = lin(m["kv_rank"] + m["rot_dim"], W), vec(m["kv_rank"])
        w[M + "uk"], w[M + "uv"] = lin(H * m["dim"], m["kv_rank"]), lin(H * m["vdim"], m["kv_rank"])
        w[M + "g"] = lin(H if lay["type"] == "latent_attention" else H * m["vdim"], W)
        w[M + "o"] = out(H * m["vdim"])
        Q = p + "mlp."
        if mlp:
            w[p + "norm2"] = vec(W)
        if mlp and mlp["kind"] == "dense":
            w[Q + "up"], w[Q + "up.b"] = lin(mlp["ff"], W), 0.3 * r.standard_normal(mlp["ff"])
            w[Q + "down"], w[Q + "down.b"] = out(mlp["ff"]), 0.3 * r.standard_normal(W)
            w[Q + "down.b"][:code] = 0.0
            w[Q + "act"] = r.standard_normal(2)
        elif mlp:
            n, f = mlp["router"]["experts"] + mlp["router"]["identity"], mlp["expert"]["ff"]
            w[Q + "router"] = np.zeros((n, W))
            w[p + "norm2"][:code] = 1.0
            w[Q + "router"][:, :code] = 2.0 * lin(n, code)
            w[Q + "correction"] = 0.3 * r.standard_normal(n) if cfg["norm"]["groups"] > 1 else np.zeros(n)
            for e in range(mlp["router"]["experts"]):
                w[Q + f"e{e}.up"], w[Q + f"e{e}.down"] = lin(f, W, 1.5), out(f, 1.5)
    w = {k: bf16(v) for k, v in w.items()}
    for _ in range(2000):
        close = np.nonzero(gaps(cfg, w) < 1.0)[0]
        if not len(close):
            break
        w["embed"][close, :code] = bf16(r.standard_normal((len(close), code)))
    return w


def decoder(cfg, w, batch, max_len, dtype="float32", **kw):
    from poptransformer_b200 import registry
    return registry.build_decoder(cfg, tensors(w), batch, max_len, dtype, **kw)


# configurations that differ in every size, in what the layers have, and in values that could be taken for granted
CONFIGS = {
    "mixed": config([latent2(mlp=moe()), latent(heads=5, dim=16, rot=32, vdim=8, kv_rank=72, q_rank=24, base=50.0, mlp=dense()), latent2(heads=2, dim=40, vdim=24, q_rank=48, kv_from=0, mlp=dense(40)),
                     latent(kv_from=0, mlp=moe(10, 2, 4, 2, 3, 72)), latent2(heads=7, dim=8, vdim=16, base=20.0)]),
    "odd-sizes": config([latent(heads=3, dim=13, rot=6, vdim=11, kv_rank=21, q_rank=17, mlp=moe(5, 1, 3, 2, 3, 7)), latent2(heads=5, dim=9, rot=2, vdim=3, kv_rank=30, q_rank=7, mlp=dense(13)),
                         latent2(heads=2, dim=5, rot=6, vdim=13, kv_rank=21, q_rank=9, kv_from=0, mlp=moe(3, 0, 1, 1, 3, 13))], width=54, groups=6, vocab=77, eps=1e-3),
    "wide-heads": config([latent2(heads=20, dim=128, rot=64, vdim=128, kv_rank=512, q_rank=96, mlp=moe(30, 3, 3, 2, 4, 64)), latent(heads=17, dim=64, rot=8, vdim=64, kv_rank=200, q_rank=64, mlp=dense(192)),
                          latent2(heads=18, dim=96, rot=64, vdim=104, kv_rank=512, q_rank=128, kv_from=0, mlp=moe(4, 4, 8, 8, 5, 192))], width=128, groups=2, vocab=256),
    "one-group": config([latent(heads=1, dim=8, rot=48, vdim=72, kv_rank=136, q_rank=136, mlp=moe(1, 3, 1, 1, 1, 24)), latent(mlp=moe(4, 0, 2, 1, 2, 24)), latent2(mlp=dense(8)),
                         latent2(heads=4, kv_from=1)], width=72, groups=1),
}
