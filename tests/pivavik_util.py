"""Small Pivavik configurations and random weights for the tests."""
import numpy as np

from seq_util import bf16, tensors

CODE = 8      # leading dimensions of the residual stream that no sublayer writes: the routers of the test models read only these, and every
#               token's values there are drawn until no expert choice is a close call that rounding could turn


def latent(heads=4, dim=24, rot=16, vdim=32, kv_rank=48, q_rank=40, base=1e3, scale=None, mlp=None):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "rot": {"base": base, "dims": rot},
                      "scale": 2.0 * (dim + rot) ** -0.5 if scale is None else scale}}


def attention(heads=6, kv_heads=2, dim=32, vdim=24, window=40, softcap=3.0, scale=None, mlp=None):
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window}, "softcap": softcap,
                      "scale": 2.0 * dim ** -0.5 if scale is None else scale}}


def dense(ff=72):
    return {"kind": "dense", "ff": ff}


def moe(experts=6, top=2, ff=40):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}


def config(layers, width=96, vocab=150, eps=1e-5, softcap=6.0, loop=None):
    return {"architecture": "Pivavik", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width, "logit_softcap": softcap,
            "loop": dict(zip(("start", "stop", "times"), loop)) if loop else None}


def router_order(cfg, w):
    """Per layer with experts: logits [vocab, experts] up to a positive factor per row (what the norms divide by), at every pass the same."""
    code = w["embed"][:, :CODE] * (1 + w["embed.norm"][:CODE])
    return {i: (code * (1 + w[f"l{i}.norm1"][:CODE])) @ w[f"l{i}.mlp.router"][:, :CODE].T for i, lay in enumerate(cfg["layers"]) if lay["mlp"] and lay["mlp"]["kind"] == "moe"}


def gaps(cfg, w):
    """[vocab]: the smallest gap between a chosen and a left-out expert, relative to the largest logit."""
    out = np.full(cfg["vocab"], np.inf)
    for i, z in router_order(cfg, w).items():
        top = cfg["layers"][i]["mlp"]["router"]["top"]
        if top < z.shape[1]:
            s = np.sort(z, 1)[:, ::-1]
            out = np.minimum(out, (s[:, top - 1] - s[:, top]) / np.abs(z).max(1))
    return out


def weights(cfg, seed=0):
    r = np.random.default_rng(seed)
    W, V = cfg["width"], cfg["vocab"]
    lin = lambda o, i, s=1.0: s * r.standard_normal((o, i)) * i ** -0.5
    vec = lambda n, mean=0.0: mean + 0.2 * r.standard_normal(n)

    def out(i, s=1.0):
        """Rows of an output projection: the code dimensions are never written."""
        m = lin(W, i, s)
        m[:CODE] = 0.0
        return m

    w = {"embed": 0.5 * r.standard_normal((V, W)), "embed.norm": vec(W), "final.norm": vec(W)}
    loop = cfg.get("loop")
    if loop:       # the stream's code dimensions become the embedding output's again
        w["loop.in"], w["loop.step"] = out(2 * W), 0.5 * r.standard_normal((loop["times"], W))
        w["loop.in"][np.arange(CODE), W + np.arange(CODE)] = 1.0
        w["loop.step"][:, :CODE] = 0.0
    for i, lay in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", lay["mixer"], lay["mlp"]
        M, H = p + "mix.", m["heads"]
        w[p + "norm1"] = vec(W)
        if lay["type"] == "latent_attention":
            w[M + "dq"], w[M + "dq.norm"] = lin(m["q_rank"], W), vec(m["q_rank"], 1.0)
            w[M + "uq"] = lin(H * (m["dim"] + m["rot_dim"]), m["q_rank"])
            w[M + "dkv"], w[M + "dkv.norm"] = lin(m["kv_rank"] + m["rot_dim"], W), vec(m["kv_rank"], 1.0)
            w[M + "uk"], w[M + "uv"], w[M + "g"] = lin(H * m["dim"], m["kv_rank"]), lin(H * m["vdim"], m["kv_rank"]), lin(H, W)
        else:
            for n, o in (("q", H * m["dim"]), ("k", m["kv_heads"] * m["dim"]), ("v", m["kv_heads"] * m["vdim"])):
                w[M + n], w[M + n + ".b"] = lin(o, W), 0.3 * r.standard_normal(o)
            w[M + "g"] = lin(H * m["vdim"], W)
        w[M + "o"] = out(H * m["vdim"])
        Q = p + "mlp."
        if mlp and mlp["kind"] == "dense":
            for n in ("gate", "up"):
                w[Q + n], w[Q + n + ".b"] = lin(mlp["ff"], W), 0.3 * r.standard_normal(mlp["ff"])
            w[Q + "down"], w[Q + "down.b"] = out(mlp["ff"]), 0.3 * r.standard_normal(W)
            w[Q + "down.b"][:CODE] = 0.0
        elif mlp:
            E = mlp["router"]["experts"]
            w[Q + "router"] = np.zeros((E, W))
            w[Q + "router"][:, :CODE] = r.standard_normal((E, CODE)) * 0.6
            for e in range(E):
                f = mlp["expert"]["ff"]
                w[Q + f"e{e}.gate"], w[Q + f"e{e}.up"], w[Q + f"e{e}.down"] = lin(f, W, 1.5), lin(f, W, 1.5), out(f, 1.5)
    w = {k: bf16(v) for k, v in w.items()}
    for _ in range(1000):
        close = np.nonzero(gaps(cfg, w) < 0.03)[0]
        if not len(close):
            break
        w["embed"][close, :CODE] = bf16(r.standard_normal((len(close), CODE)))
    return w


def decoder(cfg, w, batch, max_len, dtype="float32", **kw):
    from poptransformer_b200 import registry
    return registry.build_decoder(cfg, tensors(w), batch, max_len, dtype, **kw)


# configurations that differ in every size, in what the layers have, and in values that could be taken for granted
CONFIGS = {
    "mixed": config([latent(mlp=dense()), attention(mlp=moe()), latent(heads=3, dim=16, rot=32, vdim=8, kv_rank=72, q_rank=24, base=50.0, mlp=moe(9, 3, 72)),
                     attention(heads=4, kv_heads=4, dim=16, vdim=40, window=70, softcap=1.5), latent(vdim=16)], loop=(1, 3, 3)),
    "odd-sizes": config([attention(heads=5, kv_heads=5, dim=14, vdim=9, window=7, mlp=dense(13)), latent(heads=3, dim=13, rot=6, vdim=11, kv_rank=21, q_rank=17, mlp=moe(5, 5, 7)),
                         attention(heads=3, kv_heads=1, dim=22, vdim=22, window=1, softcap=20.0, mlp=moe(3, 1, 13))], width=50, vocab=77, eps=1e-3, softcap=2.0, loop=(0, 3, 2)),
    "wide-heads": config([latent(heads=20, dim=128, rot=64, vdim=128, kv_rank=512, q_rank=96, mlp=moe(33, 4, 64)),
                          attention(heads=16, kv_heads=2, dim=128, vdim=64, window=100, mlp=dense(192)),
                          latent(heads=17, dim=64, rot=8, vdim=64, kv_rank=200, q_rank=64, mlp=moe(4, 2, 192))], width=128, vocab=256),
    "plain-order": config([attention(window=500, softcap=8.0), latent(heads=1, dim=8, rot=48, vdim=72, kv_rank=136, q_rank=136, mlp=dense(8)), latent(mlp=moe(4, 4, 24))],
                          width=72, softcap=30.0, loop=(2, 3, 1)),
}
