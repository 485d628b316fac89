"""Plain restatement of the Puputar decoder in numpy, one function per mechanism, whole sequences only (no cache, no batching).

Everything is float64 unless a dtype is given.  `tests/test_gpu_puputar.py` compares the kernels with it; it shares no code with
the product path and is never timed.  Conventions: rows are tokens, linears are W[out, in] applied as x @ W.T.
"""
import numpy as np


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) along the last axis."""
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def group_norm(x, w, eps, groups):
    """Every one of `groups` equal consecutive parts of a row by its own root mean square, then all of it times w."""
    return rms(x.reshape(len(x), groups, -1), eps).reshape(x.shape) * w


def token_shift(h, mix):
    """Row t moves towards row t - 1 (zeros before the first) by the share `mix`, element by element."""
    before = np.concatenate([np.zeros_like(h[:1]), h[:-1]])
    return h + (before - h) * mix


def sigmoid(x):
    return np.exp(-np.logaddexp(0.0, -x))


def softplus(x):
    return np.logaddexp(0.0, x)


def xielu(z, p, q):
    """Quadratic for positive z, an exponential minus its tangent for the others; both with z / 2 in addition."""
    neg = np.minimum(z, 0.0)
    return np.where(z > 0, softplus(p) * z * z, (0.5 + softplus(q)) * (np.expm1(neg) - neg)) + 0.5 * z


def relu2(z):
    return np.maximum(z, 0.0) ** 2


# ------------------------------------------------------------------------------------------ attention
def rotate_pairs(x, base):
    """x [T, heads, dims], row t at position t: dimensions 2 i and 2 i + 1 are a pair that turns by t * base^(-2 i / dims)."""
    T, dims = x.shape[0], x.shape[-1]
    out = np.empty_like(x)
    for i in range(dims // 2):
        a = (np.arange(T) * float(base) ** (-2.0 * i / dims))[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = u * np.cos(a) - v * np.sin(a), v * np.cos(a) + u * np.sin(a)
    return out


def causal_attention(q, k, v, scale):
    """q, k [T, H, D], v [T, H, V]; row i sees the rows up to i.  Returns [T, H, V]."""
    T, H, _ = q.shape
    out = np.empty((T, H, v.shape[2]), q.dtype)
    hidden = np.triu(np.ones((T, T), bool), 1)
    for h in range(H):
        s = (q[:, h] @ k[:, h].T) * scale
        s[hidden] = -np.inf
        e = np.exp(s - s.max(-1, keepdims=True))
        out[:, h] = e / e.sum(-1, keepdims=True) @ v[:, h]
    return out


# ------------------------------------------------------------------------------------------ experts
def choice_scores(z, correction, groups, keep):
    """Softmax scores of the router's logits, and the scores experts are chosen by: corrected, minus infinity outside the `keep` groups
    of neighbours whose best corrected score is largest."""
    e = np.exp(z - z.max(-1, keepdims=True))
    s = e / e.sum(-1, keepdims=True)
    c = s + correction
    best = c.reshape(len(c), groups, -1).max(-1)
    kept = np.zeros_like(best, bool)
    np.put_along_axis(kept, np.argsort(-best, axis=1, kind="stable")[:, :keep], True, 1)
    return s, np.where(np.repeat(kept, c.shape[1] // groups, 1), c, -np.inf)


def choose(z, correction, top, groups, keep):
    """Indices [T, top] of the chosen experts (lowest index first among equals) and their weights."""
    s, c = choice_scores(z, correction, groups, keep)
    idx = np.argsort(-c, axis=1, kind="stable")[:, :top]
    wt = np.take_along_axis(s, idx, 1)
    return idx, wt / (wt.sum(-1, keepdims=True) + 1e-20)


# ------------------------------------------------------------------------------------------ the model
class PuputarOracle:
    """cfg: the parsed config.json; weights: {name: array}."""

    def __init__(self, cfg, weights, dtype=np.float64):
        self.cfg, self.eps = cfg, cfg["norm"]["eps"]
        self.w = {k: np.asarray(v).astype(dtype) for k, v in weights.items()}

    def lin(self, name, x):
        y = x @ self.w[name].T
        return y + self.w[name + ".b"] if name + ".b" in self.w else y

    def norm(self, name, x):
        return group_norm(x, self.w[name], self.eps, self.cfg["norm"]["groups"])

    def latents(self, p, m, h):
        """What a layer caches: the normed latent [T, rank] and the rotated key part [T, rot]."""
        down = self.lin(p + "dkv", h)
        return rms(down[:, :m["kv_rank"]], self.eps) * self.w[p + "dkv.norm"], rotate_pairs(down[:, None, m["kv_rank"]:], m["rot"]["base"])[:, 0]

    def latent_attention(self, p, m, h, cached):
        """Returns the heads' outputs [T, heads, vdim] over the cached latents."""
        T, H, D, R = len(h), m["heads"], m["dim"], m["rot_dim"]
        c, kr = cached
        q = self.lin(p + "uq", rms(self.lin(p + "dq", h), self.eps) * self.w[p + "dq.norm"]).reshape(T, H, D + R)
        q = np.concatenate([q[..., :D], rotate_pairs(q[..., D:], m["rot"]["base"])], -1)
        k = np.concatenate([self.lin(p + "uk", c).reshape(T, H, D), np.repeat(kr[:, None], H, 1)], -1)
        return causal_attention(q, k, self.lin(p + "uv", c).reshape(T, H, m["vdim"]), m["scale"])

    def mixer(self, i, h, caches):
        lay, p = self.cfg["layers"][i], f"l{i}.mix."
        m, T = lay["mixer"], len(h)
        source = m.get("kv_from")
        if source is None:
            source = i
            caches[i] = self.latents(p, m, h)
        o, gate = self.latent_attention(p, m, h, caches[source]), sigmoid(self.lin(p + "g", h))
        o = {"latent_attention": lambda: (o * gate[..., None]).reshape(T, -1), "latent_attention_2": lambda: o.reshape(T, -1) * gate}[lay["type"]]()
        return self.lin(p + "o", o)

    def dense(self, p, h):
        return self.lin(p + "down", xielu(self.lin(p + "up", h), *self.w[p + "act"]))

    def experts(self, p, m, h):
        r = m["router"]
        idx, wt = choose(self.lin(p + "router", h), self.w[p + "correction"], r["top"], r["groups"]["count"], r["groups"]["keep"])
        y = np.zeros_like(h)
        for e in range(r["experts"] + r["identity"]):
            t, k = np.nonzero(idx == e)
            out = self.lin(p + f"e{e}.down", relu2(self.lin(p + f"e{e}.up", h[t]))) if e < r["experts"] else h[t]
            y[t] += wt[t, k][:, None] * out
        return y

    def layer(self, i, x, caches):
        p, mlp = f"l{i}.", self.cfg["layers"][i].get("mlp")
        y = self.mixer(i, token_shift(self.norm(p + "norm1", x), self.w[p + "shift"]), caches)
        if mlp:
            h = self.norm(p + "norm2", x)
            y = y + (self.dense(p + "mlp.", h) if mlp["kind"] == "dense" else self.experts(p + "mlp.", mlp, h))
        return x + y

    def forward(self, tokens, layer_sums=None):
        """Logits [T, vocab] of one sequence; `layer_sums` (a list) collects the residual stream after every layer."""
        x, caches = self.norm("embed.norm", self.w["embed"][np.asarray(tokens)]), {}
        for i in range(len(self.cfg["layers"])):
            x = self.layer(i, x, caches)
            if layer_sums is not None:
                layer_sums.append(x)
        return self.norm("final.norm", x) @ self.w["head"].T
