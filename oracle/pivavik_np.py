"""Plain restatement of the Pivavik decoder in numpy, one function per mechanism, whole sequences only (no cache, no batching).

Everything is float64 unless a dtype is given.  `tests/test_gpu_pivavik.py` compares the kernels with it; it shares no code with
the product path and is never timed.  Conventions: rows are tokens, linears are W[out, in] applied as x @ W.T.
"""
import numpy as np


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) along the last axis."""
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def zero_centred_norm(x, w, eps):
    """RMS norm whose weight is stored as its distance from one."""
    return rms(x, eps) * (1.0 + w)


def sigmoid(x):
    return np.exp(-np.logaddexp(0.0, -x))


def silu(x):
    return x * sigmoid(x)


def gelu_tanh(x):
    return 0.5 * x * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (x + 0.044715 * x ** 3)))


def cap(x, limit):
    """limit * tanh(x / limit); no limit leaves x as it is."""
    return limit * np.tanh(x / limit) if limit else x


# ------------------------------------------------------------------------------------------ attention
def rotate(x, base):
    """x [T, heads, dims], row t at position t: dimension i and dimension i + dims / 2 are a pair that turns by t * base^(-2 i / dims)."""
    T, dims = x.shape[0], x.shape[-1]
    half = dims // 2
    a = np.arange(T)[:, None, None] * np.array([float(base) ** (-2.0 * i / dims) for i in range(half)])
    u, v = x[..., :half], x[..., half:]
    return np.concatenate([u * np.cos(a) - v * np.sin(a), v * np.cos(a) + u * np.sin(a)], -1)


def masked_attention(q, k, v, scale, window=0, softcap=0.0):
    """q [T, H, D], k [T, G, D], v [T, G, V]; head h reads key head h // (H / G); row i sees row j when j <= i and, with a window, i - j <
    window.  Returns [T, H, V]."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    out = np.empty((T, H, v.shape[2]), q.dtype)
    i, j = np.arange(T)[:, None], np.arange(T)
    hidden = (j > i) | ((i - j >= window) if window else False)
    for h in range(H):
        s = cap((q[:, h] @ k[:, h // per].T) * scale, softcap)
        s[hidden] = -np.inf
        e = np.exp(s - s.max(-1, keepdims=True))
        out[:, h] = e / e.sum(-1, keepdims=True) @ v[:, h // per]
    return out


# ------------------------------------------------------------------------------------------ feed-forward
def gated_unit(act, gate, up):
    return act(gate) * up


def choose(z, top):
    """Indices [T, top] of the largest scores sigmoid(z) (lowest index first among equals) and those scores."""
    s = sigmoid(z)
    idx = np.argsort(-z, axis=1, kind="stable")[:, :top]
    return idx, np.take_along_axis(s, idx, 1)


# ------------------------------------------------------------------------------------------ the model
def layer_runs(n_layers, loop):
    """[(layer, pass)] in the order they run; pass is None outside the loop."""
    runs = []
    for i in range(n_layers):
        if loop and i == loop["start"]:
            runs += [(j, t) for t in range(loop["times"]) for j in range(loop["start"], loop["stop"])]
        if not loop or not loop["start"] <= i < loop["stop"]:
            runs.append((i, None))
    return runs


class PivavikOracle:
    """cfg: the parsed config.json; weights: {name: array}."""

    def __init__(self, cfg, weights, dtype=np.float64):
        self.cfg, self.eps = cfg, cfg["norm"]["eps"]
        self.w = {k: np.asarray(v).astype(dtype) for k, v in weights.items()}

    def lin(self, name, x):
        y = x @ self.w[name].T
        return y + self.w[name + ".b"] if name + ".b" in self.w else y

    def latent_attention(self, p, m, h):
        T, H, D, R, V, rank = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
        cq = rms(self.lin(p + "dq", h), self.eps) * self.w[p + "dq.norm"]
        q = self.lin(p + "uq", cq).reshape(T, H, D + R)
        down = self.lin(p + "dkv", h)
        c = rms(down[:, :rank], self.eps) * self.w[p + "dkv.norm"]
        k = self.lin(p + "uk", c).reshape(T, H, D)
        v = self.lin(p + "uv", c).reshape(T, H, V)
        base = m["rot"]["base"]
        q_rot, k_rot = rotate(q[..., D:], base), rotate(down[:, None, rank:], base)
        q = np.concatenate([q[..., :D], q_rot], -1)
        k = np.concatenate([k, np.repeat(k_rot, H, 1)], -1)
        o = masked_attention(q, k, v, m["scale"]) * sigmoid(self.lin(p + "g", h))[..., None]
        return self.lin(p + "o", o.reshape(T, -1))

    def attention(self, p, m, h):
        T = h.shape[0]
        q, k, v = (self.lin(p + n, h).reshape(T, heads, -1) for n, heads in (("q", m["heads"]), ("k", m["kv_heads"]), ("v", m["kv_heads"])))
        o = masked_attention(q, k, v, m["scale"], m["mask"]["size"], m["softcap"]).reshape(T, -1)
        return self.lin(p + "o", o * sigmoid(self.lin(p + "g", h)))

    def dense(self, p, h, act):
        return self.lin(p + "down", gated_unit(act, self.lin(p + "gate", h), self.lin(p + "up", h)))

    def experts(self, p, m, h):
        idx, wt = choose(self.lin(p + "router", h), m["router"]["top"])
        y = np.zeros_like(h)
        for e in range(m["router"]["experts"]):
            t, k = np.nonzero(idx == e)
            y[t] += self.dense(p + f"e{e}.", wt[t, k][:, None] * h[t], silu)
        return y

    def layer(self, i, x):
        lay, p = self.cfg["layers"][i], f"l{i}."
        h = zero_centred_norm(x, self.w[p + "norm1"], self.eps)
        y = {"latent_attention": self.latent_attention, "attention": self.attention}[lay["type"]](p + "mix.", lay["mixer"], h)
        mlp = lay.get("mlp")
        if mlp:
            y = y + (self.dense(p + "mlp.", h, gelu_tanh) if mlp["kind"] == "dense" else self.experts(p + "mlp.", mlp, h))
        return x + y

    def forward(self, tokens, layer_sums=None):
        """Logits [T, vocab] of one sequence; `layer_sums` (a list) collects the residual stream after every layer run."""
        w, cfg, loop = self.w, self.cfg, self.cfg.get("loop")
        x0 = x = zero_centred_norm(w["embed"][np.asarray(tokens)], w["embed.norm"], self.eps)
        for i, t in layer_runs(len(cfg["layers"]), loop):
            if t is not None and i == loop["start"]:
                x = np.concatenate([x, x0], 1) @ w["loop.in"].T + w["loop.step"][t]
            x = self.layer(i, x)
            if layer_sums is not None:
                layer_sums.append(x)
        return cap(zero_centred_norm(x, w["final.norm"], self.eps) @ w["embed"].T, cfg.get("logit_softcap"))
