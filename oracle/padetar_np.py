"""Plain restatement of the Padetar decoder in numpy, one function per mechanism, whole sequences only (no cache, no batching).

Everything is float64 unless a dtype is given.  `tests/test_gpu_padetar.py` compares the kernels with it; it shares no code with
the product path and is never timed.  Conventions: rows are tokens, linears are W[out, in] applied as x @ W.T.
"""
import numpy as np


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) along the last axis."""
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def sigmoid(x):
    return np.exp(-np.logaddexp(0.0, -x))


def gelu_tanh(x):
    return 0.5 * x * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (x + 0.044715 * x ** 3)))


# ------------------------------------------------------------------------------------------ rotation
def frequencies(dims, base, scaling=None):
    """Angle per position of every rotated pair.  scaling (factor, low, high, original): long wavelengths are stretched by
    `factor`, short ones kept, those between blended linearly in original / wavelength."""
    out = []
    for i in range(dims // 2):
        f = float(base) ** (-2.0 * i / dims)
        if scaling:
            turns = scaling["original"] * f / (2.0 * np.pi)          # original / wavelength
            if turns < scaling["low"]:
                f = f / scaling["factor"]
            elif turns <= scaling["high"]:
                s = (turns - scaling["low"]) / (scaling["high"] - scaling["low"])
                f = (1.0 - s) * f / scaling["factor"] + s * f
        out.append(f)
    return np.array(out)


def rotate(x, freq):
    """x [T, heads, dim]: pair (i, i + len(freq)) of row t turns by t * freq[i]; dimensions beyond the pairs stay."""
    T, half = x.shape[0], len(freq)
    a = np.arange(T)[:, None, None] * freq
    u, v = x[..., :half], x[..., half:2 * half]
    return np.concatenate([u * np.cos(a) - v * np.sin(a), v * np.cos(a) + u * np.sin(a), x[..., 2 * half:]], -1)


# ------------------------------------------------------------------------------------------ attention
def causal_attention(q, k, v, scale):
    """q [T, H, D], k [T, G, D], v [T, G, V]; head h reads key head h // (H / G).  Returns [T, H * V]."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    out = np.empty((T, H, v.shape[2]), q.dtype)
    future = np.triu(np.ones((T, T), bool), 1)
    for h in range(H):
        s = (q[:, h] @ k[:, h // per].T) * scale
        s[future] = -np.inf
        e = np.exp(s - s.max(-1, keepdims=True))
        out[:, h] = e / e.sum(-1, keepdims=True) @ v[:, h // per]
    return out.reshape(T, -1)


# ------------------------------------------------------------------------------------------ matrix memory
def memory_gates(zi, zf, cap):
    """Log input and log forget gates from their pre-activations."""
    return cap * np.tanh(zi / cap), -np.logaddexp(0.0, -cap * np.tanh(zf / cap))


def matrix_memory(q, k, v, log_i, log_f):
    """Token by token.  q (already scaled), k [T, H, D], v [T, H, V], gates [T, H].  Returns [T, H, V]."""
    T, H, D = q.shape
    S, n, m = np.zeros((H, D, v.shape[2]), q.dtype), np.zeros((H, D), q.dtype), np.zeros(H, q.dtype)
    out = np.empty_like(v)
    for t in range(T):
        new = np.maximum(log_f[t] + m, log_i[t])
        keep, add = np.exp(log_f[t] + m - new), np.exp(log_i[t] - new)
        m = new
        S = keep[:, None, None] * S + add[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + add[:, None] * k[t]
        den = np.maximum(np.abs((n * q[t]).sum(-1)), np.exp(-m)) + 1e-6
        out[t] = np.einsum("hdv,hd->hv", S, q[t]) / den[:, None]
    return out


# ------------------------------------------------------------------------------------------ experts
def clamped_glu(gate, up, limit):
    g, u = np.minimum(gate, limit), np.clip(up, -limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


def choose(z, top):
    """Indices [T, top] of the largest logits (lowest index first among equals) and the softmax over them."""
    idx = np.argsort(-z, axis=1, kind="stable")[:, :top]
    c = np.take_along_axis(z, idx, 1)
    e = np.exp(c - c.max(1, keepdims=True))
    return idx, e / e.sum(1, keepdims=True)


# ------------------------------------------------------------------------------------------ the model
class PadetarOracle:
    """cfg: the parsed config.json; weights: {name: array}."""

    def __init__(self, cfg, weights, dtype=np.float64):
        self.cfg, self.eps = cfg, cfg["norm"]["eps"]
        self.w = {k: np.asarray(v).astype(dtype) for k, v in weights.items()}

    def lin(self, name, x):
        y = x @ self.w[name].T
        return y + self.w[name + ".b"] if name + ".b" in self.w else y

    def left(self, p, m, h):
        T, D = h.shape[0], m["dim"]
        q, raw = self.lin(p + "q", h).reshape(T, m["heads"], D), self.lin(p + "k", h).reshape(T, m["kv_heads"], D)
        freq = frequencies(m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling"))
        q, k = (rotate(rms(x, self.eps) * self.w[p + n + ".norm"], freq) for x, n in ((q, "q"), (raw, "k")))
        return self.lin(p + "o", causal_attention(q, k, raw, m["scale"]))

    def right(self, p, m, h):
        T, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
        li, lf = memory_gates(self.lin(p + "i", h), self.lin(p + "f", h), m["gate_cap"])
        o = matrix_memory(self.lin(p + "q", h).reshape(T, H, D) * D ** -0.5, self.lin(p + "k", h).reshape(T, H, D), self.lin(p + "v", h).reshape(T, H, V), li, lf)
        return self.lin(p + "o", rms(o, self.eps).reshape(T, H * V) * self.w[p + "norm"] * sigmoid(self.lin(p + "g", h)))

    def glu(self, p, h, limit):
        return self.lin(p + "down", clamped_glu(self.lin(p + "gate", h), self.lin(p + "up", h), limit))

    def experts(self, p, m, h):
        idx, wt = choose(h @ self.w[p + "router"].T + self.w[p + "router.b"], m["router"]["top"])
        y = np.zeros_like(h)
        for e in range(m["router"]["experts"]):
            t, k = np.nonzero(idx == e)
            y[t] += wt[t, k][:, None] * self.glu(p + f"e{e}.", h[t], m["expert"]["limit"])
        return y + self.glu(p + "shared.", h, m["shared"]["limit"]) if m.get("shared") else y

    def side(self, p, i, tokens, x):
        d = self.cfg["token_side"]["dim"]
        e = self.w["side.embed"][tokens][:, i * d:(i + 1) * d]
        return self.lin(p + "proj", gelu_tanh(self.lin(p + "gate", x)) * e)

    def forward(self, tokens, layer_sums=None):
        """Logits [T, vocab] of one sequence; `layer_sums` (a list) collects the residual stream after every layer."""
        w, eps, tokens = self.w, self.eps, np.asarray(tokens)
        x = w["embed"][tokens]
        for i, lay in enumerate(self.cfg["layers"]):
            p, m = f"l{i}.", lay["mixer"]
            y = m["left_scale"] * self.left(p + "mix.left.", m["left"], x) + m["right_scale"] * self.right(p + "mix.right.", m["right"], x)
            x = x + rms(y, eps) * w[p + "norm1"]
            if lay.get("mlp"):
                x = x + rms(self.experts(p + "mlp.", lay["mlp"], x), eps) * w[p + "norm2"]
            if self.cfg.get("token_side"):
                x = x + rms(self.side(p + "side.", i, tokens, x), eps) * w[p + "side.norm"]
            if layer_sums is not None:
                layer_sums.append(x)
        return rms(x, eps) * w["final.norm"] @ w["head"].T
