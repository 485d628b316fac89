"""Plain restatement of the Sabisun decoder in numpy, one function per mechanism, whole sequences only (no cache, no batching).

Everything is float64 unless a dtype is given.  `tests/test_gpu_sabisun.py` compares the kernels with it; it shares no code with
the product path and is never timed.  Conventions: rows are tokens, linears are W[out, in] applied as x @ W.T.
"""
import numpy as np


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) along the last axis."""
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def silu(x):
    return x / (1.0 + np.exp(-x))


def softplus(x):
    return np.logaddexp(0.0, x)


# ------------------------------------------------------------------------------------------ hyper-connections
def stream_read(xs, w_in):
    """Input of a sublayer: sum over streams of w_in[s] * xs[s].  xs [S, T, W]."""
    return np.tensordot(w_in, xs, axes=(0, 0))


def stream_write(xs, y, mix, w_out, mult):
    """New streams: out[t] = sum_s mix[s, t] * xs[s] + mult * w_out[t] * y."""
    return np.tensordot(mix.T, xs, axes=(1, 0)) + mult * w_out[:, None, None] * y[None]


# ------------------------------------------------------------------------------------------ attention
def visible(n, size=None, keep_first=0):
    """Boolean [query, key]: causal, and either less than `size` tokens back or one of the first `keep_first` tokens."""
    i, j = np.arange(n)[:, None], np.arange(n)[None, :]
    ok = j <= i
    if size is not None:
        ok &= ((i - j) < size) | (j < keep_first)
    return ok


def sink_softmax(scores, sink):
    """Softmax of [..., keys] whose denominator also holds exp(sink) (sink broadcasts over the leading axes; None: plain)."""
    m = scores.max(-1, keepdims=True)
    if sink is not None:
        m = np.maximum(m, sink)
    e = np.exp(scores - m)
    den = e.sum(-1, keepdims=True)
    if sink is not None:
        den = den + np.exp(sink - m)
    return e / den


def attention(q, k, v, scale, mask, sink):
    """q [T, H, D], k [T, G, D], v [T, G, V]: grouped heads, no rotation.  Returns [T, H * V]."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = np.empty((T, H, v.shape[2]), q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = np.where(mask, (q[:, h] @ k[:, g].T) * scale, -np.inf)
        out[:, h] = sink_softmax(s, None if sink is None else sink[h]) @ v[:, g]
    return out.reshape(T, -1)


# ------------------------------------------------------------------------------------------ state-space layer
def causal_conv(x, w, b):
    """Per channel: y[t] = b + sum_k w[:, k] * x[t - (taps - 1) + k], zeros before the first token.  x [T, C], w [C, taps]."""
    taps = w.shape[1]
    pad = np.concatenate([np.zeros((taps - 1, x.shape[1]), x.dtype), x], 0)
    return b + sum(pad[k:k + x.shape[0]] * w[:, k] for k in range(taps))


def ssm_scan(x, B, C, dt, A_log, D):
    """The recurrence token by token.  x [T, heads, P], B / C [T, G, N], dt [T, heads] (already positive).
    S <- exp(-exp(A_log) dt) S + dt B x^T, y = S^T C + D x.  Returns y [T, heads, P]."""
    T, H, P = x.shape
    G, N = B.shape[1:]
    grp = np.arange(H) // (H // G)
    S = np.zeros((H, N, P), x.dtype)
    y = np.empty_like(x)
    for t in range(T):
        decay = np.exp(-np.exp(A_log) * dt[t])
        S = decay[:, None, None] * S + dt[t][:, None, None] * B[t][grp][:, :, None] * x[t][:, None, :]
        y[t] = np.einsum("hnp,hn->hp", S, C[t][grp]) + D[:, None] * x[t]
    return y


def gated_group_norm(y, z, w, groups, eps):
    """y * silu(z), then RMS norm of `groups` equal parts, then the weight.  [T, inner]."""
    g = y * silu(z)
    return rms(g.reshape(g.shape[0], groups, -1), eps).reshape(g.shape) * w


# ------------------------------------------------------------------------------------------ the model
class SabisunOracle:
    """cfg: the parsed config.json; weights: {name: array}."""

    def __init__(self, cfg, weights, dtype=np.float64):
        self.cfg = cfg
        self.w = {k: np.asarray(v).astype(dtype) for k, v in weights.items()}

    def _mixer_attention(self, i, m, h, kv):
        w, T = self.w, h.shape[0]
        p = f"l{i}.mix."
        q = (h @ w[p + "q"].T).reshape(T, m["heads"], m["dim"])
        src = m.get("kv_from")
        if src is None:
            kv[i] = ((h @ w[p + "k"].T).reshape(T, m["kv_heads"], m["dim"]), (h @ w[p + "v"].T).reshape(T, m["kv_heads"], m["vdim"]))
            src = i
        mask = m.get("mask") or {}
        y = attention(q, *kv[src], m["scale"], visible(T, mask.get("size"), mask.get("keep_first", 0)), w.get(p + "sink"))
        return y @ w[p + "o"].T

    def _mixer_mamba2(self, i, m, h):
        w, T = self.w, h.shape[0]
        p = f"l{i}.mix."
        H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
        inner = H * P
        z, xbc, dt = np.split(h @ w[p + "in"].T, [inner, 2 * inner + 2 * G * N], axis=1)
        x, B, C = np.split(silu(causal_conv(xbc, w[p + "conv"], w[p + "conv.b"])), [inner, inner + G * N], axis=1)
        y = ssm_scan(x.reshape(T, H, P), B.reshape(T, G, N), C.reshape(T, G, N), softplus(dt + w[p + "dt_bias"]), w[p + "A_log"], w[p + "D"])
        return gated_group_norm(y.reshape(T, inner), z, w[p + "norm"], m["norm_groups"], self.cfg["norm"]["eps"]) @ w[p + "o"].T

    def forward(self, tokens, layer_sums=None):
        """Logits [T, vocab] of one sequence; `layer_sums` (a list) collects the sum of the streams after every layer."""
        c, w = self.cfg, self.w
        eps, mult = c["norm"]["eps"], c["residual_mult"]
        x = w["embed"][np.asarray(tokens)]
        xs = np.repeat(x[None], c["streams"], 0)
        kv = {}
        for i, lay in enumerate(c["layers"]):
            subs = [("1", (lambda h: self._mixer_attention(i, lay["mixer"], h, kv)) if lay["type"] == "attention"
                     else (lambda h: self._mixer_mamba2(i, lay["mixer"], h)))]
            if lay.get("mlp"):
                subs.append(("2", lambda h: np.maximum(h @ w[f"l{i}.mlp.up"].T, 0.0) ** 2 @ w[f"l{i}.mlp.down"].T))
            for q, f in subs:
                u = stream_read(xs, w[f"l{i}.hc{q}.in"])
                y = f(rms(u, eps) * w[f"l{i}.norm{q}"])
                xs = stream_write(xs, y, w[f"l{i}.hc{q}.mix"], w[f"l{i}.hc{q}.out"], mult)
            if layer_sums is not None:
                layer_sums.append(xs.sum(0))
        return rms(xs.sum(0), eps) * w["final.norm"] @ w["embed"].T * c["logit_scale"]
