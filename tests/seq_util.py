"""What the tests of decoders with per-sequence positions share: types, batches, model folders, portions, comparisons."""
import json
import os

import numpy as np
import torch


def bf16(x):
    """float array rounded to bfloat16 (as float32)."""
    return torch.from_numpy(np.ascontiguousarray(x, dtype=np.float32)).to(torch.bfloat16).float().numpy()


def tensors(w):
    return {k: torch.from_numpy(v).to(torch.bfloat16) for k, v in w.items()}


def write_model(path, cfg, w):
    """config.json + model.safetensors (bfloat16)."""
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    head, blobs, at = {}, [], 0
    for k, t in tensors(w).items():
        b = t.contiguous().view(torch.int16).numpy().tobytes()
        head[k] = {"dtype": "BF16", "shape": list(t.shape), "data_offsets": [at, at + len(b)]}
        blobs.append(b)
        at += len(b)
    h = json.dumps(head).encode()
    with open(os.path.join(path, "model.safetensors"), "wb") as f:
        f.write(len(h).to_bytes(8, "little") + h + b"".join(blobs))


def rel(got, want):
    """rms of the difference over the rms of the expected values."""
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    return float(np.sqrt(((got - want) ** 2).mean()) / np.sqrt((want ** 2).mean()))


def i32(x, dev):
    return torch.tensor(np.asarray(x), dtype=torch.int32, device=dev)


def view_of(lens, starts, slots, dev):
    from poptransformer_b200 import ops
    cu = np.concatenate([[0], np.cumsum(lens)])
    return ops.batch_view(len(lens), int(cu[-1]), i32(cu, dev), i32(starts, dev), i32(slots, dev), i32(np.repeat(np.arange(len(lens)), lens), dev))


def as_type(x, dt, dev):
    return torch.from_numpy(np.ascontiguousarray(x, dtype=np.float32)).to(dev).to(dt)


def prompt(n, vocab, seed=0):
    return np.random.default_rng(100 + seed).integers(0, vocab, n).astype(np.int32)


def run_cut(dec, tokens, cuts):
    """One sequence in portions; logits of every token."""
    s, out, at = dec.open(), [], 0
    for n in cuts:
        out.append(dec.extend([(s, tokens[at:at + n], list(range(n)))]).cpu().numpy())
        at += n
    assert at == len(tokens)
    dec.close(s)
    return np.concatenate(out)


def greedy_ok(orc, ids, lens, tol):
    """Every generated id is the oracle's best along the generated stream, or within `tol` of it (relative to the logits' rms)."""
    exact = total = 0
    for row, n in zip(ids, lens):
        lg = orc.forward(row[:-1])
        for i in range(n, len(row)):
            best, got = lg[i - 1].max(), lg[i - 1][row[i]]
            assert best - got <= tol * np.sqrt((lg[i - 1] ** 2).mean()), i
            exact += int(lg[i - 1].argmax() == row[i])
            total += 1
    return exact / total


class PagedAttention:
    """One attention call site over a cache whose pages lie in shuffled order."""

    def __init__(self, dev, dt, n_seq, G, D, V, max_len, poison=True, page=64, seed=0):
        from poptransformer_b200 import ops
        self.ops, self.dev, self.dt, self.G, self.D, self.V = ops, dev, dt, G, D, V
        pages = -(-max_len // page)
        table = np.random.default_rng(seed).permutation(n_seq * pages).reshape(n_seq, pages)
        self.cache = ops.PagedKVCache(n_seq, G, D, max_len, page, dev, i32(table, dev), v_dim=V, dtype=dt)
        if poison:                                   # nothing may be read that was not written
            self.cache.pool.fill_(float("nan"))
        self.flag = torch.zeros(1, dtype=torch.int32, device=dev)

    def __call__(self, q, k, v, lens, starts, slots, scale, window, keep, sink, plain, pad_cols=0, **kw):
        """q [T, H, D], k [T, G, D], v [T, G, V], packed (no k: read the cache only; no v: the keys are the values).  Further options go
        to window_attn; columns from out_cols on must stay as they were.  Returns [T, H V]."""
        ops, dev, T, H = self.ops, self.dev, q.shape[0], q.shape[1]
        parts = [q.reshape(T, -1)] + [t.reshape(T, -1) for t in (k, v) if t is not None]
        x = np.concatenate(parts, 1)
        ld = x.shape[1] + (-x.shape[1]) % 8
        buf = torch.zeros((T, ld), dtype=self.dt, device=dev)
        buf[:, :x.shape[1]] = as_type(x, self.dt, dev)
        cols = ops.pad_to(H * self.V, 64)
        out_ld = cols + pad_cols
        out = torch.full((T, out_ld), float("nan"), dtype=self.dt, device=dev)
        ws = ops.window_attn_workspace(len(lens), H, self.V, self.cache.page_size, self.cache.max_len, window, keep, dev)
        ops.window_attn(view_of(lens, starts, slots, dev), buf, ld, self.cache, out, out_ld, H, scale, window, keep,
                        None if sink is None else as_type(sink, torch.float32, dev), append=k is not None, max_tokens_per_seq=max(lens), workspace=ws,
                        error_flag=self.flag, plain=plain, out_cols=cols, values_are_keys=v is None, **kw)
        assert out[:, cols:].isnan().all() and not out[:, H * self.V:cols].any() and int(self.flag.item()) == 0
        return out[:, :H * self.V].float().cpu().numpy()
