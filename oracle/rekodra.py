"""Plain, slow NumPy statement of the Rekodra decoder -- TEST INFRASTRUCTURE ONLY.

One function per mechanism, whole sequences at a time, no cache, no batching and no code shared with the product
package. `forward` runs a token list through the model and returns logits and the residual stream after every layer run.

Notation. X is [tokens, width]; a linear weight A is [out, in] and acts as X A^T. `cfg` is the parsed config.json, `w`
maps tensor names to arrays. Arithmetic runs in the dtype of `w` (float64 in the tests).
"""
from __future__ import annotations

from typing import Any, Mapping

import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def log_sigmoid(z):
    return np.minimum(z, 0.0) - np.log1p(np.exp(-np.abs(z)))


def rms(x, eps):
    """x over its root mean square along the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def rotate_half(x, dims, base):
    """Rotary positions on the first `dims` entries of x [tokens, heads, d]; entry i turns with entry i + dims/2 by row
    number times base^(-2i/dims)."""
    half = dims // 2
    freq = float(base) ** (-2.0 * np.arange(half, dtype=np.float64) / max(dims, 1))
    angle = (np.arange(x.shape[0], dtype=np.float64)[:, None] * freq[None, :])[:, None, :]
    c, s = np.cos(angle), np.sin(angle)
    u, v = x[..., :half], x[..., half:dims]
    return np.concatenate([u * c - v * s, v * c + u * s, x[..., dims:]], axis=-1)


def seen(n, size=None):
    """[n, n] which key (column) a query (row) sees: itself and the size - 1 positions before it, or all before it."""
    gap = np.arange(n)[:, None] - np.arange(n)[None, :]
    return (gap >= 0) & (np.ones((n, n), bool) if size is None else gap < size)


def attend(q, k, v, scale, mask, sink=None):
    """q [n, heads, d], k [n, groups, d], v [n, groups, e] -> [n, heads, e]; neighbouring heads share a group. With a sink
    the denominator holds one more exp(sink[head])."""
    heads, groups = q.shape[1], k.shape[1]
    out = np.empty((q.shape[0], heads, v.shape[2]), dtype=q.dtype)
    for h in range(heads):
        g = h // (heads // groups)
        z = np.where(mask, (q[:, h] @ k[:, g].T) * scale, -np.inf)
        top = z.max(axis=1, keepdims=True)
        if sink is not None:
            top = np.maximum(top, sink[h])
        e = np.exp(z - top)
        total = e.sum(axis=1, keepdims=True)
        if sink is not None:
            total = total + np.exp(sink[h] - top)
        out[:, h] = (e / total) @ v[:, g]
    return out


def tied_attention(h, m, w, p, eps):
    """Values are the projected keys; queries and keys are normalised over the whole projection, then rotated."""
    n, heads, groups, dim = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"])
    q, k = h @ w[p + "q"].T, h @ w[p + "k"].T
    v = k.reshape(n, groups, dim)
    qn = (rms(q, eps) * w[p + "q.norm"]).reshape(n, heads, dim)
    kn = (rms(k, eps) * w[p + "k.norm"]).reshape(n, groups, dim)
    dims, base = int(m["rot"]["dims"]), m["rot"]["base"]
    o = attend(rotate_half(qn, dims, base), rotate_half(kn, dims, base), v, float(m["scale"]), seen(n), w[p + "sink"])
    return o.reshape(n, heads * dim) @ w[p + "o"].T


def window_attention(h, m, w, p, eps):
    """Queries and keys are normalised head by head; no positions; a sliding window."""
    n, heads, groups, dim, vdim = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = rms((h @ w[p + "q"].T).reshape(n, heads, dim), eps) * w[p + "q.norm"]
    k = rms((h @ w[p + "k"].T).reshape(n, groups, dim), eps) * w[p + "k.norm"]
    v = (h @ w[p + "v"].T).reshape(n, groups, vdim)
    o = attend(q, k, v, float(m["scale"]), seen(n, int(m["mask"]["size"])))
    return o.reshape(n, heads * vdim) @ w[p + "o"].T


def log_gates(h, m, w, p):
    """(log input gate, log forget gate), [tokens, heads] each."""
    cap = float(m["gate_cap"])

    def capped(z):
        return cap * np.tanh(z / cap)
    return capped(h @ w[p + "i"].T + w[p + "i.b"]), log_sigmoid(capped(h @ w[p + "f"].T + w[p + "f.b"]))


def matrix_memory(q, k, v, gi, gf):
    """Token by token: q, k [n, heads, d] (q already scaled), v [n, heads, e], log gates [n, heads] -> [n, heads, e]."""
    n, heads, d = q.shape
    state, norm, top = np.zeros((heads, d, v.shape[2]), q.dtype), np.zeros((heads, d), q.dtype), np.zeros(heads, q.dtype)
    out = np.empty_like(v)
    for t in range(n):
        new = np.maximum(gf[t] + top, gi[t])
        keep, take = np.exp(gf[t] + top - new), np.exp(gi[t] - new)
        state = keep[:, None, None] * state + take[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        norm = keep[:, None] * norm + take[:, None] * k[t]
        top = new
        below = np.maximum(np.abs((norm * q[t]).sum(-1)), np.exp(-top)) + 1e-6
        out[t] = np.einsum("hde,hd->he", state, q[t]) / below[:, None]
    return out


def memory_mixer(h, m, w, p, eps):
    n, heads, dim, vdim = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q = (h @ w[p + "q"].T).reshape(n, heads, dim) * dim ** -0.5
    k = (h @ w[p + "k"].T).reshape(n, heads, dim)
    v = (h @ w[p + "v"].T).reshape(n, heads, vdim)
    o = rms(matrix_memory(q, k, v, *log_gates(h, m, w, p)), eps).reshape(n, heads * vdim)
    return (o * w[p + "norm"] * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def parallel(h, m, w, p, eps):
    left = rms(window_attention(h, m["left"], w, p + "left.", eps), eps) * w[p + "left.out"]
    right = rms(memory_mixer(h, m["right"], w, p + "right.", eps), eps) * w[p + "right.out"]
    return 0.5 * (left + right)


def swiglu(h, w, p):
    g = h @ w[p + "gate"].T
    return (g * sigmoid(g) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def softmax(z):
    e = np.exp(z - z.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def route(z, correction, top, groups=1, keep=1):
    """(chosen, weights) per row of router logits. Choices go by softmax + correction within the `keep` groups whose
    best choice score is largest; the weights are the softmax itself."""
    s = softmax(z)
    choice = s + correction
    best = choice.reshape(len(z), groups, -1).max(axis=-1)
    kept = np.argsort(-best, axis=-1, kind="stable")[:, :keep]
    mask = np.zeros_like(best, dtype=bool)
    np.put_along_axis(mask, kept, True, axis=-1)
    choice = np.where(np.repeat(mask, z.shape[1] // groups, axis=1), choice, -np.inf)
    chosen = np.argsort(-choice, axis=-1, kind="stable")[:, :top]
    return chosen, np.take_along_axis(s, chosen, axis=-1)


def mixture(h, m, w, p):
    r = m["router"]
    groups = r.get("groups") or {"count": 1, "keep": 1}
    chosen, weight = route(h @ w[p + "router"].T, w[p + "correction"], int(r["top"]), int(groups["count"]), int(groups["keep"]))
    y = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, a in zip(chosen[t], weight[t]):
            y[t] += a * (h[t] if e >= int(r["experts"]) else swiglu(h[t:t + 1], w, f"{p}e{e}.")[0])
    if m.get("shared") is not None:
        y = y + swiglu(h, w, p + "shared.") * sigmoid(h @ w[p + "shared.sg"].T)
    return y


def layer_runs(cfg):
    """(layer, whether the embedding output joins right before it) in the order in which layers run."""
    n = len(cfg["layers"])
    loop = cfg.get("loop") or {"start": 0, "stop": 0, "times": 1}
    start, stop = int(loop["start"]), int(loop["stop"])
    runs = [(i, False) for i in range(start)]
    for turn in range(int(loop["times"])):
        runs += [(i, turn > 0 and i == start) for i in range(start, stop)]
    return runs + [(i, False) for i in range(stop, n)]


def forward(cfg: Mapping[str, Any], w: Mapping[str, np.ndarray], tokens) -> tuple[np.ndarray, list[np.ndarray]]:
    """(logits [tokens, vocab], residual stream after every layer run)."""
    eps = float(cfg["norm"]["eps"])
    embedded = w["embed"][np.asarray(tokens, dtype=np.int64)] * float(cfg["embedding"]["scale"])
    x, residuals = embedded, []
    for i, again in layer_runs(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        if again:
            x = x + embedded
        h = rms(x, eps) * w[p + "norm1"]
        x = x + {"attention": tied_attention, "parallel": parallel}[layer["type"]](h, layer["mixer"], w, p + "mix.", eps)
        if layer.get("mlp") is not None:
            x = x + mixture(rms(x, eps) * w[p + "norm2"], layer["mlp"], w, p + "mlp.")
        residuals.append(x)
    return (rms(x, eps) * w["final.norm"]) @ w["embed"].T * float(cfg["logit_scale"]), residuals
