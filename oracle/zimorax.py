"""Plain, slow NumPy statement of the Zimorax decoder -- TEST INFRASTRUCTURE ONLY.

One function per mechanism, whole sequences at a time, no cache, no batching and no code shared with the product
package. `forward` runs a token list through the model and returns logits and the residual stream after every layer run.

Notation. X is [tokens, width]; a linear weight A is [out, in] and acts as X A^T. `cfg` is the parsed config.json, `w`
maps tensor names to arrays. Arithmetic runs in the dtype of `w` (float64 in the tests).
"""
from __future__ import annotations

import math
from typing import Any, Mapping

import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def rms(x, eps):
    """x over its root mean square along the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def layer_norm(x, weight, eps):
    d = x - x.mean(axis=-1, keepdims=True)
    return rms(d, eps) * weight


def yarn_frequencies(dims, base, scaling=None):
    """(frequencies [dims/2], factor of cos and sin)"""
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if scaling is None:
        return np.array(f), 1.0
    factor, original = float(scaling["factor"]), float(scaling["original"])

    def place(turns):
        """The (fractional) pair that turns that often within the original length."""
        return dims * math.log(original / (2 * math.pi * turns)) / (2 * math.log(base))
    lo = max(math.floor(place(float(scaling["fast"]))), 0)
    hi = min(math.ceil(place(float(scaling["slow"]))), dims - 1)
    out = []
    for i, x in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(x / factor * ramp + x * (1.0 - ramp))
    return np.array(out), 0.1 * math.log(factor) + 1.0


def rotate_half(x, freq, factor):
    """Rotary positions on the first 2 len(freq) entries of x [tokens, heads, d]; entry i turns with entry i + len(freq)."""
    half = len(freq)
    angle = (np.arange(x.shape[0], dtype=np.float64)[:, None] * freq[None, :])[:, None, :]
    c, s = np.cos(angle) * factor, np.sin(angle) * factor
    u, v = x[..., :half], x[..., half:2 * half]
    return np.concatenate([u * c - v * s, v * c + u * s, x[..., 2 * half:]], axis=-1)


def seen(n, size=None):
    """[n, n] which key (column) a query (row) sees: itself and the size - 1 positions before it, or all before it."""
    gap = np.arange(n)[:, None] - np.arange(n)[None, :]
    return (gap >= 0) & (np.ones((n, n), bool) if size is None else gap < size)


def attend(q, k, v, scale, talk, mask):
    """q [n, H, d], k [n, G, d], v [n, G, e] -> [n, H, e]. Every head's scores become the mixture talk[h] of all heads' scores
    before the softmax, whose denominator holds one more exp(0)."""
    n, heads, groups = q.shape[0], q.shape[1], k.shape[1]
    raw = np.stack([(q[:, h] @ k[:, h // (heads // groups)].T) * scale for h in range(heads)])
    out = np.empty((n, heads, v.shape[2]), dtype=q.dtype)
    for h in range(heads):
        z = np.zeros((n, n), q.dtype)
        for g in range(heads):
            z = z + talk[h, g] * raw[g]
        z = np.where(mask, z, -np.inf)
        top = np.maximum(z.max(axis=1, keepdims=True), 0.0)
        e = np.exp(z - top)
        out[:, h] = (e / (np.exp(-top) + e.sum(axis=1, keepdims=True))) @ v[:, h // (heads // groups)]
    return out


def attention(h, m, w, p, eps):
    n, heads, groups, dim, vdim = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = (h @ w[p + "q"].T + w[p + "q.b"]).reshape(n, heads, dim)
    k = (h @ w[p + "k"].T + w[p + "k.b"]).reshape(n, groups, dim)
    v = rms((h @ w[p + "v"].T + w[p + "v.b"]).reshape(n, groups, vdim), eps)
    if m.get("rot"):
        freq, factor = yarn_frequencies(int(m["rot"]["dims"]), float(m["rot"]["base"]), m["rot"].get("scaling"))
        q, k = rotate_half(q, freq, factor), rotate_half(k, freq, factor)
    mask = seen(n, int(m["mask"]["size"]) if m.get("mask") else None)
    o = attend(q, k, v, float(m["scale"]), w[p + "talk"], mask)
    return o.reshape(n, heads * vdim) @ w[p + "o"].T


def causal_conv(x, taps, bias=None):
    """y[t] = sum_j taps[:, j] x[t - (taps - 1) + j], zeros before the start; then silu."""
    n, count = x.shape[0], taps.shape[1]
    y = np.zeros_like(x)
    for t in range(n):
        for j in range(count):
            s = t - (count - 1) + j
            if s >= 0:
                y[t] += taps[:, j] * x[s]
    return silu(y if bias is None else y + bias)


def state_space(x, b, c, dt, log_rate, skip):
    """x [n, H, e], b, c [n, groups, d], dt [n, H]: S <- exp(-exp(log_rate) dt) S + dt b x^T, y = S^T c + skip x."""
    n, heads, e = x.shape
    share = heads // b.shape[1]
    state = np.zeros((heads, b.shape[2], e), x.dtype)
    y = np.empty_like(x)
    for t in range(n):
        for h in range(heads):
            g = h // share
            state[h] = np.exp(-np.exp(log_rate[h]) * dt[t, h]) * state[h] + dt[t, h] * np.outer(b[t, g], x[t, h])
            y[t, h] = state[h].T @ c[t, g] + skip[h] * x[t, h]
    return y


def mamba2(h, m, w, p, eps):
    n, heads, e, d, groups = h.shape[0], int(m["heads"]), int(m["vdim"]), int(m["state"]), int(m["groups"])
    inner, parts = heads * e, int(m["norm_groups"])
    z, xbc, dt = np.split(h @ w[p + "in"].T, [inner, 2 * inner + 2 * groups * d], axis=1)
    xbc = causal_conv(xbc, w[p + "conv"], w[p + "conv.b"])
    x, b, c = np.split(xbc, [inner, inner + groups * d], axis=1)
    y = state_space(x.reshape(n, heads, e), b.reshape(n, groups, d), c.reshape(n, groups, d), softplus(dt + w[p + "dt_bias"]),
                    w[p + "A_log"], w[p + "D"])
    y = (y.reshape(n, inner) * silu(z)).reshape(n, parts, inner // parts)
    return (rms(y, eps).reshape(n, inner) * w[p + "norm"]) @ w[p + "o"].T


def delta_rule(q, k, v, beta, decay):
    """q, k [n, G, d], v [n, H, e], beta, decay [n, H] -> [n, H, e]."""
    n, heads, e = v.shape
    share = heads // q.shape[1]
    state = np.zeros((heads, q.shape[2], e), v.dtype)
    out = np.empty_like(v)
    for t in range(n):
        for h in range(heads):
            g = h // share
            s = decay[t, h] * state[h]
            u = beta[t, h] * (v[t, h] - s.T @ k[t, g])
            state[h] = s + np.outer(k[t, g], u)
            out[t, h] = state[h].T @ q[t, g]
    return out


def unit(x):
    return x / np.sqrt((x * x).sum(axis=-1, keepdims=True) + 1e-6)


def delta(h, m, w, p, eps):
    n, heads, groups, dim, e = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q, k, v = (causal_conv(h @ w[p + s].T, w[p + s + ".conv"]) for s in ("q", "k", "v"))
    q, k = unit(q.reshape(n, groups, dim)) * dim ** -0.5, unit(k.reshape(n, groups, dim))
    beta = sigmoid(h @ w[p + "b"].T)
    decay = np.exp(-np.exp(w[p + "A_log"]) * softplus(h @ w[p + "a"].T + w[p + "dt_bias"]))
    o = rms(delta_rule(q, k, v.reshape(n, heads, e), beta, decay), eps) * w[p + "norm"]
    return (o * silu(h @ w[p + "g"].T).reshape(n, heads, e)).reshape(n, heads * e) @ w[p + "o"].T


def feed_forward(h, w, p):
    a = np.maximum(h @ w[p + "up"].T + w[p + "up.b"], 0.0)
    return (a * a) @ w[p + "down"].T + w[p + "down.b"]


def layer_runs(cfg):
    """(layer, pass that begins right before it or None) in the order they run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    start, stop = int(loop["start"]), int(loop["stop"])
    runs = [(i, None) for i in range(start)]
    for t in range(int(loop["times"])):
        runs += [(i, t if i == start else None) for i in range(start, stop)]
    return runs + [(i, None) for i in range(stop, n)]


MIXERS = {"attention": attention, "mamba2": mamba2, "delta": delta}


def forward(cfg: Mapping[str, Any], w: Mapping[str, np.ndarray], tokens):
    """(logits [tokens, vocab], residual stream after every layer run)"""
    eps = float(cfg["norm"]["eps"])
    start = w["embed"][np.asarray(tokens, np.int64)]
    x, residuals = start, []
    for i, begins in layer_runs(cfg):
        if begins is not None:
            x = np.concatenate([x, start], axis=1) @ w["loop.in"].T + w["loop.step"][begins]
        layer, p = cfg["layers"][i], f"l{i}."
        x = x + MIXERS[layer["type"]](layer_norm(x, w[p + "norm1"], eps), layer["mixer"], w, p + "mix.", eps) * w[p + "ls1"]
        if layer.get("mlp"):
            x = x + feed_forward(layer_norm(x, w[p + "norm2"], eps), w, p + "mlp.") * w[p + "ls2"]
        residuals.append(x)
    return layer_norm(x, w["final.norm"], eps) @ w["head"].T, residuals
