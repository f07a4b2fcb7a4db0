"""Plain, slow NumPy statement of the Topunex decoder -- TEST INFRASTRUCTURE ONLY.

One function per mechanism, whole sequences at a time, no cache, no batching and no code shared with the product
package. `forward` runs a token list through the model and returns logits and the residual stream after every layer.

Notation. X is [tokens, width]; a linear weight A is [out, in] and acts as X A^T (+ b where the model has one). `cfg` is
the parsed config.json, `w` maps tensor names to arrays. Arithmetic runs in the dtype of `w` (float64 in the tests).
"""
from __future__ import annotations

from typing import Any, Mapping

import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def rms(x, eps):
    """x over its root mean square along the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def linear(x, w, name):
    y = x @ w[name].T
    return y + w[name + ".b"] if name + ".b" in w else y


def frequencies(dims, base, scaling=None):
    """Radians per position of each pair; with `scaling` long wavelengths are stretched by `factor`, short ones kept and
    those in between blended."""
    f = float(base) ** (-2.0 * np.arange(dims // 2, dtype=np.float64) / dims)
    if scaling is None:
        return f
    factor, low, high, original = (float(scaling[k]) for k in ("factor", "low", "high", "original"))
    out = np.empty_like(f)
    for i, v in enumerate(f):
        wavelength = 2.0 * np.pi / v
        if wavelength < original / high:
            out[i] = v
        elif wavelength > original / low:
            out[i] = v / factor
        else:
            keep = (original / wavelength - low) / (high - low)
            out[i] = (1.0 - keep) * v / factor + keep * v
    return out


def rotate_half(x, freq):
    """Rotary positions on the first 2 len(freq) entries of x [tokens, heads, d]; entry i turns with entry
    i + len(freq), p = row number."""
    half = len(freq)
    angle = (np.arange(x.shape[0], dtype=np.float64)[:, None] * freq[None, :])[:, None, :]
    c, s = np.cos(angle), np.sin(angle)
    u, v = x[..., :half], x[..., half:2 * half]
    return np.concatenate([u * c - v * s, v * c + u * s, x[..., 2 * half:]], axis=-1)


def seen(n, size=None, keep_first=0):
    """[n, n] which key (column) a query (row) sees: the last `size` positions and the first `keep_first`."""
    i = np.arange(n)
    gap = i[:, None] - i[None, :]
    inside = np.ones((n, n), bool) if size is None else gap < size
    return (gap >= 0) & (inside | (i[None, :] < keep_first))


def softcap(score, cap):
    return score if cap is None else cap * np.tanh(score / cap)


def sink_softmax(score, mask, sink):
    """Rows of softmax over the seen columns with one more exp(sink) in the denominator (nothing without one)."""
    z = np.where(mask, score, -np.inf)
    top = z.max(axis=-1, keepdims=True)
    if sink is not None:
        top = np.maximum(top, sink)
    e = np.exp(z - top)
    total = e.sum(axis=-1, keepdims=True)
    return e / (total if sink is None else total + np.exp(sink - top))


def tied_attention(h, m, w, p, eps):
    """Grouped-query attention whose values are the projected keys."""
    n = h.shape[0]
    heads, groups, dim = int(m["heads"]), int(m["kv_heads"]), int(m["dim"])
    q = linear(h, w, p + "q").reshape(n, heads, dim)
    v = linear(h, w, p + "k").reshape(n, groups, dim)
    freq = frequencies(int(m["rot"]["dims"]), m["rot"]["base"], m["rot"].get("scaling"))
    q, k = rms(rotate_half(q, freq), eps), rms(rotate_half(v, freq), eps)
    mask = seen(n, (m.get("mask") or {}).get("size"), int((m.get("mask") or {}).get("keep_first", 0)))
    out = np.empty((n, heads, dim), dtype=h.dtype)
    for head in range(heads):
        g = head // (heads // groups)
        score = softcap((q[:, head] @ k[:, g].T) * float(m["scale"]), m.get("softcap"))
        out[:, head] = sink_softmax(score, mask, w[p + "sink"][head]) @ v[:, g]
    gated = out.reshape(n, heads * dim) * sigmoid(linear(h, w, p + "g"))
    return linear(gated, w, p + "o")


def swiglu(h, w, p):
    g = linear(h, w, p + "gate")
    return linear(g * sigmoid(g) * linear(h, w, p + "up"), w, p + "down")


def clamped_expert(h, w, p, limit):
    g = np.minimum(h @ w[p + "gate"].T, limit)
    u = np.clip(h @ w[p + "up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].T


def route(z, top, scale):
    """(chosen experts, weights) per row of router logits; equal scores go to the lower index."""
    chosen = np.argsort(-z, axis=-1, kind="stable")[:, :top]
    return chosen, sigmoid(np.take_along_axis(z, chosen, axis=-1)) * scale


def mixture(h, m, w, p):
    chosen, weight = route(h @ w[p + "router"].T, int(m["router"]["top"]), float(m["router"]["scale"]))
    y = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, a in zip(chosen[t], weight[t]):
            y[t] += a * clamped_expert(h[t:t + 1], w, f"{p}e{e}.", float(m["expert"]["limit"]))[0]
    if m.get("shared") is not None:
        y = y + clamped_expert(h, w, p + "shared.", float(m["shared"]["limit"]))
    return y


def forward(cfg: Mapping[str, Any], w: Mapping[str, np.ndarray], tokens) -> tuple[np.ndarray, list[np.ndarray]]:
    """(logits [tokens, vocab], residual stream after every layer)."""
    eps = float(cfg["norm"]["eps"])
    x = w["embed"][np.asarray(tokens, dtype=np.int64)]
    residuals = []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        if layer["type"] != "attention":
            raise ValueError(f"unknown mixer {layer['type']!r}")
        x = x + rms(tied_attention(x, layer["mixer"], w, p + "mix.", eps), eps) * w[p + "norm1"]
        m = layer.get("mlp")
        if m is not None:
            y = swiglu(x, w, p + "mlp.") if m["kind"] == "dense" else mixture(x, m, w, p + "mlp.")
            x = x + rms(y, eps) * w[p + "norm2"]
        residuals.append(x)
    return (rms(x, eps) * w["final.norm"]) @ w["head"].T, residuals
