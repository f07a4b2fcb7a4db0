"""Plain, slow NumPy statement of the Gutorax decoder -- TEST INFRASTRUCTURE ONLY.

One function per mechanism, whole sequences at a time, no cache, no batching and no code shared with the product
package. `forward` runs a token list through the model and returns logits and the residual stream after every layer.

Notation. X is [tokens, width]; a linear weight A is [out, in] and acts as X A^T. `cfg` is the parsed config.json,
`w` maps tensor names to arrays. Arithmetic runs in the dtype of `w` (float64 in the tests).
"""
from __future__ import annotations

from typing import Any, Mapping

import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def rms(x, eps):
    """x over its root mean square along the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def dynamic_tanh(x, w, name):
    """Elementwise squashing in place of a normalisation: w * tanh(alpha x) + b."""
    return np.tanh(w[name + ".alpha"] * x) * w[name] + w[name + ".b"]


def rotate_half(x, base, dims):
    """Rotary positions on the first `dims` entries of x [tokens, ..., d]; entry i turns with entry i + dims/2 by
    p * base^(-2i/dims), p = row number."""
    half = dims // 2
    i = np.arange(half, dtype=np.float64)
    p = np.arange(x.shape[0], dtype=np.float64)
    angle = p[:, None] * base ** (-2.0 * i / dims)
    shape = (x.shape[0],) + (1,) * (x.ndim - 2) + (half,)
    c, s = np.cos(angle).reshape(shape), np.sin(angle).reshape(shape)
    u, v = x[..., :half], x[..., half:dims]
    return np.concatenate([u * c - v * s, v * c + u * s, x[..., dims:]], axis=-1)


def latent_cache(h, m, w, prefix, eps):
    """(c, r): the normalised latent and the rotated key part shared by all heads, one row per token."""
    down = h @ w[prefix + "dkv"].T
    rank = int(m["kv_rank"])
    c = rms(down[:, :rank], eps) * w[prefix + "dkv.norm"]
    r = rotate_half(down[:, rank:], float(m["rot"]["base"]), int(m["rot"]["dims"]))
    return c, r


def windowed_sink_attention(q, k, v, scale, window, sink):
    """Causal attention [tokens, heads, *] over the last `window` tokens (the row's own included); one extra term
    exp(sink[head]) in each denominator."""
    n = q.shape[0]
    i = np.arange(n)
    gap = i[:, None] - i[None, :]
    seen = (gap >= 0) & (gap < window)
    out = np.empty((n, q.shape[1], v.shape[2]), dtype=q.dtype)
    for head in range(q.shape[1]):
        score = np.where(seen, (q[:, head] @ k[:, head].T) * scale, -np.inf)
        top = np.maximum(score.max(axis=1), sink[head])
        e = np.exp(score - top[:, None])
        out[:, head] = (e @ v[:, head]) / (e.sum(axis=1) + np.exp(sink[head] - top))[:, None]
    return out


def latent_attention(h, m, w, prefix, cached, eps):
    """Attention whose keys and values are linear in a cached latent; `cached` = (c, r) of this layer or of the layer
    it borrows them from."""
    n = h.shape[0]
    heads, dim, rot, vdim = (int(m[k]) for k in ("heads", "dim", "rot_dim", "vdim"))
    c, r = cached
    q = (h @ w[prefix + "q"].T).reshape(n, heads, dim + rot)
    q = np.concatenate([q[..., :dim], rotate_half(q[..., dim:], float(m["rot"]["base"]), int(m["rot"]["dims"]))], axis=-1)
    k = (c @ w[prefix + "uk"].T).reshape(n, heads, dim)
    k = np.concatenate([k, np.broadcast_to(r[:, None, :], (n, heads, rot))], axis=-1)
    v = (c @ w[prefix + "uv"].T).reshape(n, heads, vdim)
    o = windowed_sink_attention(q, k, v, float(m["scale"]), int(m["mask"]["size"]), w[prefix + "sink"])
    o = o.reshape(n, heads * vdim) * sigmoid(h @ w[prefix + "g"].T)
    return o @ w[prefix + "o"].T


def decayed_outer_recurrence(q, k, v, decay, state=None):
    """Per head S <- decay S + k v^T, o = S^T q, token by token. q, k [tokens, heads, d], v [tokens, heads, e]."""
    n, heads, d = q.shape
    state = np.zeros((heads, d, v.shape[2]), dtype=q.dtype) if state is None else state.copy()
    out = np.empty_like(v)
    decay = np.asarray(decay, dtype=q.dtype)[:, None, None]
    for t in range(n):
        state = decay * state + k[t][:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hde,hd->he", state, q[t])
    return out, state


def lightning(h, m, w, prefix, eps):
    n = h.shape[0]
    heads, dim, vdim = (int(m[k]) for k in ("heads", "dim", "vdim"))
    q = silu(h @ w[prefix + "q"].T).reshape(n, heads, dim)
    k = silu(h @ w[prefix + "k"].T).reshape(n, heads, dim)
    v = silu(h @ w[prefix + "v"].T).reshape(n, heads, vdim)
    o, _ = decayed_outer_recurrence(q, k, v, m["decay"])
    o = rms(o.reshape(n, heads * vdim), eps) * w[prefix + "norm"]
    return (o * sigmoid(h @ w[prefix + "g"].T)) @ w[prefix + "o"].T


def feed_forward(h, w, prefix):
    return (gelu_tanh(h @ w[prefix + "gate"].T) * (h @ w[prefix + "up"].T)) @ w[prefix + "down"].T


def token_side_input(x, tokens, w, layer, prefix, dim, eps):
    """Second embedding table, one `dim`-wide part per layer, let in through a gate computed from the residual."""
    e = w["side.embed"][tokens, layer * dim:(layer + 1) * dim]
    y = (gelu_tanh(x @ w[prefix + "gate"].T) * e) @ w[prefix + "proj"].T
    return x + rms(y, eps) * w[prefix + "norm"]


def forward(cfg: Mapping[str, Any], w: Mapping[str, np.ndarray], tokens) -> tuple[np.ndarray, list[np.ndarray]]:
    """(logits [tokens, vocab], residual stream after every layer)."""
    tokens = np.asarray(tokens, dtype=np.int64)
    eps = float(cfg["norm"]["eps"])
    x = w["embed"][tokens] * float(cfg["embedding"]["scale"])
    caches: dict[int, tuple[np.ndarray, np.ndarray]] = {}
    residuals = []
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = dynamic_tanh(x, w, p + "norm1")
        if layer["type"] == "latent_attention":
            source = m.get("kv_from")
            if source is None:
                caches[i] = latent_cache(h, m, w, p + "mix.", eps)
                source = i
            y = latent_attention(h, m, w, p + "mix.", caches[int(source)], eps)
        elif layer["type"] == "lightning":
            y = lightning(h, m, w, p + "mix.", eps)
        else:
            raise ValueError(f"unknown mixer {layer['type']!r}")
        x = x + dynamic_tanh(y, w, p + "norm1b")
        if layer.get("mlp") is not None:
            x = x + dynamic_tanh(feed_forward(dynamic_tanh(x, w, p + "norm2"), w, p + "mlp."), w, p + "norm2b")
        if cfg.get("token_side"):
            x = token_side_input(x, tokens, w, i, p + "side.", int(cfg["token_side"]["dim"]), eps)
        residuals.append(x)
    return dynamic_tanh(x, w, "final.norm") @ w["head"].T, residuals
