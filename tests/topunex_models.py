"""Small Topunex configurations with random weights for the tests (bf16-representable, so that a float64 oracle and both
runtime types start from the same numbers)."""
import numpy as np
import torch

from gutorax_models import row_errors, save_model  # noqa: F401  (shared helpers)


def attention(heads, kv_heads, dim, *, size=None, keep=0, rot=None, base=10000.0, scale=None, cap=30.0, scaling=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": 1.4 * dim ** -0.5 if scale is None else scale,
         "rot": {"base": base, "dims": dim if rot is None else rot}, "mask": {"keep_first": keep}}
    if size is not None:
        m["mask"]["size"] = size
    if cap is not None:
        m["softcap"] = cap
    if scaling is not None:
        m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return m


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, *, limit=1.2, scale=1.5, shared=None, shared_limit=0.9):
    m = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top, "scale": scale}}
    if shared is not None:
        m["shared"] = {"ff": shared, "limit": shared_limit}
    return m


def config(width, vocab, layers, *, eps=1e-5):
    """layers: (mixer, mlp or None) pairs."""
    return {"architecture": "Topunex", "norm": {"eps": eps}, "vocab": vocab, "width": width,
            "layers": [{"type": "attention", "mixer": m, "mlp": f} for m, f in layers]}


# fast: every tensor-core path; wide: groups of one and of many heads, large heads; odd: extents none of them takes; ones:
# sizes equal to one
CONFIGS = {
    "fast": config(136, 168, [(attention(6, 2, 40, size=37, keep=3, rot=24), dense(104)),
                              (attention(4, 1, 64, size=130, keep=70, rot=64, base=500.0, scaling=(8.0, 1.0, 4.0, 64)), moe(7, 3, 24, shared=40)),
                              (attention(3, 3, 32, keep=0, rot=16, cap=None), moe(5, 1, 56)),
                              (attention(5, 5, 16, size=1, keep=2, rot=0, cap=4.0), None)]),
    "wide": config(256, 96, [(attention(20, 1, 128, size=100, keep=5, rot=32, cap=15.0), dense(72)),
                             (attention(4, 2, 256, size=70, keep=1, rot=128, scale=0.05), moe(12, 3, 16, shared=8)),
                             (attention(6, 3, 192, size=200, rot=96, scale=0.25, cap=60.0), moe(3, 3, 64, limit=0.5)),
                             (attention(34, 2, 72, size=90, keep=64, rot=72, scale=0.3, cap=None), None)]),
    "odd": config(90, 77, [(attention(3, 1, 10, size=13, keep=2, rot=6), dense(51)), (attention(4, 2, 7, size=50, rot=2, cap=5.0), moe(6, 2, 11, shared=5)),
                           (attention(1, 1, 25, keep=9, rot=24), None)]),
    "ones": config(16, 40, [(attention(1, 1, 2, size=2, keep=1, rot=2), dense(1)), (attention(2, 1, 8, size=100, rot=8), moe(1, 1, 1, shared=1)),
                            (attention(1, 1, 8, size=3, rot=0), moe(4, 4, 8))]),
}


def random_weights(cfg, seed=0):
    """name -> float32 array of bf16 values."""
    from cacheir_b200.topunex import TopunexConfig, build_topunex_graph

    rng = np.random.default_rng(seed)
    out = {}
    for name, spec in build_topunex_graph(TopunexConfig.from_dict(cfg)).weights.items():
        shape = spec.shape
        if name.endswith(".b"):
            a = rng.normal(0, 0.2, shape)
        elif name.endswith("sink"):
            a = rng.normal(1.0, 1.0, shape)
        elif "norm" in name.split(".")[-1]:
            a = rng.uniform(0.5, 1.5, shape)
        elif name == "embed":
            a = rng.normal(0, 1.0, shape)
        elif name.endswith("router"):
            a = rng.normal(0, 1.5 / np.sqrt(shape[1]), shape)
        else:
            a = rng.normal(0, 1.1 / np.sqrt(shape[1]), shape)
        out[name] = torch.from_numpy(np.asarray(a, np.float32)).to(torch.bfloat16).float().numpy()
    return out


def clear_choices(cfg, weights, tokens, margin):
    """Positions of `tokens` whose routers choose with at least `margin` between the last chosen and the next logit in every
    mixture (a rounding may swap closer ones, which moves the whole row)."""
    from oracle import topunex as O

    gaps = np.full(len(tokens), np.inf)
    plain = O.route

    def watched(z, top, scale):
        if top < z.shape[1]:
            s = -np.sort(-z, axis=-1)
            np.minimum(gaps, s[:, top - 1] - s[:, top], out=gaps)
        return plain(z, top, scale)
    O.route = watched
    try:
        logits, _ = O.forward(cfg, weights, tokens)
    finally:
        O.route = plain
    return logits, gaps >= margin
