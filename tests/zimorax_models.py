"""Small Zimorax configurations with random weights for the tests (bf16-representable, so that a float64 oracle and both
runtime types start from the same numbers)."""
import numpy as np
import torch

from gutorax_models import row_errors, save_model  # noqa: F401  (shared helpers)


def attention(heads, kv_heads, dim, vdim, *, window=None, rot=None, base=10000.0, yarn=(4.0, 64.0, 8.0, 0.5), scale=None):
    """yarn: (factor, original, fast, slow); rot 0: no positions"""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": 1.3 * dim ** -0.5 if scale is None else scale}
    rot = dim // 2 * 2 if rot is None else rot
    if rot:
        m["rot"] = {"base": base, "dims": rot}
        if yarn:
            m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
    if window is not None:
        m["mask"] = {"size": window}
    return "attention", m


def mamba2(heads, vdim, state, *, groups=1, norm_groups=1, conv=4):
    return "mamba2", {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": norm_groups, "conv": conv}


def delta(heads, kv_heads, dim, vdim, *, conv=4):
    return "delta", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def config(width, vocab, layers, *, loop=None, eps=1e-5):
    """layers: ((type, mixer), ff or None) pairs; loop: (start, stop, times)."""
    cfg = {"architecture": "Zimorax", "norm": {"eps": eps}, "vocab": vocab, "width": width,
           "layers": [{"type": t, "mixer": m, "mlp": None if ff is None else {"kind": "dense", "ff": ff}} for (t, m), ff in layers]}
    if loop is not None:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


# fast: every tensor-core path; wide: many heads, one and many per key, large heads, long windows; odd: extents that none of them
# takes; ones: sizes equal to one
CONFIGS = {
    "fast": config(136, 168, [(mamba2(6, 40, 48, groups=3, norm_groups=2), 72), (attention(6, 2, 40, 24, window=37, rot=24), 56),
                              (delta(6, 2, 48, 24, conv=3), 40), (attention(4, 4, 64, 72, yarn=(8.0, 128.0, 4.0, 1.0)), None),
                              (mamba2(4, 16, 128, conv=2), 8), (delta(3, 3, 16, 72, conv=2), None)], loop=(1, 3, 2)),
    "wide": config(256, 96, [(attention(20, 1, 128, 128, window=70, rot=32, scale=0.02), 16), (delta(4, 1, 128, 256), 264), (mamba2(8, 64, 64, norm_groups=4), None),
                             (attention(8, 8, 64, 200, window=130, yarn=None), None), (delta(2, 2, 112, 8, conv=1), 24), (attention(2, 2, 256, 256, window=1), None)],
                   loop=(0, 2, 3)),
    "odd": config(90, 77, [(delta(3, 1, 10, 7, conv=5), 11), (attention(4, 2, 7, 11, window=13, rot=6, yarn=(2.0, 16.0, 2.0, 0.25)), 13),
                           (mamba2(5, 6, 12, groups=5, norm_groups=3, conv=3), 90), (attention(3, 3, 25, 9, window=50, rot=0), None),
                           (mamba2(2, 9, 20, groups=2, conv=6), None)], loop=(2, 5, 2)),
    "ones": config(16, 40, [(attention(1, 1, 2, 1, window=2, rot=2), 1), (mamba2(1, 1, 1, conv=1), 8), (delta(1, 1, 1, 1, conv=1), 1),
                            (mamba2(2, 8, 16, groups=2, conv=2), None), (delta(2, 1, 16, 8, conv=2), 16)], loop=(3, 4, 1)),
}


def random_weights(cfg, seed=0):
    """name -> float32 array of bf16 values."""
    from cacheir_b200.zimorax import ZimoraxConfig, build_zimorax_graph

    rng = np.random.default_rng(seed)
    out = {}
    for name, spec in build_zimorax_graph(ZimoraxConfig.from_dict(cfg)).weights.items():
        shape, last = spec.shape, name.split(".")[-1]
        if last == "A_log":
            a = rng.uniform(-3.0, 1.0, shape)           # long and short memories
        elif last == "dt_bias":
            a = rng.normal(-2.0, 1.0, shape)
        elif last in ("ls1", "ls2"):
            a = rng.uniform(0.2, 0.8, shape)
        elif "norm" in last:
            a = rng.uniform(0.5, 1.5, shape)
        elif last in ("conv", "step", "D"):
            a = rng.normal(0, 0.6, shape)
        elif last == "talk":
            a = np.eye(shape[0]) + rng.normal(0, 0.4 / np.sqrt(shape[0]), shape)
        elif len(shape) == 1:
            a = rng.normal(0, 0.3, shape)
        elif name == "embed":
            a = rng.normal(0, 1.0, shape)
        else:
            a = rng.normal(0, 1.1 / np.sqrt(shape[1]), shape)
        out[name] = torch.from_numpy(np.asarray(a, np.float32)).to(torch.bfloat16).float().numpy()
    return out
