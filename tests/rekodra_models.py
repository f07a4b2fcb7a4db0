"""Small Rekodra configurations with random weights for the tests (bf16-representable, so that a float64 oracle and both
runtime types start from the same numbers)."""
import numpy as np
import torch

from gutorax_models import row_errors, save_model  # noqa: F401  (shared helpers)


def attention(heads, kv_heads, dim, *, rot=None, base=10000.0, scale=None):
    return "attention", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": 1.4 * dim ** -0.5 if scale is None else scale,
                         "rot": {"base": base, "dims": dim if rot is None else rot}}


def parallel(left, right, *, scale=None):
    """left: (heads, kv_heads, dim, vdim, window), right: (heads, dim, vdim, gate cap)"""
    names = (("heads", "kv_heads", "dim", "vdim"), ("heads", "dim", "vdim", "gate_cap"))
    sides = [dict(zip(n, v)) for n, v in zip(names, (left[:4], right))]
    sides[0].update(mask={"size": left[4]}, scale=1.3 * left[2] ** -0.5 if scale is None else scale)
    return "parallel", {"left": sides[0], "right": sides[1]}


def moe(experts, top, ff, *, identity=1, groups=(1, 1), shared=None):
    router = {"experts": experts, "top": top, "identity": identity, "groups": {"count": groups[0], "keep": groups[1]}}
    m = {"kind": "moe", "expert": {"ff": ff}, "router": router}
    if shared is not None:
        m["shared"] = {"ff": shared}
    return m


def config(width, vocab, layers, *, loop=None, embed=0.7, logit=0.6, eps=1e-5):
    """layers: ((type, mixer), mlp or None) pairs; loop: (start, stop, times)."""
    cfg = {"architecture": "Rekodra", "norm": {"eps": eps}, "vocab": vocab, "width": width, "embedding": {"scale": embed}, "logit_scale": logit,
           "layers": [{"type": t, "mixer": m, "mlp": f} for (t, m), f in layers]}
    if loop is not None:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


# fast: every tensor-core path; wide: groups of one and of many heads, large heads, long windows; odd: extents none of them
# takes; ones: sizes equal to one
CONFIGS = {
    "fast": config(136, 168, [(parallel((6, 2, 40, 24, 37), (3, 32, 72, 9.0)), moe(10, 3, 24, identity=2, groups=(4, 2), shared=40)),
                              (attention(6, 2, 40, rot=24), moe(5, 2, 56, identity=0)),
                              (parallel((3, 3, 16, 64, 130), (5, 48, 16, 3.0)), None),
                              (attention(4, 1, 64, base=500.0), moe(6, 4, 32, identity=3, groups=(3, 2), shared=8))], loop=(0, 3, 2)),
    "wide": config(256, 96, [(attention(20, 1, 128, rot=32), moe(12, 3, 16, identity=4, groups=(2, 1), shared=72)),
                             (parallel((4, 1, 128, 200, 70), (2, 128, 64, 15.0), scale=0.05), moe(3, 3, 64, identity=0)),
                             (parallel((2, 2, 256, 256, 1), (1, 64, 128, 5.0)), None), (attention(3, 3, 192, rot=0, scale=0.2), None)],
                   loop=(1, 2, 3), embed=1.0, logit=1.0),
    "odd": config(90, 77, [(attention(3, 1, 10, rot=6), moe(5, 2, 11, identity=1, groups=(3, 2), shared=5)),
                           (parallel((4, 2, 7, 11, 13), (5, 12, 18, 2.0)), moe(6, 2, 13, identity=2, groups=(2, 2))),
                           (parallel((1, 1, 25, 3, 50), (1, 20, 7, 8.0)), None)], loop=(0, 3, 2)),
    "ones": config(16, 40, [(attention(1, 1, 2, rot=2), moe(1, 1, 1, identity=0, shared=1)),
                            (parallel((2, 1, 8, 1, 2), (1, 1, 1, 0.5)), moe(1, 2, 1, identity=3, groups=(4, 4))),
                            (parallel((1, 1, 1, 8, 100), (2, 16, 8, 30.0)), moe(4, 4, 8, identity=0))], loop=(2, 3, 1)),
}


def random_weights(cfg, seed=0):
    """name -> float32 array of bf16 values."""
    from cacheir_b200.rekodra import RekodraConfig, build_rekodra_graph

    rng = np.random.default_rng(seed)
    out = {}
    for name, spec in build_rekodra_graph(RekodraConfig.from_dict(cfg)).weights.items():
        shape, last = spec.shape, name.split(".")[-1]
        if name.endswith("i.b"):
            a = rng.normal(0.0, 1.5, shape)
        elif name.endswith("f.b"):
            a = rng.uniform(0.0, 6.0, shape)          # short and long memories
        elif name.endswith("correction"):
            a = rng.normal(0, 0.4, shape)
        elif last == "sink":
            a = rng.normal(1.0, 1.0, shape)
        elif "norm" in last or last == "out":
            a = rng.uniform(0.5, 1.5, shape)
        elif name == "embed":
            a = rng.normal(0, 1.0, shape)
        elif last == "router":
            a = rng.normal(0, 1.5 / np.sqrt(shape[1]), shape)
        else:
            a = rng.normal(0, 1.1 / np.sqrt(shape[1]), shape)
        out[name] = torch.from_numpy(np.asarray(a, np.float32)).to(torch.bfloat16).float().numpy()
    return out


def clear_choices(cfg, weights, tokens, margin):
    """(logits, positions whose routers choose with at least `margin` between the last chosen and the next choice score, and
    between the last kept and the next group, in every mixture). A rounding may swap closer ones, which moves the whole row."""
    from oracle import rekodra as O

    gaps = np.full(len(tokens), np.inf)
    plain = O.route

    def watched(z, correction, top, groups=1, keep=1):
        choice = O.softmax(z) + correction
        best = choice.reshape(len(z), groups, -1).max(axis=-1)
        order = -np.sort(-best, axis=-1)
        if keep < groups:
            np.minimum(gaps, order[:, keep - 1] - order[:, keep], out=gaps)
        inside = np.repeat(best >= order[:, keep - 1:keep], z.shape[1] // groups, axis=1)
        s = -np.sort(-np.where(inside, choice, -np.inf), axis=-1)
        if top < z.shape[1]:
            np.minimum(gaps, s[:, top - 1] - s[:, top], out=gaps)
        return plain(z, correction, top, groups, keep)
    O.route = watched
    try:
        logits, _ = O.forward(cfg, weights, tokens)
    finally:
        O.route = plain
    return logits, gaps >= margin
