"""Small Gutorax configurations with random weights for the tests (bf16-representable, so that a float64 oracle and both
runtime types start from the same numbers)."""
import json
import struct

import numpy as np
import torch


def latent(heads, dim, rot, vdim, rank, window, *, base=10000.0, scale=None, kv_from=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "mask": {"size": window},
         "rot": {"base": base, "dims": rot}, "scale": (dim + rot) ** -0.5 if scale is None else scale}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return "latent_attention", m


def lightning(heads, dim, vdim, decay=None):
    return "lightning", {"heads": heads, "dim": dim, "vdim": vdim,
                         "decay": [1.0 - 2.0 ** -(1 + h) for h in range(heads)] if decay is None else list(decay)}


def config(width, vocab, layers, *, side=16, scale=4.0, eps=1e-5):
    """layers: ((type, mixer), ff or None) pairs."""
    cfg = {"architecture": "Gutorax", "embedding": {"scale": scale}, "norm": {"eps": eps}, "vocab": vocab, "width": width,
           "layers": [{"type": t, "mixer": m, "mlp": None if ff is None else {"kind": "dense", "ff": ff}} for (t, m), ff in layers]}
    if side is not None:
        cfg["token_side"] = {"dim": side}
    return cfg


# fast: every bf16 tensor-core path; odd: extents none of them takes; ones: sizes equal to one
CONFIGS = {
    "fast": config(128, 160, [(latent(5, 24, 16, 40, 48, 9), 96), (lightning(3, 32, 72), 200),
                              (latent(2, 8, 16, 16, 48, 70, kv_from=0), None), (lightning(4, 16, 24, [1.0, 0.5, 0.97, 0.0]), 64)], side=24),
    "wide_latent": config(192, 96, [(lightning(2, 128, 64), 64), (latent(20, 32, 64, 64, 256, 130, base=500.0), 128),
                                    (latent(33, 16, 64, 32, 256, 65, base=500.0, kv_from=1), 96), (latent(3, 16, 8, 16, 16, 1), None)], side=8),
    "odd": config(90, 77, [(latent(3, 10, 6, 14, 20, 13), 50), (lightning(5, 12, 18), 30), (latent(1, 7, 6, 5, 20, 40, kv_from=0), 33),
                           (lightning(1, 20, 7), None)], side=10),
    "ones": config(16, 40, [(lightning(1, 1, 1, [0.75]), 8), (latent(1, 1, 2, 1, 1, 2), 1), (latent(1, 16, 8, 16, 16, 100), 16)], side=1),
    "no_side": config(64, 64, [(latent(4, 16, 32, 16, 32, 33), 64), (lightning(2, 48, 40), None)], side=None, scale=1.0, eps=1e-3),
}


def random_weights(cfg, seed=0):
    """name -> float32 array of bf16 values."""
    from cacheir_b200.gutorax import GutoraxConfig, build_gutorax_graph

    rng = np.random.default_rng(seed)
    out = {}
    for name, spec in build_gutorax_graph(GutoraxConfig.from_dict(cfg)).weights.items():
        shape = spec.shape
        if name.endswith(".alpha"):
            a = rng.uniform(0.4, 1.2, shape)
        elif name.endswith(".b"):
            a = rng.normal(0, 0.1, shape)
        elif name.endswith("sink"):
            a = rng.normal(0.5, 1.0, shape)
        elif "norm" in name.split(".")[-1]:
            a = rng.uniform(0.5, 1.5, shape)
        elif name in ("embed", "side.embed"):
            a = rng.normal(0, 0.5, shape)
        else:
            gain = 1.7 if name.endswith(("mix.q", "mix.uk", "mix.dkv")) else 1.2      # sharp scores: single keys matter
            a = rng.normal(0, gain / np.sqrt(shape[1]), shape)
        out[name] = torch.from_numpy(np.asarray(a, np.float32)).to(torch.bfloat16).float().numpy()
    return out


def save_model(folder, cfg, weights):
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(cfg))
    header, blobs, off = {}, [], 0
    for name, a in weights.items():
        raw = torch.from_numpy(np.array(a)).to(torch.bfloat16).view(torch.int16).numpy().tobytes()
        header[name] = {"dtype": "BF16", "shape": list(a.shape), "data_offsets": [off, off + len(raw)]}
        blobs.append(raw)
        off += len(raw)
    head = json.dumps(header).encode()
    (folder / "model.safetensors").write_bytes(struct.pack("<Q", len(head)) + head + b"".join(blobs))
    return folder


def row_errors(got, want):
    """Per row: rms of the difference over the rms of all expected rows (means taken off)."""
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    d = got - want
    d -= d.mean(axis=-1, keepdims=True)
    return np.sqrt((d ** 2).mean(axis=-1)) / np.sqrt(((want - want.mean(axis=-1, keepdims=True)) ** 2).mean())
