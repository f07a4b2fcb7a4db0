"""`bench.py --family gutorax|topunex|rekodra|zimorax`: prefill and decode throughput of a ragged family beside the other ones at equal
width, (active) feed-forward, heads and layer count (random weights), and every kernel's distance from its roofline.

Throughput: decode is `decode_greedy_batch` (CUDA-graph replay, argmax fed back on the device) over `batch` sequences
with `ctx` cached tokens; prefill is one prompt through the runtime's own entry point, with the last position's logits
wanted where the runtime lets a caller say so. Kernel times: all launches of one kind in a step (every layer's, so that
weights and caches come from HBM) as one CUDA graph, timed with events; the roofline is the larger of algorithmic bytes
over the measured copy bandwidth and FLOPs over the measured bf16 rate, summed over the same launches.
"""
from __future__ import annotations

from collections import defaultdict

SIZES = {
    # width, ff, heads, kv_heads, head dim, latent rank, rotated dims, window, layers, vocab; mixtures (every second Topunex
    # layer, every Rekodra layer): top experts and the shared one add up to ff
    "4096": dict(width=4096, ff=14336, heads=32, kv_heads=8, dim=128, rank=512, rot=64, window=4096, layers=8, vocab=32768, side=256,
                 experts=32, top=4, expert_ff=1792, shared_ff=7168, keep=4),
    "2048": dict(width=2048, ff=5632, heads=16, kv_heads=8, dim=128, rank=256, rot=64, window=1024, layers=12, vocab=32768, side=128,
                 experts=32, top=4, expert_ff=704, shared_ff=2816, keep=4),
}


def gutorax_config(s: dict) -> dict:
    """Layers in groups of four: latent attention, recurrence, latent attention on the first one's cache, recurrence."""
    layers = []
    for i in range(s["layers"]):
        if i % 2:
            t, m = "lightning", {"heads": s["heads"], "dim": s["dim"], "vdim": s["dim"], "decay": [1 - 2.0 ** -(2 + h * 8 / s["heads"]) for h in range(s["heads"])]}
        else:
            t, m = "latent_attention", {"heads": s["heads"], "dim": s["dim"], "rot_dim": s["rot"], "vdim": s["dim"], "kv_rank": s["rank"],
                                        "scale": (s["dim"] + s["rot"]) ** -0.5, "mask": {"size": s["window"]},
                                        "rot": {"base": 500000.0, "dims": s["rot"]}}
            if i % 4 == 2:
                m["kv_from"] = i - 2
        layers.append({"type": t, "mixer": m, "mlp": {"kind": "dense", "ff": s["ff"]}})
    return {"architecture": "Gutorax", "width": s["width"], "vocab": s["vocab"], "embedding": {"scale": s["width"] ** 0.5},
            "norm": {"eps": 1e-5}, "token_side": {"dim": s["side"]}, "layers": layers}


def topunex_config(s: dict) -> dict:
    """Dense layers and mixtures of experts in turn."""
    mixer = {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": s["dim"], "vdim": s["dim"], "scale": s["dim"] ** -0.5, "softcap": 30.0,
             "mask": {"size": s["window"], "keep_first": s["keep"]},
             "rot": {"base": 500000.0, "dims": s["rot"], "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}}
    moe = {"kind": "moe", "expert": {"ff": s["expert_ff"], "limit": 7.0}, "shared": {"ff": s["shared_ff"], "limit": 7.0},
           "router": {"experts": s["experts"], "top": s["top"], "scale": 2.0}}
    return {"architecture": "Topunex", "width": s["width"], "vocab": s["vocab"], "norm": {"eps": 1e-6},
            "layers": [{"type": "attention", "mixer": mixer, "mlp": moe if i % 2 else {"kind": "dense", "ff": s["ff"]}} for i in range(s["layers"])]}


def rekodra_config(s: dict) -> dict:
    """Attention over all tokens, and window attention beside matrix memory with half of the heads each, in turn. An eighth of the
    router's outputs are identity experts."""
    half = s["heads"] // 2
    full = {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": s["dim"], "vdim": s["dim"], "scale": s["dim"] ** -0.5,
            "rot": {"base": 500000.0, "dims": s["rot"]}}
    both = {"left": {"heads": half, "kv_heads": s["kv_heads"], "dim": s["dim"], "vdim": s["dim"], "scale": s["dim"] ** -0.5, "mask": {"size": s["window"]}},
            "right": {"heads": half, "dim": s["dim"], "vdim": s["dim"], "gate_cap": 15.0}}
    moe = {"kind": "moe", "expert": {"ff": s["expert_ff"]}, "shared": {"ff": s["shared_ff"]},
           "router": {"experts": s["experts"] * 7 // 8, "identity": s["experts"] // 8, "top": s["top"], "groups": {"count": 4, "keep": 2}}}
    return {"architecture": "Rekodra", "width": s["width"], "vocab": s["vocab"], "norm": {"eps": 1e-6}, "embedding": {"scale": 1.0}, "logit_scale": 1.0,
            "layers": [{"type": "parallel", "mixer": both, "mlp": moe} if i % 2 else {"type": "attention", "mixer": full, "mlp": moe}
                       for i in range(s["layers"])]}


def zimorax_shape(s: dict, i: int) -> dict:
    """Mixer sizes of layer i: talking-heads attention, a state space of twice the width, a delta rule with a key head per two heads,
    in turn."""
    if i % 3 == 0:
        return {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": s["dim"], "vdim": s["dim"]}
    if i % 3 == 1:
        return {"heads": 2 * s["width"] // 64, "vdim": 64, "state": 128, "groups": 8, "norm_groups": 8, "conv": 4}
    return {"heads": s["heads"], "kv_heads": s["heads"] // 2, "dim": s["dim"], "vdim": s["dim"], "conv": 4}


def zimorax_config(s: dict) -> dict:
    """Feed-forward layers without a gate have 3/2 of the width, so that their weights are as many."""
    layers = []
    for i in range(s["layers"]):
        m = zimorax_shape(s, i)
        if i % 3 == 0:
            m.update(scale=s["dim"] ** -0.5, mask={"size": s["window"]},
                     rot={"base": 500000.0, "dims": s["rot"], "scaling": {"factor": 8.0, "original": 8192, "fast": 32.0, "slow": 1.0}})
        layers.append({"type": ("attention", "mamba2", "delta")[i % 3], "mixer": m, "mlp": {"kind": "dense", "ff": s["ff"] * 3 // 2}})
    return {"architecture": "Zimorax", "width": s["width"], "vocab": s["vocab"], "norm": {"eps": 1e-6}, "layers": layers}


def synthetic(device):
    import zlib

    import torch
    gen = torch.Generator(device=device)

    def make(key: str, shape: tuple[int, ...]):
        if len(shape) == 1 and key.endswith((".q.b", ".k.b", ".o.b", ".gate.b", ".up.b", ".down.b")):
            return torch.zeros(shape, device=device)      # (a constant added to every token would send them all to the same experts)
        if key.endswith(("mix.right.i.b", "mlp.correction")):
            return torch.zeros(shape, device=device)
        if key.endswith("mix.right.f.b"):
            return torch.full(shape, 4.0, device=device)
        if key.endswith(".talk"):
            return torch.eye(shape[0], device=device) + 0.02
        if key.endswith(("dt_bias", "A_log")):
            return torch.full(shape, -2.0, device=device)
        if len(shape) <= 1:
            return torch.full(shape, 0.6 if key.endswith("alpha") else 1.0, device=device)
        gen.manual_seed(zlib.crc32(key.encode()))
        return torch.randn(shape, device=device, generator=gen) * 0.02
    return make


def build(family: str, s: dict, *, batch: int, positions: int):
    import torch

    from cacheir_b200 import (B200DecodeRuntime, B200KVPageAllocator, GutoraxConfig, ModelConfig, build_decoder_artifact,
                              RekodraConfig, TopunexConfig, ZimoraxConfig, build_gutorax_artifact, build_rekodra_artifact, build_topunex_artifact,
                              build_zimorax_artifact)
    dev = torch.device("cuda", torch.cuda.current_device())
    if family == "gutorax":
        art, page = build_gutorax_artifact(GutoraxConfig.from_dict(gutorax_config(s))), 64
        dtype = "bfloat16"
    elif family == "topunex":
        art, page, dtype = build_topunex_artifact(TopunexConfig.from_dict(topunex_config(s))), 64, "bfloat16"
    elif family == "rekodra":
        art, page, dtype = build_rekodra_artifact(RekodraConfig.from_dict(rekodra_config(s))), 64, "bfloat16"
    elif family == "zimorax":
        art, page, dtype = build_zimorax_artifact(ZimoraxConfig.from_dict(zimorax_config(s))), 64, "bfloat16"
    else:
        art = build_decoder_artifact(ModelConfig(
            architecture="LlamaForCausalLM", hidden_size=s["width"], intermediate_size=s["ff"], num_layers=s["layers"],
            num_attention_heads=s["heads"], num_key_value_heads=s["kv_heads"], vocab_size=s["vocab"], max_position_embeddings=positions,
            rope_theta=500000.0, dtype="float16"), quant="int8", modes=("decode",))
        page, dtype = 16, "float16"
    alloc = B200KVPageAllocator(page_size=page, initial_slots=(batch + 1) * ((positions + page - 1) // page), initial_states=batch + 1)
    return B200DecodeRuntime(art, dtype=dtype, tensor_source=synthetic(dev), kv_allocator=alloc, max_seq_len=positions, clone_outputs=False)


def fill(rt, batch: int, ctx: int):
    """`batch` sessions with `ctx` cached tokens of synthetic content."""
    sessions = [rt.fork() for _ in range(batch)]
    for s in sessions:
        s.kv_cache.extend(ctx)
    for pool in rt.kv_allocator._pools.values():
        for name, t in pool.items():
            t.fill_(1.0) if name == "inv_rms" else t.normal_()
    for state in rt.kv_allocator._states.values():
        state.normal_()            # (a matrix memory's maxima and normalisers too: any values do)
    return sessions


def timed(fn, iters: int) -> float:
    """Milliseconds per call on the device."""
    import torch
    for _ in range(3):
        fn()
    start, stop = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    torch.cuda.synchronize()
    start.record()
    for _ in range(iters):
        fn()
    stop.record()
    torch.cuda.synchronize()
    return start.elapsed_time(stop) / iters


def kind_times(plan, iters: int = 5) -> dict[str, tuple[int, float]]:
    """kind -> (launch groups per step, microseconds per step)."""
    import torch
    groups: dict[str, list] = defaultdict(list)
    for fn, (key, _) in zip(plan.program, plan._count_keys):
        if key != "b200.advance_positions":
            groups[key].append(fn)
    out = {}
    for key, fns in groups.items():
        graph = torch.cuda.CUDAGraph()
        for fn in fns:
            fn()
        torch.cuda.synchronize()
        with torch.cuda.graph(graph):
            for _ in range(2):
                for fn in fns:
                    fn()
        out[key] = (len(fns), timed(graph.replay, iters) * 1e3 / 2)
    return out


def gutorax_work(s: dict, rows: int, logit_rows: int, keys_per_row: float, cached_rows: float, decode: bool) -> dict[str, list[tuple[float, float]]]:
    """kind -> (bytes, FLOPs) of every launch. `keys_per_row`: cache rows a token attends to on average; `cached_rows`:
    distinct cache rows of the step."""
    w, ff, h, d, rank, rot, side = s["width"], s["ff"], s["heads"], s["dim"], s["rank"], s["rot"], s["side"]
    work: dict[str, list[tuple[float, float]]] = defaultdict(list)

    def gemm(kind, n, k, n_out, t=rows, extra=0.0):
        work["b200.dense_gemm" + kind].append((2.0 * (n * k + t * k + t * n_out) + extra, 2.0 * t * n * k))

    for i in range(s["layers"]):
        if i % 2:
            gemm(".silu", 4 * h * d, w, 4 * h * d)
            state = rows * h * d * d * 4.0 * 2 if decode else h * d * d * 4.0 * 2
            io = rows * h * d * 4 * 2.0
            work["b200.recurrence_step" if decode else "b200.recurrence_chunked"].append((state + io, rows * h * 4.0 * d * d))
            work["b200.gated_rms"].append((rows * h * d * 3 * 2.0, 0.0))
        else:
            own = i % 4 == 0
            n = h * (d + rot) + (rank + rot if own else 0) + h * d
            gemm("", n, w, n)
            work["b200.latent_prepare"].append((rows * (h * rot * 2 + (2 * (rank + rot) if own else 0)) * 2.0, 0.0))
            work["b200.dense_gemm.heads"].append((2.0 * (h * rank * d + rows * h * (d + rank)), 2.0 * rows * h * rank * d))
            work["b200.latent_attention"].append((2.0 * (cached_rows * (rank + rot) + rows * h * (2 * rank + rot)),
                                                  2.0 * rows * h * keys_per_row * (2 * rank + rot)))
            work["b200.dense_gemm.heads_gated"].append((2.0 * (h * rank * d + rows * h * (rank + 2 * d)), 2.0 * rows * h * rank * d))
        gemm(".residual_dyt", w, h * d, 0, extra=rows * w * (8 + 2))
        gemm(".geglu", 2 * ff, w, ff)
        gemm(".residual_dyt", w, ff, 0, extra=rows * w * (8 + 2))
        gemm(".gelu_embed", side, w, 2 * side)
        gemm(".side", w, side, w)
        work["b200.residual_rms"].append((rows * w * (2 + 8 + 2.0), 0.0))
    work["b200.scaled_embedding"].append((rows * w * (2 + 4 + 2.0), 0.0))
    work["b200.dyt_rows"].append((logit_rows * w * 6.0, 0.0))
    gemm(".lm_head", s["vocab"], w, 2 * s["vocab"], t=logit_rows)
    return work


def topunex_work(s: dict, rows: int, logit_rows: int, keys_per_row: float, cached_rows: float, decode: bool, touched: int) -> dict[str, list[tuple[float, float]]]:
    """`touched`: experts with at least one token."""
    w, ff, h, g, d, rot = s["width"], s["ff"], s["heads"], s["kv_heads"], s["dim"], s["rot"]
    work: dict[str, list[tuple[float, float]]] = defaultdict(list)

    def gemm(kind, n, k, n_out, t=rows, weights=1.0):
        work["b200." + kind].append((2.0 * (weights * n * k + t * k + t * n_out), 2.0 * t * n * k))

    qw = d + rot - rot // 64 * 64
    for i in range(s["layers"]):
        n = (2 * h + g) * d
        gemm("dense_gemm", n, w, n)
        work["b200.tied_prepare"].append((2.0 * rows * (h * (d + qw) + g * (2 * d + rot)), 0.0))
        work["b200.tied_attention_step" if decode else "b200.tied_attention_prompt"].append(
            (cached_rows * g * (2.0 * (d + rot) + 4) + 2.0 * rows * h * (qw + 2 * d), 4.0 * rows * h * keys_per_row * d))
        gemm("dense_gemm.o", w, h * d, w)
        work["b200.residual_rms"].append((rows * w * (2 + 8 + 2.0), 0.0))
        if i % 2:
            places = rows * s["top"]
            gemm("dense_gemm.clamped_glu", 2 * s["shared_ff"] + s["experts"], w, s["shared_ff"])
            gemm("dense_gemm.down", w, s["shared_ff"], w)
            work["b200.route"].append((rows * (s["experts"] * 4.0 + s["top"] * 16), 0.0))
            gemm("grouped_gemm.clamped_glu", 2 * s["expert_ff"], w, s["expert_ff"], t=places, weights=touched)
            gemm("grouped_gemm", w, s["expert_ff"], w, t=places, weights=touched)
            work["b200.combine_residual_rms"].append((rows * w * (2 * s["top"] + 2 + 8 + 2.0), 0.0))
        else:
            gemm("dense_gemm.swiglu", 2 * ff, w, ff)
            gemm("dense_gemm.down", w, ff, w)
            work["b200.residual_rms"].append((rows * w * (2 + 8 + 2.0), 0.0))
    work["b200.scaled_embedding"].append((rows * w * (2 + 4 + 2.0), 0.0))
    work["b200.rms_rows"].append((logit_rows * w * 6.0, 0.0))
    gemm("dense_gemm.lm_head", s["vocab"], w, 2 * s["vocab"], t=logit_rows)
    return work


def rekodra_work(s: dict, rows: int, logit_rows: int, span: int, decode: bool, touched: int, places: int) -> dict[str, list[tuple[float, float]]]:
    """`span`: tokens a decoded row has seen, or the prompt's; `touched`: experts with at least one token, `places`: their rows."""
    w, h, g, d, rot = s["width"], s["heads"], s["kv_heads"], s["dim"], s["rot"]
    half, scored = h // 2, s["experts"]
    work: dict[str, list[tuple[float, float]]] = defaultdict(list)

    def gemm(kind, n, k, n_out, t=rows, weights=1.0):
        work["b200." + kind].append((2.0 * (weights * n * k + t * k + t * n_out), 2.0 * t * n * k))

    def attention(heads, width, qw, window):
        keys = min(span, window) if decode else sum(min(i + 1, window) for i in range(span)) / span
        cached = rows * keys if decode else span
        work["b200.tied_prepare"].append((2.0 * rows * (heads * (d + qw) + g * (2 * width - rot if width < 2 * d else 2 * width)), 0.0))
        work["b200.tied_attention_step" if decode else "b200.tied_attention_prompt"].append(
            (cached * g * (2.0 * width + 4) + 2.0 * rows * heads * (qw + d), 2.0 * rows * heads * keys * (qw + d)))

    for i in range(s["layers"]):
        if i % 2:
            n = (half + 2 * g) * d + 4 * half * d + 2 * half
            gemm("dense_gemm", n, w, n)
            attention(half, 2 * d, d, s["window"])
            gemm("dense_gemm.o", w, half * d, w)
            io = rows * half * d * 2.0
            state = half * d * (d + 1) * 8.0
            if decode:
                work["b200.memory_step"].append((rows * state + 5 * io, rows * half * 4.0 * d * d))
            else:
                work["b200.memory_gates"].append((rows * half * 20.0, 0.0))
                work["b200.recurrence_chunked"].append((state + 4 * io, rows * half * 4.0 * d * d))
                work["b200.memory_norm"].append((3 * io, 0.0))
            gemm("dense_gemm.o", w, half * d, w)
            work["b200.residual_rms_pair"].append((rows * w * (4 + 8 + 2.0), 0.0))
        else:
            n = (h + g) * d
            gemm("dense_gemm", n, w, n)
            attention(h, d + rot, d + rot - rot // 64 * 64, 1 << 30)
            gemm("dense_gemm.o", w, h * d, w)
            work["b200.residual_add"].append((rows * w * (2 + 8 + 2.0), 0.0))
        gemm("dense_gemm.swiglu", 2 * s["shared_ff"] + scored + 1, w, s["shared_ff"])
        gemm("dense_gemm.down", w, s["shared_ff"], w)
        work["b200.route"].append((rows * (scored * 4.0 + s["top"] * 16) + (0 if decode else 2.0 * w * (rows + places)), 0.0))
        gemm("grouped_gemm.swiglu", 2 * s["expert_ff"], w, s["expert_ff"], t=places, weights=touched)
        gemm("grouped_gemm", w, s["expert_ff"], w, t=places, weights=touched)
        work["b200.combine_residual"].append((2.0 * places * w + rows * w * (2 + 2 + 8 + 2.0), 0.0))
    work["b200.scaled_embedding"].append((rows * w * (2 + 4 + 2.0), 0.0))
    work["b200.rms_rows"].append((logit_rows * w * 6.0, 0.0))
    gemm("dense_gemm.lm_head", s["vocab"], w, 2 * s["vocab"], t=logit_rows)
    return work


def zimorax_work(s: dict, rows: int, logit_rows: int, keys_per_row: float, cached_rows: float, decode: bool) -> dict[str, list[tuple[float, float]]]:
    """Talking heads: the mixture of scores counts as heads^2 multiplications per key, whatever form a kernel gives it."""
    w, ff = s["width"], s["ff"] * 3 // 2
    work: dict[str, list[tuple[float, float]]] = defaultdict(list)

    def gemm(kind, n, k, n_out, t=rows):
        work["b200.dense_gemm" + kind].append((2.0 * (n * k + t * k + t * n_out), 2.0 * t * n * k))

    for i in range(s["layers"]):
        m = zimorax_shape(s, i)
        h, e = m["heads"], m["vdim"]
        io = rows * h * e * 2.0
        if i % 3 == 0:
            g, d = m["kv_heads"], m["dim"]
            n = h * d + g * (d + e)
            gemm("", n, w, n)
            work["b200.talking_prepare"].append((2.0 * rows * 2 * n, 0.0))
            work["b200.talking_step" if decode else "b200.talking_prompt"].append(
                (2.0 * (cached_rows * g * (d + e) + rows * h * (d + e)), 2.0 * rows * h * keys_per_row * (d + h + e)))
        else:
            d = m["state"] if i % 3 == 1 else m["dim"]
            channels = h * e + 2 * d * (m["groups"] if i % 3 == 1 else m["kv_heads"])
            state = h * d * e * 8.0 * (rows if decode else 1)
            n = channels + h * e + h * (1 if i % 3 == 1 else 2)
            gemm("", n, w, n)
            work["b200.short_conv"].append((rows * channels * 4.0 + (rows * (m["conv"] - 1) * channels * 8.0 if decode else 0.0), 0.0))
            inputs = rows * (channels * 2.0 + h * 4)
            if i % 3 == 1:
                if not decode:
                    work["b200.state_space_gates"].append((rows * h * 12.0, 0.0))
                work["b200.state_space_step" if decode else "b200.recurrence_chunked"].append((state + inputs + io, rows * h * 4.0 * d * e))
                work["b200.gated_parts_rms"].append((3 * io, 0.0))
            else:
                work["b200.delta_step" if decode else "b200.delta_chunked"].append((state + inputs + (2 if decode else 1) * io, rows * h * 6.0 * d * e))
                if not decode:
                    work["b200.gated_parts_rms"].append((3 * io, 0.0))
        gemm(".o", w, h * e, w)
        gemm(".up", ff, w, ff)
        gemm(".down", w, ff, w)
        work["b200.residual_add"] += [(rows * w * (2 + 8 + 2.0), 0.0)] * 2
    work["b200.scaled_embedding"].append((rows * w * (2 + 4 + 2.0), 0.0))
    work["b200.layer_norm_rows"].append((logit_rows * w * 6.0, 0.0))
    gemm(".lm_head", s["vocab"], w, 2 * s["vocab"], t=logit_rows)
    return work


def llama_work(s: dict, rows: int, keys_per_row: float, cached_rows: float) -> dict[str, list[tuple[float, float]]]:
    w, ff, d = s["width"], s["ff"], s["width"] // s["heads"]
    kv = s["kv_heads"] * d
    work: dict[str, list[tuple[float, float]]] = defaultdict(list)

    def gemm(key, n, k, n_out):
        work[key].append((n * k + 8.0 * n + 2.0 * rows * (k + n_out), 2.0 * rows * n * k))

    for _ in range(s["layers"]):
        gemm("b200.qkv_rope_append", w + 2 * kv, w, w + 2 * kv)
        work["b200.paged_attention_decode_batch.persistent_shared"].append(
            (2.0 * (cached_rows * 2 * kv + 2 * rows * w), 4.0 * rows * w * keys_per_row))
        gemm("b200.qgemv.int8.residual", w, w, 2 * w)
        gemm("b200.qgemv.int8.swiglu", 2 * ff, w, ff)
        gemm("b200.qgemv.int8.residual", w, ff, 2 * w)
        work["b200.rms_norm_quantize"] += [(rows * w * 4.0, 0.0)] * 2
    work["b200.rms_norm_quantize"].append((rows * w * 4.0, 0.0))
    gemm("b200.qgemv.int8", s["vocab"], w, s["vocab"])
    return work


def against_roofline(times: dict[str, tuple[int, float]], work: dict, hbm_gbs: float, tflops: float) -> list[dict]:
    out = []
    for key, (n, us) in sorted(times.items(), key=lambda kv: -kv[1][1]):
        ideal = sum(max(b / hbm_gbs / 1e3, f / tflops / 1e6) for b, f in work.get(key, []))
        memory = sum(b / hbm_gbs / 1e3 for b, _ in work.get(key, []))
        out.append({"kernel": key.replace("b200.", ""), "launches": n, "us": round(us / n, 2), "us_per_step": round(us, 1),
                    "bound": "hbm" if memory >= ideal * 0.999 else "tensor", "frac_of_roofline": round(ideal / us, 3) if ideal else None})
    return out


RAGGED = ("gutorax", "topunex", "rekodra", "zimorax")


def ragged_kernels(family: str, rt, plan, s: dict, rows: int, logit_rows: int, keys: float, cached: float, span: int, decode: bool, hbm: float,
                   tf: float) -> list[dict]:
    import torch
    times = kind_times(plan)
    if family == "gutorax":
        return against_roofline(times, gutorax_work(s, rows, logit_rows, keys, cached, decode), hbm, tf)
    if family == "zimorax":
        return against_roofline(times, zimorax_work(s, rows, logit_rows, keys, cached, decode), hbm, tf)
    if family == "rekodra":
        cu = rt._engine.scratch("route_cu", 0).view(torch.int32)[: s["experts"] * 7 // 8 + 1]
        return against_roofline(times, rekodra_work(s, rows, logit_rows, span, decode, int((cu.diff() > 0).sum()), int(cu[-1])), hbm, tf)
    cu = rt._engine.scratch("route_cu", 0).view(torch.int32)[: s["experts"] + 1]      # what the timed products ran on
    return against_roofline(times, topunex_work(s, rows, logit_rows, keys, cached, decode, int((cu.diff() > 0).sum())), hbm, tf)


def run(size: str, batch: int, ctx: int, prompt: int, steps: int, peaks: dict, families: tuple[str, ...] = ("gutorax",)) -> dict:
    import torch

    s = SIZES[size]
    hbm, tf = peaks["hbm_gbs"], peaks["bf16_tflops"]
    line: dict = {"size": size, **s, "batch": batch, "ctx": ctx, "prompt": prompt}
    for family in families + ("llama-shaped int8",):
        rt = build(family, s, batch=batch, positions=max(ctx, prompt) + 8 * steps + 64)
        sessions = fill(rt, batch, ctx)
        first = [(7919 * i + 1) % s["vocab"] for i in range(batch)]
        torch.cuda.synchronize()
        rt.decode_greedy_batch(sessions, first, 3)
        start, stop = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        start.record()
        rt.decode_greedy_batch(sessions, first, steps)
        stop.record()
        torch.cuda.synchronize()
        ms = start.elapsed_time(stop) / steps
        seen = ctx + steps // 2
        plan = rt._engine.plans[("decode", batch)]
        if family in RAGGED:
            keys = min(seen, s["window"])
            decode_kernels = ragged_kernels(family, rt, plan, s, batch, batch, keys, batch * keys, seen, True, hbm, tf)
        else:
            decode_kernels = against_roofline(kind_times(plan), llama_work(s, batch, seen, batch * seen), hbm, tf)
        for x in sessions:
            x.kv_cache.clear()
        session = rt.fork()
        ids = [int(t) for t in torch.randint(0, s["vocab"], (prompt,))]

        def prefill():
            session.kv_cache.clear()
            if family in RAGGED:
                session.run_step_batch([session], [ids])
            else:
                session.run([ids], mode="prefill")
        prefill_ms = timed(prefill, 5)
        if family in RAGGED:
            plan = rt._engine.portion_plan(prompt, 1, 1)
            avg = sum(min(i + 1, s["window"]) for i in range(prompt)) / prompt
            prefill_kernels = ragged_kernels(family, rt, plan, s, prompt, 1, avg, prompt, prompt, False, hbm, tf)
        else:      # the last pass of the prompt: 64 rows that attend to all of it
            plan = rt._engine.prefill_plan(64, 1)
            prefill_kernels = against_roofline(kind_times(plan), llama_work(s, 64, prompt, prompt), hbm, tf)
        rt.check_device_status()
        line[family] = {"decode_ms_per_step": round(ms, 3), "decode_tokens_per_s": round(batch / ms * 1e3, 1),
                        "prefill_ms": round(prefill_ms, 3), "prefill_tokens_per_s": round(prompt / prefill_ms * 1e3, 1),
                        "decode_kernels": decode_kernels, "prefill_kernels": prefill_kernels}
        del rt, sessions, session, plan
        torch.cuda.empty_cache()
    return line
