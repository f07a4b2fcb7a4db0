"""The Topunex family: configuration and decode graph.

A decoder whose attention uses its projected keys as values (sliding window with kept first tokens, capped scores, a sink,
an output gate, queries and keys normalised after rotation), with biased SwiGLU or a mixture of clamped experts behind it,
and an RMS norm on each sublayer's output only. Everything a model may choose comes from its config.json; the graph names
weights by their tensor names.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any

from .artifact import CompileArtifact, Graph, Node, WeightSpec
from .gutorax import PAGE_SIZE, positive_int as _positive

ARCHITECTURE = "Topunex"
UNBOUNDED = 1 << 30       # a window no sequence outgrows


@dataclass(frozen=True)
class RotaryScaling:
    """Stretching of long wavelengths: kept below original/high, divided by factor above original/low, blended between."""

    factor: float
    low: float
    high: float
    original: float


@dataclass(frozen=True)
class TiedMixer:
    heads: int
    kv_heads: int
    dim: int
    scale: float
    softcap: float | None
    window: int
    keep_first: int
    rot_dims: int
    rot_base: float
    rot_scaling: RotaryScaling | None


@dataclass(frozen=True)
class ClampedExpert:
    ff: int
    limit: float


@dataclass(frozen=True)
class DenseMlp:
    ff: int


@dataclass(frozen=True)
class MoeMlp:
    experts: int
    top: int
    scale: float
    expert: ClampedExpert
    shared: ClampedExpert | None


@dataclass(frozen=True)
class LayerConfig:
    mixer: TiedMixer
    mlp: DenseMlp | MoeMlp | None


def _mixer(kind: str, m: dict[str, Any], index: int) -> TiedMixer:
    where = f"layer {index} mixer"
    if kind != "attention":
        raise ValueError(f"layer {index}: unknown mixer type {kind!r}")
    rot, mask = m.get("rot") or {}, m.get("mask") or {}
    scaling = rot.get("scaling")
    dim = _positive(m["dim"], f"{where} dim")
    mixer = TiedMixer(
        heads=_positive(m["heads"], f"{where} heads"), kv_heads=_positive(m["kv_heads"], f"{where} kv_heads"), dim=dim,
        scale=float(m["scale"]), softcap=None if m.get("softcap") is None else float(m["softcap"]),
        window=UNBOUNDED if mask.get("size") is None else _positive(mask["size"], f"{where} mask.size"),
        keep_first=int(mask.get("keep_first") or 0), rot_dims=int(rot.get("dims", 0)), rot_base=float(rot.get("base", 1.0)),
        rot_scaling=None if scaling is None else RotaryScaling(*(float(scaling[k]) for k in ("factor", "low", "high", "original"))))
    if mixer.heads % mixer.kv_heads:
        raise ValueError(f"{where}: {mixer.heads} heads do not share {mixer.kv_heads} key/value heads evenly")
    if int(m.get("vdim", dim)) != dim:
        raise ValueError(f"{where}: values are the keys, so vdim must equal dim")
    if not 0 <= mixer.rot_dims <= dim or mixer.rot_dims % 2:
        raise ValueError(f"{where}: rot.dims must be even and at most dim")
    if mixer.softcap is not None and mixer.softcap <= 0:
        raise ValueError(f"{where}: softcap must be positive")
    if mixer.keep_first < 0:
        raise ValueError(f"{where}: mask.keep_first must not be negative")
    return mixer


def _expert(m: dict[str, Any], where: str) -> ClampedExpert:
    return ClampedExpert(_positive(m["ff"], f"{where}.ff"), float(m["limit"]))


def _mlp(m: dict[str, Any] | None, index: int) -> DenseMlp | MoeMlp | None:
    where = f"layer {index} mlp"
    if m is None:
        return None
    if m["kind"] == "dense":
        return DenseMlp(_positive(m["ff"], f"{where}.ff"))
    if m["kind"] != "moe":
        raise ValueError(f"layer {index}: unknown feed-forward kind {m['kind']!r}")
    router = m["router"]
    mlp = MoeMlp(_positive(router["experts"], f"{where}.router.experts"), _positive(router["top"], f"{where}.router.top"),
                 float(router.get("scale", 1.0)), _expert(m["expert"], f"{where}.expert"),
                 None if m.get("shared") is None else _expert(m["shared"], f"{where}.shared"))
    if mlp.top > mlp.experts:
        raise ValueError(f"{where}: {mlp.top} of {mlp.experts} experts cannot be chosen")
    return mlp


@dataclass
class TopunexConfig:
    """The parsed config.json, with the attributes every runtime configuration has (`hidden_size`, `vocab_size`, ...)."""

    raw: dict[str, Any]
    architecture: str = ARCHITECTURE
    hidden_size: int = 0
    vocab_size: int = 0
    norm_eps: float = 1e-6
    layers: list[LayerConfig] = field(default_factory=list)
    max_position_embeddings: int = 8192
    dtype: str = "bfloat16"
    ragged = True                 # steps carry portions of any length (see ragged.RaggedPlan)

    @classmethod
    def from_dict(cls, data: dict[str, Any]) -> "TopunexConfig":
        layers = [LayerConfig(_mixer(entry["type"], entry["mixer"], i), _mlp(entry.get("mlp"), i)) for i, entry in enumerate(data["layers"])]
        return cls(raw=dict(data), hidden_size=_positive(data["width"], "width"), vocab_size=_positive(data["vocab"], "vocab"),
                   norm_eps=float(data["norm"]["eps"]), layers=layers, max_position_embeddings=int(data.get("max_position_embeddings", 8192)))

    def to_dict(self) -> dict[str, Any]:
        return dict(self.raw, architecture=self.architecture, max_position_embeddings=self.max_position_embeddings)

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    def cache_layout(self, page_size: int, dtype: Any) -> tuple[dict[int, dict[str, tuple[tuple[int, ...], Any]]], dict[int, tuple[int, ...]]]:
        """(pool tensors per layer, no states) for `B200KVPageAllocator.configure_layout`: a row per token and key/value
        head holds the key as projected and its rotated entries, and beside it one over its root mean square."""
        import torch
        pools = {}
        for i, layer in enumerate(self.layers):
            m = layer.mixer
            pools[i] = {"rows": ((m.kv_heads, page_size, m.dim + m.rot_dims), dtype), "inv_rms": ((m.kv_heads, page_size), torch.float32)}
        return pools, {}


def build_topunex_graph(config: TopunexConfig, *, mode: str = "decode", target: str = "cuda") -> Graph:
    graph = Graph(name=config.architecture, mode=mode, target=target)
    graph.attrs = {"model_config": config.to_dict(), "execution_mode": mode,
                   "kv_cache": {"policy": "paged"}, "execution_hints": {"target": target, "mode": mode, "page_size": PAGE_SIZE}}
    width, vocab, eps = config.hidden_size, config.vocab_size, config.norm_eps

    def weight(name: str, *shape: int) -> str:
        graph.weights[name] = WeightSpec(key=name, shape=tuple(shape), dtype=config.dtype, file="model.safetensors")
        return name

    def node(op: str, inputs: list[str], outputs: list[str], name: str, **attrs: Any) -> str:
        graph.nodes.append(Node(op=op, inputs=inputs, outputs=outputs, attrs=attrs, name=name))
        return outputs[0]

    def clamped(x: str, p: str, e: ClampedExpert, out: str) -> str:
        return node("fused_glu", [x, weight(f"{p}.gate", e.ff, width), weight(f"{p}.up", e.ff, width)], [out], p, activation="clamped", limit=e.limit)

    x = node("scaled_token_embedding", ["input_ids", weight("embed", vocab, width)], ["hidden"], "embed", scale=1.0)
    for i, layer in enumerate(config.layers):
        p, m = f"l{i}", layer.mixer
        hd, gd = m.heads * m.dim, m.kv_heads * m.dim
        names = [weight(f"{p}.mix.q", hd, width), weight(f"{p}.mix.k", gd, width), weight(f"{p}.mix.g", hd, width)]
        node("concat_matmul", [x] + names, [f"{p}_q", f"{p}_k", f"{p}_g"], f"{p}.in_proj",
             bias=[weight(f"{p}.mix.q.b", hd), weight(f"{p}.mix.k.b", gd), None])
        s = m.rot_scaling
        y = node("tied_attention", [f"{p}_q", f"{p}_k", f"{p}_g", weight(f"{p}.mix.sink", m.heads)], [f"{p}_attn"], f"{p}.attention",
                 layer=i, heads=m.heads, kv_heads=m.kv_heads, dim=m.dim, scale=m.scale, softcap=m.softcap, window=m.window,
                 keep_first=m.keep_first, rot_dims=m.rot_dims, rot_base=m.rot_base, eps=eps,
                 rot_scaling=None if s is None else [s.factor, s.low, s.high, s.original])
        y = node("matmul", [y, weight(f"{p}.mix.o", width, hd)], [f"{p}_mixed"], f"{p}.o_proj", layer=i, projection="o",
                 bias=weight(f"{p}.mix.o.b", width))
        x = node("residual_rms_norm", [x, y, weight(f"{p}.norm1", width)], [f"{p}_post_mix"], f"{p}.mix_residual", eps=eps)
        f = f"{p}.mlp"
        if isinstance(layer.mlp, DenseMlp):
            ff = layer.mlp.ff
            h = node("fused_glu", [x, weight(f"{f}.gate", ff, width), weight(f"{f}.up", ff, width)], [f"{p}_gated"], f"{p}.swiglu", layer=i,
                     activation="silu", bias=[weight(f"{f}.gate.b", ff), weight(f"{f}.up.b", ff)])
            y = node("matmul", [h, weight(f"{f}.down", width, ff)], [f"{p}_down"], f"{p}.down_proj", layer=i, projection="down",
                     bias=weight(f"{f}.down.b", width))
            x = node("residual_rms_norm", [x, y, weight(f"{p}.norm2", width)], [f"{p}_post_mlp"], f"{p}.mlp_residual", eps=eps)
        elif isinstance(layer.mlp, MoeMlp):
            c = layer.mlp
            node("expert_router", [x, weight(f"{f}.router", c.experts, width)], [f"{p}_routing"], f"{p}.router", layer=i, top=c.top, scale=c.scale)
            shared = []
            if c.shared is not None:
                h = clamped(x, f"{f}.shared", c.shared, f"{p}_shared_gated")
                shared = [node("matmul", [h, weight(f"{f}.shared.down", width, c.shared.ff)], [f"{p}_shared"], f"{p}.shared_down", layer=i,
                               projection="down")]
            each = range(c.experts)
            y = node("expert_mixture", [x, f"{p}_routing"] + [weight(f"{f}.e{e}.gate", c.expert.ff, width) for e in each]
                     + [weight(f"{f}.e{e}.up", c.expert.ff, width) for e in each] + [weight(f"{f}.e{e}.down", width, c.expert.ff) for e in each],
                     [f"{p}_experts"], f"{p}.experts", layer=i, experts=c.experts, activation="clamped", limit=c.expert.limit)
            x = node("combine_residual_rms_norm", [x, y, f"{p}_routing", weight(f"{p}.norm2", width)] + shared, [f"{p}_post_mlp"],
                     f"{p}.mlp_residual", eps=eps)
    h = node("rms_norm", [x, weight("final.norm", width)], ["final_hidden"], "final_norm", rows="logits", eps=eps)
    node("matmul", [h, weight("head", vocab, width)], ["logits"], "head", projection="lm_head")
    graph.outputs = ["logits"]
    return graph


def build_topunex_artifact(config: TopunexConfig, *, model_path: str = "", target: str = "cuda", quant: str | None = None,
                           modes: tuple[str, ...] = ("decode",)) -> CompileArtifact:
    if quant:
        raise ValueError(f"{ARCHITECTURE} runs unquantised weights only (got quant={quant!r})")
    return CompileArtifact(target=target, quant=None, model_path=str(model_path), config=config,
                           graphs={mode: build_topunex_graph(config, mode=mode, target=target) for mode in modes})
