"""The Rekodra family: configuration and decode graph.

A pre-norm decoder whose mixers are attention over projected keys that are also the values (queries and keys normalised over
the whole projection, rotated, with a sink), or sliding-window attention beside a matrix memory (their normalised outputs
averaged); its feed-forward is a mixture of experts with grouped choices, experts that return their input, and a gated shared
expert. A range of layers may run several times in a row, each pass with a cache and state of its own and the embedding output
joining before it. Everything a model may choose comes from its config.json; the graph names weights by their tensor names.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any

from .artifact import CompileArtifact, Graph, Node, WeightSpec
from .gutorax import PAGE_SIZE, positive_int as _positive
from .topunex import UNBOUNDED

ARCHITECTURE = "Rekodra"


@dataclass(frozen=True)
class SinkMixer:
    """Causal attention whose values are its projected keys."""

    heads: int
    kv_heads: int
    dim: int
    scale: float
    rot_dims: int
    rot_base: float


@dataclass(frozen=True)
class WindowMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int


@dataclass(frozen=True)
class MemoryMixer:
    heads: int
    dim: int
    vdim: int
    gate_cap: float


@dataclass(frozen=True)
class ParallelMixer:
    left: WindowMixer
    right: MemoryMixer


@dataclass(frozen=True)
class MoeMlp:
    experts: int
    identity: int
    top: int
    groups: int
    keep: int
    ff: int
    shared_ff: int | None


@dataclass(frozen=True)
class LayerConfig:
    mixer: SinkMixer | ParallelMixer
    mlp: MoeMlp | None


@dataclass(frozen=True)
class LayerRun:
    """One run of layer `layer`; `rejoin`: the embedding output is added right before it."""

    layer: int
    rejoin: bool


def _heads(m: dict[str, Any], where: str) -> tuple[int, int, int]:
    heads, kv_heads = _positive(m["heads"], f"{where} heads"), _positive(m["kv_heads"], f"{where} kv_heads")
    if heads % kv_heads:
        raise ValueError(f"{where}: {heads} heads do not share {kv_heads} key/value heads evenly")
    return heads, kv_heads, _positive(m["dim"], f"{where} dim")


def _mixer(kind: str, m: dict[str, Any], index: int) -> SinkMixer | ParallelMixer:
    where = f"layer {index} mixer"
    if kind == "attention":
        heads, kv_heads, dim = _heads(m, where)
        rot = m.get("rot") or {}
        mixer = SinkMixer(heads, kv_heads, dim, float(m["scale"]), int(rot.get("dims", 0)), float(rot.get("base", 1.0)))
        if int(m.get("vdim", dim)) != dim:
            raise ValueError(f"{where}: values are the keys, so vdim must equal dim")
        if not 0 <= mixer.rot_dims <= dim or mixer.rot_dims % 2:
            raise ValueError(f"{where}: rot.dims must be even and at most dim")
        return mixer
    if kind == "parallel":
        left, right = m["left"], m["right"]
        heads, kv_heads, dim = _heads(left, f"{where}.left")
        window = WindowMixer(heads, kv_heads, dim, _positive(left["vdim"], f"{where}.left vdim"), float(left["scale"]),
                             _positive(left["mask"]["size"], f"{where}.left mask.size"))
        memory = MemoryMixer(_positive(right["heads"], f"{where}.right heads"), _positive(right["dim"], f"{where}.right dim"),
                             _positive(right["vdim"], f"{where}.right vdim"), float(right["gate_cap"]))
        if memory.gate_cap <= 0:
            raise ValueError(f"{where}.right: gate_cap must be positive")
        return ParallelMixer(window, memory)
    raise ValueError(f"layer {index}: unknown mixer type {kind!r}")


def _mlp(m: dict[str, Any] | None, index: int) -> MoeMlp | None:
    where = f"layer {index} mlp"
    if m is None:
        return None
    if m["kind"] != "moe":
        raise ValueError(f"layer {index}: unknown feed-forward kind {m['kind']!r}")
    router, groups = m["router"], m["router"].get("groups") or {}
    shared = m.get("shared")
    mlp = MoeMlp(experts=_positive(router["experts"], f"{where}.router.experts"), identity=int(router.get("identity") or 0),
                 top=_positive(router["top"], f"{where}.router.top"), groups=_positive(groups.get("count", 1), f"{where}.router.groups.count"),
                 keep=_positive(groups.get("keep", groups.get("count", 1)), f"{where}.router.groups.keep"), ff=_positive(m["expert"]["ff"], f"{where}.expert.ff"),
                 shared_ff=None if shared is None else _positive(shared["ff"], f"{where}.shared.ff"))
    scored = mlp.experts + mlp.identity
    if mlp.identity < 0 or scored % mlp.groups or mlp.keep > mlp.groups:
        raise ValueError(f"{where}: {scored} router outputs do not form {mlp.groups} equal groups of which {mlp.keep} are kept")
    if mlp.top > scored // mlp.groups * mlp.keep:
        raise ValueError(f"{where}: {mlp.top} experts cannot be chosen from {mlp.keep} groups of {scored // mlp.groups}")
    return mlp


@dataclass
class RekodraConfig:
    """The parsed config.json, with the attributes every runtime configuration has (`hidden_size`, `vocab_size`, ...)."""

    raw: dict[str, Any]
    architecture: str = ARCHITECTURE
    hidden_size: int = 0
    vocab_size: int = 0
    embedding_scale: float = 1.0
    logit_scale: float = 1.0
    norm_eps: float = 1e-5
    layers: list[LayerConfig] = field(default_factory=list)
    runs: list[LayerRun] = field(default_factory=list)
    max_position_embeddings: int = 8192
    dtype: str = "bfloat16"
    ragged = True                 # steps carry portions of any length (see ragged.RaggedPlan)

    @classmethod
    def from_dict(cls, data: dict[str, Any]) -> "RekodraConfig":
        layers = [LayerConfig(_mixer(entry["type"], entry["mixer"], i), _mlp(entry.get("mlp"), i)) for i, entry in enumerate(data["layers"])]
        loop = data.get("loop")
        start, stop, times = (0, 0, 1) if loop is None else (int(loop["start"]), int(loop["stop"]), _positive(loop["times"], "loop.times"))
        if loop is not None and not 0 <= start < stop <= len(layers):
            raise ValueError(f"loop: layers {start} .. {stop} are not a range of the {len(layers)} layers")
        runs = [LayerRun(i, False) for i in range(start)]
        for turn in range(times):
            runs += [LayerRun(i, turn > 0 and i == start) for i in range(start, stop)]
        runs += [LayerRun(i, False) for i in range(stop, len(layers))]
        return cls(raw=dict(data), hidden_size=_positive(data["width"], "width"), vocab_size=_positive(data["vocab"], "vocab"),
                   embedding_scale=float((data.get("embedding") or {}).get("scale", 1.0)), logit_scale=float(data.get("logit_scale", 1.0)),
                   norm_eps=float(data["norm"]["eps"]), layers=layers, runs=runs,
                   max_position_embeddings=int(data.get("max_position_embeddings", 8192)))

    def to_dict(self) -> dict[str, Any]:
        return dict(self.raw, architecture=self.architecture, max_position_embeddings=self.max_position_embeddings)

    @property
    def num_layers(self) -> int:
        """Layer runs: each has a cache or state of its own."""
        return len(self.runs)

    def cache_layout(self, page_size: int, dtype: Any) -> tuple[dict[int, dict[str, tuple[tuple[int, ...], Any]]], dict[int, tuple[int, ...]]]:
        """(pool tensors, state shapes) per layer run for `B200KVPageAllocator.configure_layout`: a row per token and
        key/value head holds value and key, and beside it one over the key's root mean square."""
        import torch

        from .expert_ops import row_layout
        from .hybrid_ops import memory_state_size
        pools, states = {}, {}
        for run, at in enumerate(self.runs):
            m = self.layers[at.layer].mixer
            if isinstance(m, ParallelMixer):
                states[run] = (memory_state_size(m.right.heads, m.right.dim, m.right.vdim),)
                kv_heads, (width, _) = m.left.kv_heads, row_layout(m.left.vdim, 0, m.left.dim)
            else:
                kv_heads, (width, _) = m.kv_heads, row_layout(m.dim, m.rot_dims)
            pools[run] = {"rows": ((kv_heads, page_size, width), dtype), "inv_rms": ((kv_heads, page_size), torch.float32)}
        return pools, states


def build_rekodra_graph(config: RekodraConfig, *, mode: str = "decode", target: str = "cuda") -> Graph:
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

    def sink_attention(x: str, h: str, w: str, r: str, run: int, m: SinkMixer) -> str:
        hd, gd = m.heads * m.dim, m.kv_heads * m.dim
        node("concat_matmul", [h, weight(f"{w}.q", hd, width), weight(f"{w}.k", gd, width)], [f"{r}_q", f"{r}_k"], f"{r}.in_proj")
        y = node("tied_attention", [f"{r}_q", f"{r}_k", "", weight(f"{w}.sink", m.heads), "", weight(f"{w}.q.norm", hd), weight(f"{w}.k.norm", gd)],
                 [f"{r}_attn"], f"{r}.attention", layer=run, heads=m.heads, kv_heads=m.kv_heads, dim=m.dim, scale=m.scale, softcap=None,
                 window=UNBOUNDED, keep_first=0, rot_dims=m.rot_dims, rot_base=m.rot_base, eps=eps, whole_norm=True)
        y = node("matmul", [y, weight(f"{w}.o", width, hd)], [f"{r}_mixed"], f"{r}.o_proj", layer=run, projection="o")
        return node("residual_add", [x, y], [f"{r}_post_mix"], f"{r}.mix_residual")

    def parallel(x: str, h: str, w: str, r: str, run: int, mixer: ParallelMixer) -> str:
        a, m = mixer.left, mixer.right
        wl, wr, qk, vd = f"{w}.left", f"{w}.right", m.heads * m.dim, m.heads * m.vdim
        node("concat_matmul", [h, weight(f"{wr}.q", qk, width), weight(f"{wr}.k", qk, width), weight(f"{wr}.v", vd, width), weight(f"{wr}.g", vd, width),
                               weight(f"{wl}.q", a.heads * a.dim, width), weight(f"{wl}.k", a.kv_heads * a.dim, width),
                               weight(f"{wl}.v", a.kv_heads * a.vdim, width), weight(f"{wr}.i", m.heads, width), weight(f"{wr}.f", m.heads, width)],
             [f"{r}_mq", f"{r}_mk", f"{r}_mv", f"{r}_mg", f"{r}_q", f"{r}_k", f"{r}_v", f"{r}_gates"], f"{r}.in_proj", float_tail=2)
        y = node("tied_attention", [f"{r}_q", f"{r}_k", "", "", f"{r}_v", weight(f"{wl}.q.norm", a.dim), weight(f"{wl}.k.norm", a.dim)],
                 [f"{r}_attn"], f"{r}.attention", layer=run, heads=a.heads, kv_heads=a.kv_heads, dim=a.vdim, key_dim=a.dim, scale=a.scale,
                 softcap=None, window=a.window, keep_first=0, rot_dims=0, rot_base=1.0, eps=eps)
        left = node("matmul", [y, weight(f"{wl}.o", width, a.heads * a.vdim)], [f"{r}_left"], f"{r}.left_o_proj", layer=run, projection="o")
        y = node("matrix_memory", [f"{r}_mq", f"{r}_mk", f"{r}_mv", f"{r}_gates", f"{r}_mg", weight(f"{wr}.i.b", m.heads), weight(f"{wr}.f.b", m.heads),
                                   weight(f"{wr}.norm", vd)],
                 [f"{r}_memory"], f"{r}.memory", layer=run, heads=m.heads, dim=m.dim, vdim=m.vdim, gate_cap=m.gate_cap, eps=eps)
        right = node("matmul", [y, weight(f"{wr}.o", width, vd)], [f"{r}_right"], f"{r}.right_o_proj", layer=run, projection="o", role="sublayer_right")
        return node("residual_rms_pair", [x, left, weight(f"{wl}.out", width), right, weight(f"{wr}.out", width)], [f"{r}_post_mix"],
                    f"{r}.mix_residual", factor=0.5, eps=eps)

    def mixture(x: str, h: str, w: str, r: str, run: int, c: MoeMlp) -> str:
        scored = c.experts + c.identity
        gated = c.shared_ff is not None
        node("expert_router", [h, weight(f"{w}.router", scored, width), weight(f"{w}.correction", scored)]
             + ([weight(f"{w}.shared.sg", 1, width)] if gated else []), [f"{r}_routing"] + ([f"{r}_shared_gate"] if gated else []), f"{r}.router",
             layer=run, scores="softmax", top=c.top, scale=1.0, groups=c.groups, keep=c.keep, identity=c.identity)
        shared = []
        if gated:
            y = node("fused_glu", [h, weight(f"{w}.shared.gate", c.shared_ff, width), weight(f"{w}.shared.up", c.shared_ff, width)],
                     [f"{r}_shared_gated"], f"{r}.shared_swiglu", layer=run, activation="silu")
            shared = [node("matmul", [y, weight(f"{w}.shared.down", width, c.shared_ff)], [f"{r}_shared"], f"{r}.shared_down", layer=run,
                           projection="down"), f"{r}_shared_gate"]
        each = range(c.experts)
        y = node("expert_mixture", [h, f"{r}_routing"] + [weight(f"{w}.e{e}.gate", c.ff, width) for e in each]
                 + [weight(f"{w}.e{e}.up", c.ff, width) for e in each] + [weight(f"{w}.e{e}.down", width, c.ff) for e in each],
                 [f"{r}_experts"], f"{r}.experts", layer=run, experts=c.experts, activation="silu")
        return node("combine_residual", [x, y, f"{r}_routing", h] + shared, [f"{r}_post_mlp"], f"{r}.mlp_residual")

    embed = weight("embed", vocab, width)
    x = node("scaled_token_embedding", ["input_ids", embed], ["hidden"], "embed", scale=config.embedding_scale)
    for run, at in enumerate(config.runs):
        w, r, layer = f"l{at.layer}", f"r{run}", config.layers[at.layer]
        if at.rejoin:
            x = node("add_token_embedding", [x, "input_ids", embed], [f"{r}_rejoined"], f"{r}.rejoin", scale=config.embedding_scale)
        h = node("rms_norm", [x, weight(f"{w}.norm1", width)], [f"{r}_n1"], f"{r}.norm1", eps=eps)
        mix = parallel if isinstance(layer.mixer, ParallelMixer) else sink_attention
        x = mix(x, h, f"{w}.mix", r, run, layer.mixer)
        if layer.mlp is not None:
            h = node("rms_norm", [x, weight(f"{w}.norm2", width)], [f"{r}_n2"], f"{r}.norm2", eps=eps)
            x = mixture(x, h, f"{w}.mlp", r, run, layer.mlp)
    h = node("rms_norm", [x, weight("final.norm", width)], ["final_hidden"], "final_norm", rows="logits", eps=eps, scale=config.logit_scale)
    node("matmul", [h, embed], ["logits"], "head", projection="lm_head")
    graph.outputs = ["logits"]
    return graph


def build_rekodra_artifact(config: RekodraConfig, *, model_path: str = "", target: str = "cuda", quant: str | None = None,
                           modes: tuple[str, ...] = ("decode",)) -> CompileArtifact:
    if quant:
        raise ValueError(f"{ARCHITECTURE} runs unquantised weights only (got quant={quant!r})")
    return CompileArtifact(target=target, quant=None, model_path=str(model_path), config=config,
                           graphs={mode: build_rekodra_graph(config, mode=mode, target=target) for mode in modes})
