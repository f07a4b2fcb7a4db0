"""The Zimorax family: configuration and decode graph.

A pre-norm decoder (layer norms without bias, a scale per column on each sublayer's output) whose mixers are sliding-window
attention with talking heads (YaRN positions, normalised values, one added to the softmax denominator), a Mamba-2 state space, or
a gated delta rule, the latter two behind short convolutions; its feed-forward is a squared ReLU with biases. A range of layers
may run several times in a row, each pass with a cache and state of its own; right before a pass the residual stream becomes a
product of itself and the embedding output, plus a vector of the pass. Everything a model may choose comes from its config.json;
the graph names weights by their tensor names.
"""
from __future__ import annotations

import math
from dataclasses import dataclass, field
from typing import Any

from .artifact import CompileArtifact, Graph, Node, WeightSpec
from .gutorax import PAGE_SIZE, positive_int as _positive
from .topunex import UNBOUNDED

ARCHITECTURE = "Zimorax"


@dataclass(frozen=True)
class YarnScaling:
    """Frequencies that turn rarely within the original length are divided by factor, those that turn often are kept."""

    factor: float
    original: float
    fast: float
    slow: float


@dataclass(frozen=True)
class TalkingMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int
    rot_dims: int
    rot_base: float
    rot_scaling: YarnScaling | None


@dataclass(frozen=True)
class StateSpaceMixer:
    heads: int
    vdim: int
    state: int
    groups: int
    norm_groups: int
    taps: int

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def channels(self) -> int:
        """Columns that pass the convolution: x, B and C."""
        return self.inner + 2 * self.groups * self.state


@dataclass(frozen=True)
class DeltaMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int

    @property
    def channels(self) -> int:
        """Columns that pass the convolutions: q, k and v."""
        return 2 * self.kv_heads * self.dim + self.heads * self.vdim


@dataclass(frozen=True)
class LayerConfig:
    mixer: TalkingMixer | StateSpaceMixer | DeltaMixer
    ff: int | None           # feed-forward width, None: no feed-forward


@dataclass(frozen=True)
class LayerRun:
    """One run of layer `layer`; `begins`: the pass of the loop that begins right before it."""

    layer: int
    begins: int | None


def _divides(n: int, heads: int, where: str, what: str) -> int:
    if heads % n:
        raise ValueError(f"{where}: {heads} heads do not share {n} {what} evenly")
    return n


def _mixer(kind: str, m: dict[str, Any], index: int) -> TalkingMixer | StateSpaceMixer | DeltaMixer:
    where = f"layer {index} mixer"

    def size(name: str) -> int:
        return _positive(m[name], f"{where} {name}")
    if kind == "mamba2":
        heads = size("heads")
        mixer = StateSpaceMixer(heads, size("vdim"), size("state"), _divides(size("groups"), heads, where, "groups"), size("norm_groups"), size("conv"))
        if mixer.inner % mixer.norm_groups:
            raise ValueError(f"{where}: {mixer.inner} columns do not form {mixer.norm_groups} equal norm groups")
        return mixer
    if kind == "delta":
        heads = size("heads")
        return DeltaMixer(heads, _divides(size("kv_heads"), heads, where, "key/value heads"), size("dim"), size("vdim"), size("conv"))
    if kind == "attention":
        heads, rot, mask = size("heads"), m.get("rot") or {}, m.get("mask") or {}
        scaling = rot.get("scaling")
        mixer = TalkingMixer(
            heads=heads, kv_heads=_divides(size("kv_heads"), heads, where, "key/value heads"), dim=size("dim"), vdim=size("vdim"),
            scale=float(m["scale"]), window=_positive(mask["size"], f"{where} mask.size") if "size" in mask else UNBOUNDED,
            rot_dims=int(rot.get("dims", 0)), rot_base=float(rot.get("base", 1.0)),
            rot_scaling=None if not scaling else YarnScaling(*(float(scaling[k]) for k in ("factor", "original", "fast", "slow"))))
        if not 0 <= mixer.rot_dims <= mixer.dim or mixer.rot_dims % 2:
            raise ValueError(f"{where}: rot.dims must be even and at most dim")
        s = mixer.rot_scaling
        if s is not None and (min(s.factor, s.original, s.fast, s.slow) <= 0 or mixer.rot_base <= 0 or math.log(mixer.rot_base) == 0):
            raise ValueError(f"{where}: rot.scaling needs positive numbers and a base other than 1")
        return mixer
    raise ValueError(f"layer {index}: unknown mixer type {kind!r}")


def _feed_forward(m: dict[str, Any] | None, index: int) -> int | None:
    if m is None:
        return None
    if m.get("kind", "dense") != "dense":
        raise ValueError(f"layer {index}: unknown feed-forward kind {m['kind']!r}")
    return _positive(m["ff"], f"layer {index} mlp.ff")


def state_floats(mixer: StateSpaceMixer | DeltaMixer) -> tuple[int, int]:
    """(offset of the convolution's inputs, size) of a state slot in float32 entries: matrices first; whole 16-byte pieces."""
    matrices = mixer.heads * mixer.vdim * (mixer.state if isinstance(mixer, StateSpaceMixer) else mixer.dim)
    offset = (matrices + 3) // 4 * 4
    return offset, (offset + (mixer.taps - 1) * mixer.channels + 3) // 4 * 4


@dataclass
class ZimoraxConfig:
    """The parsed config.json, with the attributes every runtime configuration has (`hidden_size`, `vocab_size`, ...)."""

    raw: dict[str, Any]
    architecture: str = ARCHITECTURE
    hidden_size: int = 0
    vocab_size: int = 0
    norm_eps: float = 1e-6
    passes: int = 0               # of the loop; 0: there is none
    layers: list[LayerConfig] = field(default_factory=list)
    runs: list[LayerRun] = field(default_factory=list)
    max_position_embeddings: int = 8192
    dtype: str = "bfloat16"
    ragged = True                 # steps carry portions of any length (see ragged.RaggedPlan)

    @classmethod
    def from_dict(cls, data: dict[str, Any]) -> "ZimoraxConfig":
        layers = [LayerConfig(_mixer(entry["type"], entry["mixer"], i), _feed_forward(entry.get("mlp"), i)) for i, entry in enumerate(data["layers"])]
        loop = data.get("loop")
        start, stop, times = (0, 0, 0) if loop is None else (int(loop["start"]), int(loop["stop"]), _positive(loop["times"], "loop.times"))
        if loop is not None and not 0 <= start < stop <= len(layers):
            raise ValueError(f"loop: layers {start} .. {stop} are not a range of the {len(layers)} layers")
        runs = [LayerRun(i, None) for i in range(start)]
        for turn in range(times):
            runs += [LayerRun(i, turn if i == start else None) for i in range(start, stop)]
        runs += [LayerRun(i, None) for i in range(stop, len(layers))]
        return cls(raw=dict(data), hidden_size=_positive(data["width"], "width"), vocab_size=_positive(data["vocab"], "vocab"),
                   norm_eps=float(data["norm"]["eps"]), passes=times, layers=layers, runs=runs,
                   max_position_embeddings=int(data.get("max_position_embeddings", 8192)))

    def to_dict(self) -> dict[str, Any]:
        return dict(self.raw, architecture=self.architecture, max_position_embeddings=self.max_position_embeddings)

    @property
    def num_layers(self) -> int:
        """Layer runs: each has a cache or state of its own."""
        return len(self.runs)

    def cache_layout(self, page_size: int, dtype: Any) -> tuple[dict[int, dict[str, tuple[tuple[int, ...], Any]]], dict[int, tuple[int, ...]]]:
        """(pool tensors, state shapes) per layer run for `B200KVPageAllocator.configure_layout`: a row of keys and one of values
        per token, all key/value heads side by side; a recurrence's matrices and its convolutions' last inputs."""
        pools, states = {}, {}
        for run, at in enumerate(self.runs):
            m = self.layers[at.layer].mixer
            if isinstance(m, TalkingMixer):
                pools[run] = {"key_rows": ((page_size, m.kv_heads * m.dim), dtype), "value_rows": ((page_size, m.kv_heads * m.vdim), dtype)}
            else:
                states[run] = (state_floats(m)[1],)
        return pools, states


def build_zimorax_graph(config: ZimoraxConfig, *, mode: str = "decode", target: str = "cuda") -> Graph:
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

    def attention(h: str, w: str, r: str, run: int, m: TalkingMixer) -> tuple[str, int]:
        sizes = {"q": m.heads * m.dim, "k": m.kv_heads * m.dim, "v": m.kv_heads * m.vdim}
        node("concat_matmul", [h] + [weight(f"{w}.{n}", size, width) for n, size in sizes.items()], [f"{r}_{n}" for n in sizes], f"{r}.in_proj",
             bias=[weight(f"{w}.{n}.b", size) for n, size in sizes.items()])
        s = m.rot_scaling
        y = node("talking_attention", [f"{r}_q", f"{r}_k", f"{r}_v", weight(f"{w}.talk", m.heads, m.heads)], [f"{r}_attn"], f"{r}.attention", layer=run,
                 heads=m.heads, kv_heads=m.kv_heads, dim=m.dim, vdim=m.vdim, scale=m.scale, window=m.window, rot_dims=m.rot_dims, rot_base=m.rot_base,
                 yarn=None if s is None else [s.factor, s.original, s.fast, s.slow], eps=eps)
        return y, m.heads * m.vdim

    def state_space(h: str, w: str, r: str, run: int, m: StateSpaceMixer) -> tuple[str, int]:
        offset, _ = state_floats(m)
        node("concat_matmul", [h, weight(f"{w}.in", m.inner + m.channels + m.heads, width)], [f"{r}_z", f"{r}_xbc", f"{r}_dt"], f"{r}.in_proj",
             sizes=[m.inner, m.channels, m.heads], float_tail=1)
        node("short_conv", [f"{r}_xbc", weight(f"{w}.conv.b", m.channels), weight(f"{w}.conv", m.channels, m.taps)],
             [f"{r}_x", f"{r}_B", f"{r}_C"], f"{r}.conv", layer=run, offset=offset, sizes=[m.inner] + [m.groups * m.state] * 2)
        y = node("state_space", [f"{r}_C", f"{r}_B", f"{r}_x", f"{r}_dt", weight(f"{w}.dt_bias", m.heads), weight(f"{w}.A_log", m.heads),
                                 weight(f"{w}.D", m.heads)], [f"{r}_y"], f"{r}.state_space", layer=run, heads=m.heads, key_heads=m.groups, dim=m.state, vdim=m.vdim)
        y = node("gated_parts_rms", [y, f"{r}_z", weight(f"{w}.norm", m.inner)], [f"{r}_y_norm"], f"{r}.out_norm", parts=m.norm_groups, gate_first=True,
                 eps=eps)
        return y, m.inner

    def delta(h: str, w: str, r: str, run: int, m: DeltaMixer) -> tuple[str, int]:
        sizes = {"q": m.kv_heads * m.dim, "k": m.kv_heads * m.dim, "v": m.heads * m.vdim, "g": m.heads * m.vdim}
        names = [weight(f"{w}.{n}", size, width) for n, size in sizes.items()]
        node("concat_matmul", [h] + names + [weight(f"{w}.b", m.heads, width), weight(f"{w}.a", m.heads, width)], [f"{r}_qkv", f"{r}_g", f"{r}_gates"],
             f"{r}.in_proj", sizes=[m.channels, sizes["g"], m.heads, m.heads], float_tail=2)
        node("short_conv", [f"{r}_qkv", ""] + [weight(f"{w}.{n}.conv", sizes[n], m.taps) for n in "qkv"], [f"{r}_{n}" for n in "qkv"], f"{r}.conv", layer=run,
             offset=state_floats(m)[0], sizes=[sizes[n] for n in "qkv"])
        y = node("delta_rule", [f"{r}_q", f"{r}_k", f"{r}_v", f"{r}_gates", f"{r}_g", weight(f"{w}.dt_bias", m.heads), weight(f"{w}.A_log", m.heads),
                                weight(f"{w}.norm", m.vdim)],
                 [f"{r}_o"], f"{r}.delta", layer=run, heads=m.heads, key_heads=m.kv_heads, dim=m.dim, vdim=m.vdim, eps=eps)
        return y, m.heads * m.vdim

    embed = weight("embed", vocab, width)
    x = node("scaled_token_embedding", ["input_ids", embed], ["hidden"], "embed", scale=1.0)
    for run, at in enumerate(config.runs):
        w, r, layer = f"l{at.layer}", f"r{run}", config.layers[at.layer]
        if at.begins is not None:
            x = node("join_embedding", [x, "input_ids", embed, weight("loop.in", width, 2 * width), weight("loop.step", config.passes, width)],
                     [f"{r}_joined"], f"{r}.join", step=at.begins)
        h = node("layer_norm", [x, weight(f"{w}.norm1", width)], [f"{r}_n1"], f"{r}.norm1", eps=eps)
        mix = {TalkingMixer: attention, StateSpaceMixer: state_space, DeltaMixer: delta}[type(layer.mixer)]
        y, mixed = mix(h, f"{w}.mix", r, run, layer.mixer)
        y = node("matmul", [y, weight(f"{w}.mix.o", width, mixed)], [f"{r}_mixed"], f"{r}.o_proj", layer=run, projection="o")
        x = node("residual_add", [x, y, weight(f"{w}.ls1", width)], [f"{r}_post_mix"], f"{r}.mix_residual")
        if layer.ff is not None:
            h = node("layer_norm", [x, weight(f"{w}.norm2", width)], [f"{r}_n2"], f"{r}.norm2", eps=eps)
            h = node("matmul", [h, weight(f"{w}.mlp.up", layer.ff, width)], [f"{r}_up"], f"{r}.up", layer=run, projection="up", activation="relu2",
                     role="gated", bias=weight(f"{w}.mlp.up.b", layer.ff))
            y = node("matmul", [h, weight(f"{w}.mlp.down", width, layer.ff)], [f"{r}_down"], f"{r}.down", layer=run, projection="down",
                     bias=weight(f"{w}.mlp.down.b", width))
            x = node("residual_add", [x, y, weight(f"{w}.ls2", width)], [f"{r}_post_mlp"], f"{r}.mlp_residual")
    h = node("layer_norm", [x, weight("final.norm", width)], ["final_hidden"], "final_norm", rows="logits", eps=eps)
    node("matmul", [h, weight("head", vocab, width)], ["logits"], "head", projection="lm_head")
    graph.outputs = ["logits"]
    return graph


def build_zimorax_artifact(config: ZimoraxConfig, *, model_path: str = "", target: str = "cuda", quant: str | None = None,
                           modes: tuple[str, ...] = ("decode",)) -> CompileArtifact:
    if quant:
        raise ValueError(f"{ARCHITECTURE} runs unquantised weights only (got quant={quant!r})")
    return CompileArtifact(target=target, quant=None, model_path=str(model_path), config=config,
                           graphs={mode: build_zimorax_graph(config, mode=mode, target=target) for mode in modes})
