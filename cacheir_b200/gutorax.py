"""The Gutorax family: configuration and decode graph.

A decoder whose layers mix latent attention (window, sink, output gate, optionally another layer's cache) with a
decayed linear recurrence, with Dynamic Tanh before and after each sublayer and a per-layer token input behind the
feed-forward. Everything a model may choose comes from its config.json; the graph names weights by their tensor names.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any

from .artifact import CompileArtifact, Graph, Node, WeightSpec

ARCHITECTURE = "Gutorax"
PAGE_SIZE = 64          # cache rows per page: one attention tile


@dataclass(frozen=True)
class LatentMixer:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    window: int
    rot_dims: int
    rot_base: float
    kv_from: int | None = None


@dataclass(frozen=True)
class LightningMixer:
    heads: int
    dim: int
    vdim: int
    decay: tuple[float, ...]


@dataclass(frozen=True)
class LayerConfig:
    mixer: LatentMixer | LightningMixer
    ff: int | None           # dense feed-forward width, None: no feed-forward


def positive_int(value: Any, what: str) -> int:
    n = int(value)
    if n <= 0 or n != value:
        raise ValueError(f"{what} must be a positive integer, got {value!r}")
    return n


def _mixer(kind: str, m: dict[str, Any], index: int) -> LatentMixer | LightningMixer:
    where = f"layer {index} mixer"
    if kind == "lightning":
        heads = positive_int(m["heads"], f"{where} heads")
        decay = tuple(float(v) for v in m["decay"])
        if len(decay) != heads:
            raise ValueError(f"{where}: {len(decay)} decays for {heads} heads")
        return LightningMixer(heads, positive_int(m["dim"], f"{where} dim"), positive_int(m["vdim"], f"{where} vdim"), decay)
    if kind == "latent_attention":
        rot = m["rot"]
        mixer = LatentMixer(
            heads=positive_int(m["heads"], f"{where} heads"), dim=positive_int(m["dim"], f"{where} dim"),
            rot_dim=positive_int(m["rot_dim"], f"{where} rot_dim"), vdim=positive_int(m["vdim"], f"{where} vdim"),
            kv_rank=positive_int(m["kv_rank"], f"{where} kv_rank"), scale=float(m["scale"]),
            window=positive_int(m["mask"]["size"], f"{where} mask.size"), rot_dims=positive_int(rot["dims"], f"{where} rot.dims"),
            rot_base=float(rot["base"]), kv_from=None if m.get("kv_from") is None else int(m["kv_from"]))
        if mixer.rot_dims % 2 or mixer.rot_dims > mixer.rot_dim:
            raise ValueError(f"{where}: rot.dims must be even and at most rot_dim")
        return mixer
    raise ValueError(f"layer {index}: unknown mixer type {kind!r}")


@dataclass
class GutoraxConfig:
    """The parsed config.json, with the attributes every runtime configuration has (`hidden_size`, `vocab_size`, ...)."""

    raw: dict[str, Any]
    architecture: str = ARCHITECTURE
    hidden_size: int = 0
    vocab_size: int = 0
    embedding_scale: float = 1.0
    norm_eps: float = 1e-5
    side_dim: int | None = None
    layers: list[LayerConfig] = field(default_factory=list)
    max_position_embeddings: int = 8192
    dtype: str = "bfloat16"
    ragged = True                 # steps carry portions of any length (see ragged.RaggedPlan)

    @classmethod
    def from_dict(cls, data: dict[str, Any]) -> "GutoraxConfig":
        layers = []
        for i, entry in enumerate(data["layers"]):
            mixer = _mixer(entry["type"], entry["mixer"], i)
            mlp = entry.get("mlp")
            if mlp is not None and mlp.get("kind", "dense") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
            if isinstance(mixer, LatentMixer) and mixer.kv_from is not None:
                j = mixer.kv_from
                owner = layers[j].mixer if 0 <= j < i else None
                if not isinstance(owner, LatentMixer) or owner.kv_from is not None:
                    raise ValueError(f"layer {i}: kv_from {j} is not an earlier latent attention layer with its own cache")
                same = ("kv_rank", "rot_dim", "rot_dims", "rot_base")
                if any(getattr(owner, k) != getattr(mixer, k) for k in same):
                    raise ValueError(f"layer {i}: latent size and rotation differ from those of layer {j}, whose cache it reads")
            layers.append(LayerConfig(mixer, None if mlp is None else positive_int(mlp["ff"], f"layer {i} mlp.ff")))
        side = data.get("token_side")
        return cls(raw=dict(data), hidden_size=positive_int(data["width"], "width"), vocab_size=positive_int(data["vocab"], "vocab"),
                   embedding_scale=float((data.get("embedding") or {}).get("scale", 1.0)), norm_eps=float(data["norm"]["eps"]),
                   side_dim=None if side is None else positive_int(side["dim"], "token_side.dim"), layers=layers,
                   max_position_embeddings=int(data.get("max_position_embeddings", 8192)))

    def to_dict(self) -> dict[str, Any]:
        return dict(self.raw, architecture=self.architecture, max_position_embeddings=self.max_position_embeddings)

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    def cache_layout(self, page_size: int, dtype: Any) -> tuple[dict[int, dict[str, tuple[tuple[int, ...], Any]]], dict[int, tuple[int, ...]]]:
        """(pool tensors per caching layer, state shape per recurrent layer) for `B200KVPageAllocator.configure_layout`."""
        pools, states = {}, {}
        for i, layer in enumerate(self.layers):
            m = layer.mixer
            if isinstance(m, LightningMixer):
                states[i] = (m.heads, m.dim, m.vdim)
            elif m.kv_from is None:
                pools[i] = {"latent": ((page_size, m.kv_rank + m.rot_dim), dtype)}
        return pools, states


def build_gutorax_graph(config: GutoraxConfig, *, mode: str = "decode", target: str = "cuda") -> Graph:
    graph = Graph(name=config.architecture, mode=mode, target=target)
    graph.attrs = {"model_config": config.to_dict(), "execution_mode": mode,
                   "kv_cache": {"policy": "paged"}, "execution_hints": {"target": target, "mode": mode, "page_size": PAGE_SIZE}}
    width, vocab, eps = config.hidden_size, config.vocab_size, config.norm_eps

    def weight(name: str, *shape: int) -> str:
        graph.weights[name] = WeightSpec(key=name, shape=tuple(shape), dtype=config.dtype, file="model.safetensors")
        return name

    def dyt(name: str) -> list[str]:
        return [weight(name, width), weight(name + ".b", width), weight(name + ".alpha")]

    def node(op: str, inputs: list[str], outputs: list[str], name: str, **attrs: Any) -> str:
        graph.nodes.append(Node(op=op, inputs=inputs, outputs=outputs, attrs=attrs, name=name))
        return outputs[0]

    x = node("scaled_token_embedding", ["input_ids", weight("embed", vocab, width)], ["hidden"], "embed", scale=config.embedding_scale)
    if config.side_dim is not None:
        weight("side.embed", vocab, config.side_dim * config.num_layers)
    for i, layer in enumerate(config.layers):
        p, m = f"l{i}", layer.mixer
        h = node("dynamic_tanh", [x] + dyt(f"{p}.norm1"), [f"{p}_n1"], f"{p}.norm1")
        if isinstance(m, LatentMixer):
            w_q = weight(f"{p}.mix.q", m.heads * (m.dim + m.rot_dim), width)
            w_g = weight(f"{p}.mix.g", m.heads * m.vdim, width)
            own = m.kv_from is None
            down = [weight(f"{p}.mix.dkv", m.kv_rank + m.rot_dim, width)] if own else []
            node("concat_matmul", [h, w_q] + down + [w_g], [f"{p}_q"] + ([f"{p}_down"] if own else []) + [f"{p}_g"], f"{p}.in_proj")
            uk, uv = weight(f"{p}.mix.uk", m.heads * m.dim, m.kv_rank), weight(f"{p}.mix.uv", m.heads * m.vdim, m.kv_rank)
            sink = weight(f"{p}.mix.sink", m.heads)
            cached = [f"{p}_down", weight(f"{p}.mix.dkv.norm", m.kv_rank)] if own else []
            y = node("latent_attention", [f"{p}_q", f"{p}_g", uk, uv, sink] + cached, [f"{p}_attn"], f"{p}.attention",
                     layer=i, cache_layer=i if own else m.kv_from, heads=m.heads, dim=m.dim, rot_dim=m.rot_dim, vdim=m.vdim,
                     kv_rank=m.kv_rank, scale=m.scale, window=m.window, rot_dims=m.rot_dims, rot_base=m.rot_base, eps=eps)
            mixed = m.heads * m.vdim
        else:
            qk, vd = m.heads * m.dim, m.heads * m.vdim
            names = [weight(f"{p}.mix.q", qk, width), weight(f"{p}.mix.k", qk, width), weight(f"{p}.mix.v", vd, width), weight(f"{p}.mix.g", vd, width)]
            node("concat_matmul", [h] + names, [f"{p}_q", f"{p}_k", f"{p}_v", f"{p}_g"], f"{p}.in_proj", activation="silu", activated=3)
            node("linear_recurrence", [f"{p}_q", f"{p}_k", f"{p}_v"], [f"{p}_rec"], f"{p}.recurrence", layer=i, heads=m.heads,
                 dim=m.dim, vdim=m.vdim, decay=list(m.decay))
            y = node("gated_rms_norm", [f"{p}_rec", f"{p}_g", weight(f"{p}.mix.norm", vd)], [f"{p}_rec_norm"], f"{p}.out_norm", eps=eps)
            mixed = vd
        y = node("matmul", [y, weight(f"{p}.mix.o", width, mixed)], [f"{p}_mixed"], f"{p}.o_proj", layer=i, projection="o")
        x = node("residual_dynamic_tanh", [x, y] + dyt(f"{p}.norm1b"), [f"{p}_post_mix"], f"{p}.mix_residual")
        if layer.ff is not None:
            h = node("dynamic_tanh", [x] + dyt(f"{p}.norm2"), [f"{p}_n2"], f"{p}.norm2")
            h = node("fused_geglu", [h, weight(f"{p}.mlp.gate", layer.ff, width), weight(f"{p}.mlp.up", layer.ff, width)], [f"{p}_gated"],
                     f"{p}.geglu", layer=i)
            y = node("matmul", [h, weight(f"{p}.mlp.down", width, layer.ff)], [f"{p}_down_proj"], f"{p}.down_proj", layer=i, projection="down")
            x = node("residual_dynamic_tanh", [x, y] + dyt(f"{p}.norm2b"), [f"{p}_post_mlp"], f"{p}.mlp_residual")
        if config.side_dim is not None:
            d = config.side_dim
            h = node("token_side_gate", [x, weight(f"{p}.side.gate", d, width), "side.embed", "input_ids"], [f"{p}_side"], f"{p}.side_gate", column=i * d)
            y = node("matmul", [h, weight(f"{p}.side.proj", width, d)], [f"{p}_side_proj"], f"{p}.side_proj", layer=i, projection="side")
            x = node("residual_rms_norm", [x, y, weight(f"{p}.side.norm", width)], [f"{p}_post_side"], f"{p}.side_residual", eps=eps)
    h = node("dynamic_tanh", [x] + dyt("final.norm"), ["final_hidden"], "final_norm", rows="logits")
    node("matmul", [h, weight("head", vocab, width)], ["logits"], "head", projection="lm_head")
    graph.outputs = ["logits"]
    return graph


def build_gutorax_artifact(config: GutoraxConfig, *, model_path: str = "", target: str = "cuda", quant: str | None = None,
                           modes: tuple[str, ...] = ("decode",)) -> CompileArtifact:
    if quant:
        raise ValueError(f"{ARCHITECTURE} runs unquantised weights only (got quant={quant!r})")
    return CompileArtifact(target=target, quant=None, model_path=str(model_path), config=config,
                           graphs={mode: build_gutorax_graph(config, mode=mode, target=target) for mode in modes})
