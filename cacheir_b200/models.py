"""Model registry: which configuration class and graph builder serve a config.json, by its architecture."""
from __future__ import annotations

import json
from dataclasses import dataclass
from pathlib import Path
from typing import Any, Callable

from . import gutorax, rekodra, topunex, zimorax
from .artifact import CompileArtifact, ModelConfig, build_decoder_artifact


@dataclass(frozen=True)
class ModelFamily:
    name: str
    config_from_dict: Callable[[dict[str, Any]], Any]
    build_artifact: Callable[..., CompileArtifact]
    kernel_groups: tuple[str, ...] = ("core",)          # libraries the family needs (cacheir_b200.build)


_FAMILIES: dict[str, ModelFamily] = {}
LLAMA_SHAPED = ModelFamily("llama-shaped", ModelConfig.from_dict, build_decoder_artifact)


def register_family(architecture: str, family: ModelFamily) -> None:
    _FAMILIES[architecture] = family


def architectures() -> list[str]:
    """Architectures with a family of their own; any other one is taken as a Llama-shaped decoder."""
    return sorted(_FAMILIES)


def family_for(config: dict[str, Any]) -> ModelFamily:
    name = config.get("architecture") or (config.get("architectures") or [""])[0]
    return _FAMILIES.get(str(name), LLAMA_SHAPED)


def config_from_dict(data: dict[str, Any]) -> Any:
    return family_for(data).config_from_dict(data)


def load_model(path: str | Path, *, quant: str | None = None) -> CompileArtifact:
    """A model folder (config.json plus model.safetensors or weights.npz) as an artifact the runtime executes."""
    folder = Path(path)
    data = json.loads((folder / "config.json").read_text(encoding="utf-8"))
    family = family_for(data)
    return family.build_artifact(family.config_from_dict(data), model_path=str(folder), quant=quant)


register_family(gutorax.ARCHITECTURE, ModelFamily("gutorax", gutorax.GutoraxConfig.from_dict, gutorax.build_gutorax_artifact, ("ragged", "hybrid", "recurrence")))
register_family(topunex.ARCHITECTURE, ModelFamily("topunex", topunex.TopunexConfig.from_dict, topunex.build_topunex_artifact, ("ragged", "experts")))
register_family(rekodra.ARCHITECTURE, ModelFamily("rekodra", rekodra.RekodraConfig.from_dict, rekodra.build_rekodra_artifact,
                                                  ("ragged", "recurrence", "experts")))
register_family(zimorax.ARCHITECTURE, ModelFamily("zimorax", zimorax.ZimoraxConfig.from_dict, zimorax.build_zimorax_artifact,
                                                  ("ragged", "recurrence", "talking", "delta")))
