"""One registry from an architecture's name to its configuration and model.

The name is ``config.json["architectures"][0]`` (or the single name under
``"architecture"``); a file without either key is looked up by ``model_type``.  (The reference has no registry: it keys on
``model_type`` alone, src/dli/model/config.py:91-93.)
"""

from __future__ import annotations

import json
from dataclasses import dataclass
from pathlib import Path
from typing import Any, Callable

from .gedunex import GedunexConfig, gedunex_model_spec
from .llama import LlamaConfig, UnsupportedModelError, llama_model_spec
from .lokolorn import LokolornConfig, lokolorn_model_spec
from .novunex import NovunexConfig, novunex_model_spec
from .pazenex import PazenexConfig, pazenex_model_spec
from .pokadra import PokadraConfig, pokadra_model_spec
from .spec import ModelSpec
from .sugonex import SugonexConfig, sugonex_model_spec


@dataclass(frozen=True)
class Architecture:
    name: str
    parse_config: Callable[[dict[str, Any]], Any]  # config.json dict -> typed configuration
    model_spec: Callable[[Any], ModelSpec]  # typed configuration -> parts and run order
    model_types: tuple[str, ...] = ()  # model_type values that also select it


_ARCHITECTURES: dict[str, Architecture] = {}


def register_architecture(arch: Architecture) -> None:
    _ARCHITECTURES[arch.name] = arch


def unregister_architecture(name: str) -> None:
    _ARCHITECTURES.pop(name, None)


def resolve_architecture(cfg: dict[str, Any]) -> Architecture:
    names = cfg.get("architectures") or ([cfg["architecture"]] if cfg.get("architecture") else [])
    if names:
        if names[0] in _ARCHITECTURES:
            return _ARCHITECTURES[names[0]]
        raise UnsupportedModelError(f"architecture {names[0]!r} is not registered (known: {sorted(_ARCHITECTURES)})")
    model_type = cfg.get("model_type")
    for arch in _ARCHITECTURES.values():
        if model_type in arch.model_types:
            return arch
    raise UnsupportedModelError(f"model_type={model_type!r} is not registered (known: {sorted(_ARCHITECTURES)})")


def load_config(model_dir: str | Path) -> tuple[Architecture, Any]:
    """Parse ``config.json`` of a model folder (src/dli/model/loader.py:38-40)."""
    cfg = json.loads((Path(model_dir) / "config.json").read_text())
    arch = resolve_architecture(cfg)
    return arch, arch.parse_config(cfg)


register_architecture(
    Architecture("LlamaForCausalLM", LlamaConfig.from_hf_dict, llama_model_spec, model_types=("llama",))
)
register_architecture(Architecture("Pazenex", PazenexConfig.from_dict, pazenex_model_spec))
register_architecture(Architecture("Sugonex", SugonexConfig.from_dict, sugonex_model_spec))
register_architecture(Architecture("Pokadra", PokadraConfig.from_dict, pokadra_model_spec))
register_architecture(Architecture("Lokolorn", LokolornConfig.from_dict, lokolorn_model_spec))
register_architecture(Architecture("Gedunex", GedunexConfig.from_dict, gedunex_model_spec))
register_architecture(Architecture("Novunex", NovunexConfig.from_dict, novunex_model_spec))
