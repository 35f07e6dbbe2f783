"""Model families by the ``architecture`` of a configuration.

A family names its configuration class (``from_dict``), its model class (``cls(cfg, weights, device, dtype)``)
and the random initialisation of its parameters.  A configuration dict
without an ``architecture`` is the GQA / MLA decoder family.  The engine builds every model through
``build_model``; a folder with ``config.json`` and weights is read by ``utils.loader.load_model_dir``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Callable


@dataclass(frozen=True)
class ModelFamily:
    name: str
    config_cls: type
    model_cls: type
    init_weights: Callable              # (cfg, seed) -> {parameter name: CPU tensor}


_FAMILIES: dict[str, ModelFamily] = {}
DEFAULT_FAMILY = "TransformerLM"


def register(family: ModelFamily) -> ModelFamily:
    _FAMILIES[family.name] = family
    return family


def families() -> list[str]:
    return sorted(_FAMILIES)


def family_of(config) -> ModelFamily:
    """The family of a configuration object or dict."""
    if isinstance(config, dict):
        name = config.get("architecture", DEFAULT_FAMILY)
        if name not in _FAMILIES:
            raise ValueError(f"unknown architecture {name!r}; registered: {', '.join(families())}")
        return _FAMILIES[name]
    for fam in _FAMILIES.values():
        if isinstance(config, fam.config_cls):
            return fam
    raise TypeError(f"{type(config).__name__} is not a configuration of a registered model family")


def resolve_config(config):
    """Configuration object of a dict (objects pass through)."""
    return family_of(config).config_cls.from_dict(config) if isinstance(config, dict) else config


def build_model(config, weights, device, dtype):
    cfg = resolve_config(config)
    return family_of(cfg).model_cls(cfg, weights, device, dtype)


def init_weights(config, seed: int = 0) -> dict:
    cfg = resolve_config(config)
    return family_of(cfg).init_weights(cfg, seed)
