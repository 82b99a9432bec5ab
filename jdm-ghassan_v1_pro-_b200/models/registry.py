"""Model families by what their files say they are.

A file or folder is turned into a configuration object, and the configuration decides the engine that serves it.  GGUF,
legacy and checkpoint files hold the MoE / dense decoder of ``models/config.py``; a folder with ``config.json`` names its
architecture, which is looked up here.  A further design made of known layer types is one more entry (of ``DESIGNS`` in ``models/layer_list.py``).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Callable, Dict

from .config import ModelConfig
from .layer_list import DESIGNS, LayerListConfig


@dataclass(frozen=True)
class Architecture:
    name: str
    config_type: type
    parse: Callable[[dict], object]            # parsed config.json -> configuration
    engine: str                                # "module:attribute" under the package, loaded when it is needed


ARCHITECTURES: Dict[str, Architecture] = {}


def register(a: Architecture) -> Architecture:
    ARCHITECTURES[a.name] = a
    return a


for _name in DESIGNS:
    register(Architecture(_name, LayerListConfig, LayerListConfig.from_json, "inference.layer_engine:LayerEngine"))


def from_json(d: dict) -> Architecture:
    """Architecture that a parsed ``config.json`` names."""
    name = d.get("architecture")
    if name not in ARCHITECTURES:
        raise ValueError("config.json names the architecture %r; known: %s" % (name, ", ".join(sorted(ARCHITECTURES))))
    return ARCHITECTURES[name]


def engine_class(cfg):
    """Engine class that serves a configuration (token-step engine of the MoE / dense decoder, or the registered one)."""
    import importlib
    where = "inference.engine:InferenceEngine"
    if not isinstance(cfg, ModelConfig):
        where = ARCHITECTURES[cfg.architecture].engine
    mod, attr = where.split(":")
    return getattr(importlib.import_module("ghassan_b200." + mod), attr)
