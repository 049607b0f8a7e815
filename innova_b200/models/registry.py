"""Architectures by name: which configuration and model class a ``config.json`` or a model file's header asks for.

A model directory (``config.json`` with an ``architecture`` key, ``model.safetensors``) and a ``.oil`` file of a registered
architecture load through ``formats.export.load_model`` like every other model."""
from __future__ import annotations

from typing import Dict

ARCHITECTURES: Dict[str, type] = {}


def register(name: str):
    def add(cls):
        ARCHITECTURES[name] = cls
        cls.architecture = name
        return cls
    return add


def model_class(config: dict) -> type:
    """The registered model class of a configuration dictionary."""
    from . import mekazen, vebesun  # noqa: F401  (they register themselves)
    name = config.get("architecture")
    if name not in ARCHITECTURES:
        raise ValueError(f"unknown architecture {name!r}; known: {', '.join(sorted(ARCHITECTURES))}")
    return ARCHITECTURES[name]
