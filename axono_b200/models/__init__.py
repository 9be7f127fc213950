"""Model registry: which class runs a model folder is decided by the "architecture" of its config.json.

    from axono_b200 import models
    model = models.load("path/to/folder", dtype=torch.bfloat16)     # config.json + model.safetensors
    models.create(config_dict, weights, dtype=...)                  # the same from memory

A registered class takes (config, weights, dtype, device) and offers what `axono_b200.serving` drives:
`cache_rows` (elements one token caches in each cache layer), `state_shapes` (what one sequence keeps in each state
layer, as (shape, dtype) pairs), `vocab`, `takes_segment(n)` and `forward(tokens, rows, cache, want)`; `kernel_sources` names the CUDA sources it needs
beyond those that every model does.
`TextTower`, the decode step of the reference's own model, is listed by name for `config_of`; it makes its
random weights itself and is stepped directly (axono_b200.decode, axono_b200.native_tower).
"""
from __future__ import annotations

import json
import os

_REGISTRY = {}


def register(architecture: str):
    def add(cls):
        _REGISTRY[architecture] = cls
        return cls

    return add


def architectures():
    from . import nuderax, rigozen  # noqa: F401 - they register themselves

    return sorted(_REGISTRY)


def model_class(architecture: str):
    if architecture not in architectures():
        raise ValueError(f"unknown architecture {architecture!r}; known: {', '.join(architectures())}")
    return _REGISTRY[architecture]


def config_of(config: dict):
    """The parsed configuration object of a config.json."""
    if config.get("architecture") == "TextTower":
        from ..tower_config import TextTowerConfig

        return TextTowerConfig(**{k: tuple(v) if isinstance(v, list) else v for k, v in config.items() if k != "architecture"})
    return model_class(config.get("architecture")).config_class.parse(config)


def use_library_for(folder: str) -> None:
    """Makes the library that the folder's design needs the one this process loads (see axono_b200.build)."""
    from .. import _capi

    with open(os.path.join(folder, "config.json")) as f:
        architecture = json.load(f).get("architecture")
    _capi.use_serving_library(architecture, model_class(architecture).kernel_sources)


def create(config: dict, weights, dtype, device="cuda"):
    """weights: name -> tensor (any device) or an open `weights.SafetensorsFile`."""
    cls = model_class(config.get("architecture"))
    return cls(cls.config_class.parse(config), weights, dtype, device)


def load(folder: str, dtype, device="cuda"):
    from .weights import SafetensorsFile

    with open(os.path.join(folder, "config.json")) as f:
        config = json.load(f)
    with SafetensorsFile(os.path.join(folder, "model.safetensors")) as weights:
        return create(config, weights, dtype, device)
