"""Model registry: ``config.json``'s "architecture" -> how to make an engine for it.

A builder takes the parsed configuration, a weight source (``get(name, shape)`` -> CPU or device tensor;
None for architectures without checkpoints) and engine options, and returns an object with the
step interface of ``engine.StepEngine``.
"""
from __future__ import annotations

import importlib
import os
from typing import Callable, Dict, Optional

from . import checkpoint

_MODULES = {                    # imported on first use: a model pulls in only its own kernels
    "Bidasun": "tensorwarp_b200.models.bidasun",
    "TWMarlinQ4": "tensorwarp_b200.models.tw_marlin",
    "Zukotar": "tensorwarp_b200.models.zukotar",
}
_BUILDERS: Dict[str, Callable] = {}


def register(name: str):
    def add(builder):
        _BUILDERS[name] = builder
        return builder
    return add


def architectures():
    return sorted(set(_MODULES) | set(_BUILDERS))


def builder_for(config: dict) -> Callable:
    name = config.get("architecture")
    if name not in _BUILDERS and name in _MODULES:
        importlib.import_module(_MODULES[name])
    if name not in _BUILDERS:
        raise checkpoint.CheckpointError(f"unknown architecture {name!r}; known: {', '.join(architectures())}")
    return _BUILDERS[name]


def load(folder: str, **options):
    """An engine for the checkpoint in `folder` (options: dtype, max_tokens, max_live, portion, device)."""
    config = checkpoint.read_config(folder)
    builder = builder_for(config)
    path = os.path.join(folder, "model.safetensors")
    weights: Optional[checkpoint.SafetensorsFile] = checkpoint.SafetensorsFile(path) if os.path.exists(path) else None
    try:
        return builder(config, weights, **options)
    finally:
        if weights is not None:
            weights.close()
