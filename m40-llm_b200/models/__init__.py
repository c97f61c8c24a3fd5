"""Model registry: config.json's "architecture" -> the class that reads that configuration and builds the model.

A design registers a function (config dict) -> spec; a spec has `vocab`, `width` and `build(nat, weights, ...) -> host.Model`.
"""
from __future__ import annotations

import json
import os

from ..weights import TensorFile

_REGISTRY: dict[str, object] = {}


def register(architecture: str):
    def add(reader):
        _REGISTRY[architecture] = reader
        return reader
    return add


def architectures() -> list[str]:
    return sorted(_REGISTRY)


def read_config(config: dict):
    arch = config.get("architecture")
    if arch not in _REGISTRY:
        raise ValueError(f"architecture {arch!r} is not one of {architectures()}")
    return _REGISTRY[arch](config)


def load(nat, directory: str, **options):
    """Model folder (config.json, model.safetensors) -> host.Model on `nat`'s device. Options: dtype ("bfloat16" or
    "float32"), sequences, max_len, max_rows."""
    with open(os.path.join(directory, "config.json")) as f:
        spec = read_config(json.load(f))
    return spec.build(nat, TensorFile(os.path.join(directory, "model.safetensors")), **options)


from . import lamutar, sidalorn  # noqa: E402,F401  (they register themselves)
