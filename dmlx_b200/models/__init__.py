"""Models by configuration: a folder with config.json and model.safetensors becomes a model on the device.

Each architecture registers a loader under the names its config.json may carry: `load_model(path)` reads the
configuration, picks the loader and returns a `LoadedModel`, which the engine, the command line and the trace replay
all drive the same way.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Callable, Dict, Optional

PAGE_TOKENS = 32
_REGISTRY: Dict[str, Callable] = {}


class UnsupportedDtype(ValueError):
    """The architecture does not run in the requested number format."""


class ConfigError(ValueError):
    """config.json describes something the architecture does not have."""


@dataclass
class Limits:
    """Sizes the step buffers are made for."""

    max_rows: int = 2048  # rows (tokens) of one step
    max_reqs: int = 64    # requests in one step
    max_seqs: int = 64    # sequence slots


@dataclass
class LoadedModel:
    name: str
    model: object            # device.Model
    new_cache: Callable      # (n_pages, max_pages_per_seq) -> PagedKVCache with limits.max_seqs slots
    vocab: int
    limits: Limits


def register(*names: str):
    """Decorator: `loader(config, folder, dtype, limits) -> LoadedModel` for these architecture names."""

    def add(loader):
        for n in names:
            if n in _REGISTRY:
                raise ValueError(f"architecture {n} is registered twice")
            _REGISTRY[n] = loader
        return loader

    return add


def architecture_of(config: dict) -> str:
    """The registered name a configuration asks for."""
    names = [config.get("architecture"), *(config.get("architectures") or []), config.get("model_type")]
    for n in names:
        if n in _REGISTRY:
            return n
    raise ConfigError(f"no loader for {[n for n in names if n]} (known: {', '.join(sorted(_REGISTRY))})")


def load_config(folder: str) -> dict:
    with open(os.path.join(folder, "config.json")) as f:
        return json.load(f)


def load_model(folder: str, dtype: str = "bfloat16", limits: Optional[Limits] = None) -> LoadedModel:
    if dtype not in ("bfloat16", "float32"):
        raise UnsupportedDtype(f"unknown number format {dtype}")
    config = load_config(folder)
    name = architecture_of(config)
    return _REGISTRY[name](config, folder, dtype, limits or Limits())


from . import dovorax, llama, lorulix, sotavik, tafuvik  # noqa: E402,F401  (each registers itself)
