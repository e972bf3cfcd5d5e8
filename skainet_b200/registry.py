"""Model registry: the `architecture` of a model folder's config.json -> how to load it.  A folder holds config.json
and model.safetensors."""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Callable, Dict

from .safetensors import SafetensorsFile


@dataclass
class Architecture:
    name: str
    family: str          # build.FAMILIES entry with its kernels
    load: Callable       # (ctx, config dict, weights, **kw) -> decoder


ARCHITECTURES: Dict[str, Architecture] = {}


def register(name: str, family: str):
    def wrap(fn):
        ARCHITECTURES[name] = Architecture(name, family, fn)
        return fn
    return wrap


def read_config(path: str) -> dict:
    with open(os.path.join(path, "config.json")) as f:
        return json.load(f)


def architecture_of(config: dict) -> Architecture:
    name = config.get("architecture")
    if name not in ARCHITECTURES:
        raise ValueError(f"unknown architecture {name!r} (known: {', '.join(sorted(ARCHITECTURES))})")
    return ARCHITECTURES[name]


def load_model(ctx, path: str, **kw):
    """Decoder of the model folder `path`; keywords go to its class (max_seqs, max_tokens, max_ctx, dtype)."""
    config = read_config(path)
    return architecture_of(config).load(ctx, config, SafetensorsFile(os.path.join(path, "model.safetensors")), **kw)
