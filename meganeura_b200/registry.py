"""Model registry: config.json's "architecture" (or a built-in decoder's name) -> how to build it.

Folders with a config.json and a model.safetensors are loaded with load_model; the built-in decode
shapes of decode_model.py are listed under their own names (they carry seeded weights).
"""
from __future__ import annotations

import os

from . import decode_model
from .petotar import Petotar
from .tobovik import Tobovik
from .weights import SafeTensors, read_config

ARCHITECTURES = {"Petotar": Petotar, "Tobovik": Tobovik}
DECODERS = {c.name: c for c in (decode_model.SMOLLM2_135M, decode_model.QWEN3_8B)}


def model_class(config: dict):
    name = config.get("architecture")
    if name not in ARCHITECTURES:
        raise ValueError(f"unknown architecture {name!r} (known: {', '.join(sorted(ARCHITECTURES))})")
    return ARCHITECTURES[name]


def load_model(folder: str, **kw):
    """kw: dtype ("bfloat16" / "float32"), max_rows, max_picked, max_tokens."""
    config = read_config(folder)
    return model_class(config).from_tensors(config, SafeTensors(os.path.join(folder, "model.safetensors")), **kw)
