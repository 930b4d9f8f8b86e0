"""Model registry: which class a model folder holds, and how it is read.

A folder holds either config.json + model.safetensors (``architecture`` in config.json names the class) or tnsr's own
parameter archive (manifest.json), which is a ``Gpt``.
"""
from __future__ import annotations

import json
import os
from typing import Callable, Dict

from .bolonex import Bolonex, BolonexConfig
from .described import DEFAULT_CONTEXT
from .ganupel import Ganupel, GanupelConfig
from .nn import CachedModel, TnsrError
from .parameters import load_gpt, read_safetensors

DTYPES = {"bfloat16": "bf16", "float32": "f32", "bf16": "bf16", "f32": "f32"}


def _bolonex(config: dict, tensors: dict, weight_dtype: str, max_sequence_length: int) -> CachedModel:
    return Bolonex(BolonexConfig.from_dict(config, weight_dtype, max_sequence_length), tensors)


def _ganupel(config: dict, tensors: dict, weight_dtype: str, max_sequence_length: int) -> CachedModel:
    return Ganupel(GanupelConfig.from_dict(config, weight_dtype, max_sequence_length), tensors)


# architecture name in config.json -> builder(config, tensors, weight_dtype, max_sequence_length)
ARCHITECTURES: Dict[str, Callable[[dict, dict, str, int], CachedModel]] = {"Bolonex": _bolonex, "Ganupel": _ganupel}


def load_model(directory: str, dtype: str = "bfloat16", max_sequence_length: int = DEFAULT_CONTEXT) -> CachedModel:
    if dtype not in DTYPES:
        raise TnsrError(f"unknown dtype {dtype!r}")
    path = os.path.join(directory, "config.json")
    if not os.path.exists(path):
        if os.path.exists(os.path.join(directory, "manifest.json")):
            model = load_gpt(directory)
            model.config().weight_dtype = DTYPES[dtype]
            return model
        raise TnsrError(f"{directory}: neither config.json nor manifest.json")
    with open(path, "rb") as f:
        try:
            config = json.loads(f.read())
        except ValueError as e:
            raise TnsrError(f"parse config.json: {e}")
    name = config.get("architecture")
    if name not in ARCHITECTURES:
        raise TnsrError(f"unknown architecture {name!r}; known: {sorted(ARCHITECTURES)}")
    return ARCHITECTURES[name](config, read_safetensors(os.path.join(directory, "model.safetensors")), DTYPES[dtype], max_sequence_length)
