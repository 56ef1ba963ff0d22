"""Model families by the name that a config.json gives in "architecture"."""
from __future__ import annotations

import os
from typing import Optional

import torch

from . import _lib
from .checkpoint import Weights, read_config, read_safetensors

DTYPES = {"bfloat16": torch.bfloat16, "float32": torch.float32}


class UnsupportedDtype(RuntimeError):
    pass


def _llama(config: dict, weights: Optional[Weights], dtype):
    from dataclasses import fields
    from .layers import LLaMAConfig
    from .model import LLaMAModelBF16
    if dtype != torch.bfloat16:
        raise UnsupportedDtype("the LLaMA model runs in bfloat16")
    known = {f.name for f in fields(LLaMAConfig)}
    model = LLaMAModelBF16(LLaMAConfig(**{k: v for k, v in config.items() if k in known}))
    if weights is not None:
        model.load_weights(weights)
    return model


def _soluzen(config: dict, weights: Optional[Weights], dtype):
    from .soluzen import SoluzenConfig, SoluzenModel
    if weights is None:
        raise RuntimeError("a Soluzen model needs its checkpoint")
    return SoluzenModel(SoluzenConfig.from_dict(config), weights, dtype)


def _duponex(config: dict, weights: Optional[Weights], dtype):
    from .duponex import DuponexConfig, DuponexModel
    if weights is None:
        raise RuntimeError("a Duponex model needs its checkpoint")
    return DuponexModel(DuponexConfig.from_dict(config), weights, dtype)


# architecture -> (family whose kernels it launches, constructor)
ARCHITECTURES = {"LLaMA": ("llama", _llama), "Soluzen": ("soluzen", _soluzen), "Duponex": ("duponex", _duponex)}


def build_model(config: dict, weights: Optional[Weights], dtype=torch.bfloat16):
    """The model of a parsed config.json, its weights taken from `weights`."""
    name = config.get("architecture")
    if name not in ARCHITECTURES:
        raise RuntimeError(f"unknown architecture {name!r} (known: {', '.join(sorted(ARCHITECTURES))})")
    if dtype not in DTYPES.values():
        raise UnsupportedDtype(f"dtype {dtype}")
    family, make = ARCHITECTURES[name]
    _lib.load_family(family)
    return make(config, weights, dtype)


def load_model(folder: str, dtype: str = "bfloat16"):
    """The model in `folder` (config.json, model.safetensors); compiles the kernels it needs where they are missing."""
    if dtype not in DTYPES:
        raise UnsupportedDtype(f"dtype {dtype} (known: {', '.join(DTYPES)})")
    return build_model(read_config(folder), Weights(read_safetensors(os.path.join(folder, "model.safetensors"))), DTYPES[dtype])
