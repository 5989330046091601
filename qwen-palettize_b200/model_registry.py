"""Architectures by name, and loading of a model folder (config.json + model.safetensors). A model class offers

    from_config(config, tensors, dtype, device)      build from the parsed config.json and a mapping of stored tensors
    DTYPES                                           types it runs in
    new_cache(B, T_max), forward(ids, cache, want)   state of B sequences in lockstep; a step of n tokens each
    vocab
"""
from __future__ import annotations

import json
import os
import sys

import torch

_HERE = os.path.dirname(os.path.abspath(__file__))
if _HERE not in sys.path:
    sys.path.insert(0, _HERE)

import safetensors_io  # noqa: E402
from decode_model import PalettizedQwen  # noqa: E402
import hybrid_model  # noqa: E402

ARCHITECTURES = {**hybrid_model.ARCHITECTURES, "PalettizedQwen": PalettizedQwen}
DTYPES = {"bfloat16": torch.bfloat16, "float32": torch.float32}


class UnsupportedDtype(ValueError):
    pass


def read_config(folder: str) -> dict:
    with open(os.path.join(folder, "config.json")) as f:
        return json.load(f)


def model_class(config: dict):
    name = config.get("architecture")
    if name not in ARCHITECTURES:
        raise ValueError(f"unknown architecture {name!r}; known: {', '.join(sorted(ARCHITECTURES))}")
    return ARCHITECTURES[name]


def check_dtype(config: dict, dtype: str) -> torch.dtype:
    cls = model_class(config)
    if DTYPES[dtype] not in cls.DTYPES:
        raise UnsupportedDtype(f"{config['architecture']} does not run in {dtype}")
    return DTYPES[dtype]


def load_model(folder: str, dtype: str = "bfloat16", device="cuda"):
    config = read_config(folder)
    t = check_dtype(config, dtype)
    return model_class(config).from_config(config, safetensors_io.SafeTensors(os.path.join(folder, "model.safetensors")), t, device)


def save_model(folder: str, config: dict, tensors: dict):
    """Write a model folder that load_model reads."""
    model_class(config)
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(config, f, indent=1)
    safetensors_io.save(os.path.join(folder, "model.safetensors"), tensors)
