"""Base checkpoints: a folder with config.json and one or more safetensors files."""
from __future__ import annotations

import glob
import json
import os
from typing import Dict, Sequence

import torch


def read_config(path: str) -> dict:
    with open(os.path.join(path, "config.json")) as fh:
        return json.load(fh)


def read_tensors(path: str) -> Dict[str, torch.Tensor]:
    """All tensors of the folder's safetensors files, on the host."""
    from safetensors import safe_open
    files = sorted(glob.glob(os.path.join(path, "*.safetensors")))
    if not files:
        raise FileNotFoundError(f"no .safetensors file in {path}")
    out: Dict[str, torch.Tensor] = {}
    for name in files:
        with safe_open(name, framework="pt") as f:
            for key in f.keys():
                out[key] = f.get_tensor(key)
    return out


@torch.no_grad()
def copy_weights(want: Dict[str, Sequence[torch.Tensor]], tensors: Dict[str, torch.Tensor]) -> None:
    """Copies every checkpoint tensor into all of its destinations (views of parameters).  Names
    missing on either side and shapes that do not match are errors."""
    missing, extra = sorted(set(want) - set(tensors)), sorted(set(tensors) - set(want))
    if missing or extra:
        raise ValueError(f"checkpoint does not fit the model: missing {missing[:5]}, unexpected {extra[:5]}")
    for name, places in want.items():
        t = tensors[name]
        for dst in places:
            if tuple(t.shape) != tuple(dst.shape):
                raise ValueError(f"{name}: checkpoint has {tuple(t.shape)}, the model {tuple(dst.shape)}")
            dst.copy_(t)
