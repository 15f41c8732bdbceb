"""Model registry: architecture name in config.json -> configuration and model class (role of the
reference's ModelRegistry, serving/vllm/model_executor/models/__init__.py)."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Callable, Dict, Tuple

import torch

from . import loader
from .buzalorn import BuzalornConfig, BuzalornForCausalLM
from .llama import LlamaConfig, LlamaForCausalLM
from .movarax import MovaraxConfig, MovaraxForCausalLM


@dataclass(frozen=True)
class ModelEntry:
    name: str
    config_class: type
    model_class: type
    default_dtype: torch.dtype
    dtypes: Tuple[torch.dtype, ...]
    # (config, tensors, device, dtype) -> model with the checkpoint's weights
    from_tensors: Callable


def _llama_from_tensors(cfg, tensors, device, dtype):
    model = LlamaForCausalLM(cfg, device=device, dtype=dtype)
    model.load_weights(tensors)
    return model


_REGISTRY: Dict[str, ModelEntry] = {}


def register(entry: ModelEntry) -> None:
    _REGISTRY[entry.name] = entry


register(ModelEntry("LlamaForCausalLM", LlamaConfig, LlamaForCausalLM, torch.float16,
                    (torch.float16, torch.bfloat16), _llama_from_tensors))
register(ModelEntry("Buzalorn", BuzalornConfig, BuzalornForCausalLM, torch.bfloat16,
                    (torch.float16, torch.bfloat16, torch.float32), BuzalornForCausalLM.from_tensors))
register(ModelEntry("Movarax", MovaraxConfig, MovaraxForCausalLM, torch.bfloat16,
                    (torch.float16, torch.bfloat16, torch.float32), MovaraxForCausalLM.from_tensors))


def names():
    return sorted(_REGISTRY)


def lookup(config: dict) -> ModelEntry:
    """By "architecture", or the first known name of "architectures"."""
    named = [config["architecture"]] if "architecture" in config else list(config.get("architectures") or [])
    for name in named:
        if name in _REGISTRY:
            return _REGISTRY[name]
    raise ValueError(f"no model for architecture {named}; known: {names()}")


def entry_for(cfg) -> ModelEntry:
    for entry in _REGISTRY.values():
        if type(cfg) is entry.config_class:
            return entry
    raise ValueError(f"no model takes a {type(cfg).__name__}")


def build_model(cfg, device="cuda", seed: int = 0, dtype=None):
    """A randomly initialised model of a configuration object."""
    entry = entry_for(cfg)
    return entry.model_class(cfg, device=device, seed=seed, dtype=dtype or entry.default_dtype)


def load_model(path: str, device="cuda", dtype=None):
    """The model in a checkpoint folder, its class chosen by config.json.  Returns (config, model)."""
    raw = loader.read_config(path)
    entry = lookup(raw)
    dtype = dtype or entry.default_dtype
    if dtype not in entry.dtypes:
        raise ValueError(f"{entry.name} does not run in {dtype}")
    cfg = entry.config_class.from_dict(raw)
    return cfg, entry.from_tensors(cfg, loader.read_tensors(path), device, dtype)
