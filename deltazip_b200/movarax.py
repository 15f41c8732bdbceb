"""Movarax: a decoder-only model whose layers are listed one by one in its configuration -- attention over
a cached latent with a sink per head, where a layer may read another one's latents, or linear attention
with a constant decay per head -- each with a gated feed-forward, with routed experts or with neither.

The residual stream is 32-bit throughout; norms are plain RMS norms; the output matrix is its own.  A
forward pass is a chain of this library's launches: per layer residual add + norm, stacked projection,
the mixer's kernels, output projection, residual add + norm, feed-forward; the routed experts' outputs
are summed by the next residual step."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, Optional, Tuple, Union

import torch
import torch.nn as nn

from . import ops
from .cache import AttnMeta, PagedKVCache
from .decoder import DecoderLayer, LayeredDecoder
from .mixers import (GatedMLP, LatentAttention, LatentAttentionSpec, Lightning, LightningSpec, RoutedExperts,
                     RoutedExpertsSpec)

MIXERS = {"latent_attention": LatentAttentionSpec, "lightning": LightningSpec, "lightning_2": LightningSpec}


@dataclass(frozen=True)
class LayerSpec:
    mixer: Union[LatentAttentionSpec, LightningSpec]
    mlp: Union[None, int, RoutedExpertsSpec]            # int: width of a gated feed-forward

    @classmethod
    def from_dict(cls, d: dict) -> "LayerSpec":
        if d["type"] not in MIXERS:
            raise ValueError(f"unknown mixer type {d['type']!r}")
        mlp = d.get("mlp")
        if mlp is not None:
            if mlp["kind"] not in ("dense", "moe"):
                raise ValueError(f"unknown feed-forward kind {mlp['kind']!r}")
            mlp = int(mlp["ff"]) if mlp["kind"] == "dense" else RoutedExpertsSpec.from_dict(mlp)
        return cls(MIXERS[d["type"]].from_dict(d["mixer"]), mlp)


@dataclass(frozen=True)
class MovaraxConfig:
    vocab_size: int
    width: int
    layers: Tuple[LayerSpec, ...]
    eps: float
    embed_scale: float

    @classmethod
    def from_dict(cls, d: dict) -> "MovaraxConfig":
        cfg = cls(int(d["vocab"]), int(d["width"]), tuple(LayerSpec.from_dict(x) for x in d["layers"]),
                  float(d["norm"]["eps"]), float(d["embedding"]["scale"]))
        for i, layer in enumerate(cfg.layers):
            owner = getattr(layer.mixer, "kv_from", None)
            if owner is None:
                continue
            own = cfg.layers[owner].mixer if 0 <= owner < i else None
            if not isinstance(own, LatentAttentionSpec) or own.kv_from is not None or \
                    (own.kv_rank, own.rot_dim, own.rot_base) != (layer.mixer.kv_rank, layer.mixer.rot_dim, layer.mixer.rot_base):
                raise ValueError(f"layer {i} cannot read the latents of layer {owner}")
        return cfg


class MovaraxForCausalLM(LayeredDecoder):
    # the matrices between latent and heads, the router and the routed experts take no deltas
    supported_delta_modules = ["q_latent_proj", "qkvg_proj", "o_proj", "gate_up_proj", "up_proj", "down_proj"]
    packed_modules_mapping = {"gate_up_proj": ["gate_proj", "up_proj"]}

    def __init__(self, cfg: MovaraxConfig, device="cuda", seed: int = 0, dtype=torch.bfloat16):
        super().__init__(cfg, device, seed, dtype)
        w = cfg.width
        self.embed_tokens = self._random(cfg.vocab_size, w, std=1.0)
        self.lm_head = self._random(cfg.vocab_size, w, std=w ** -0.5)
        self.norm = nn.Parameter(torch.ones(w, dtype=torch.float32, device=device), requires_grad=False)
        self.layers = nn.ModuleList()
        for spec in cfg.layers:
            kind = Lightning if isinstance(spec.mixer, LightningSpec) else LatentAttention
            mlp = None
            if isinstance(spec.mlp, RoutedExpertsSpec):
                mlp = RoutedExperts(spec.mlp, w, "relu2", device, dtype)
            elif spec.mlp is not None:
                mlp = GatedMLP(w, spec.mlp, "silu", device, dtype)
            self.layers.append(DecoderLayer(kind(spec.mixer, w, cfg.eps, device, dtype), mlp, w, 1.0, device))
        self.plan = list(zip(self.layers, self.plan_cache(range(len(cfg.layers)))))
        self.finalize()

    @classmethod
    def from_tensors(cls, cfg: MovaraxConfig, tensors: Dict[str, torch.Tensor], device="cuda",
                     dtype=torch.bfloat16) -> "MovaraxForCausalLM":
        model = cls(cfg, device=device, dtype=dtype)
        model.load_weights(tensors)
        return model

    def top_weights(self) -> Dict[str, torch.Tensor]:
        return {"embed": self.embed_tokens, "final.norm": self.norm, "head": self.lm_head}

    def forward(self, tokens: torch.Tensor, positions: torch.Tensor, cache: PagedKVCache, meta: AttnMeta,
                trace: Optional[list] = None) -> torch.Tensor:
        """tokens [M] (int64) at `positions` (int64); returns the hidden states [M, width] after the final
        norm.  `trace`, when a list, receives the residual after every layer."""
        eps, dt = self.cfg.eps, self.dtype
        meta.positions = positions
        x = ops.embed_norm(tokens, self.embed_tokens, None, eps, scale=self.cfg.embed_scale)
        delta = None                                                               # not yet added to x
        for layer, run in self.plan:
            h = ops.residual_norm(x, delta, layer.norm1, eps, dt)
            delta = layer.mixer(h, cache, run, meta)
            if layer.mlp is not None:
                h = ops.residual_norm(x, delta, layer.norm2, eps, dt)
                delta = layer.mlp(h)
            if trace is not None:
                trace.append(x + (delta.dense() if isinstance(delta, ops.Update) else delta))
        return ops.residual_norm(x, delta, self.norm, eps, dt)

    def logits(self, hidden: torch.Tensor) -> torch.Tensor:
        """float32 logits."""
        return ops.matmul_f32(hidden, self.lm_head)
