"""Buzalorn: a decoder-only model whose layers are listed one by one in its configuration -- sliding-
window attention with a distance bias, or a matrix memory (mLSTM), each with or without a gated
feed-forward -- with a span of layers that is run several times per token.

Every pass over the span has its own cache or state.  In front of a pass the residual x becomes
W [x; x0] + step[pass], x0 being the embedding output.  The residual stream is 32-bit throughout;
norm weights are stored around zero.

A forward pass is a chain of this library's launches like the Llama one: per layer residual add +
norm, stacked projection, the mixer's kernels, output projection, residual add + norm, gate/up
projection, gated activation, down projection."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional, Tuple, Union

import torch
import torch.nn as nn

from . import ops
from .cache import AttnMeta, PagedKVCache
from .decoder import DecoderLayer, LayeredDecoder
from .mixers import GatedMLP, Mlstm, MlstmSpec, WindowAttention, WindowAttentionSpec

NORM_OFFSET = 1.0                       # norms multiply by (1 + w)
DEFAULT_BIAS_ROWS = 32                  # of a model made without a checkpoint


@dataclass(frozen=True)
class LayerSpec:
    mixer: Union[WindowAttentionSpec, MlstmSpec]
    ff: Optional[int]                   # width of the gated feed-forward, None: the layer has none

    @classmethod
    def from_dict(cls, d: dict) -> "LayerSpec":
        specs = {"attention": WindowAttentionSpec, "mlstm": MlstmSpec}
        if d["type"] not in specs:
            raise ValueError(f"unknown mixer type {d['type']!r}")
        mlp = d.get("mlp")
        if mlp is not None and mlp["kind"] != "dense":
            raise ValueError(f"unknown feed-forward kind {mlp['kind']!r}")
        return cls(specs[d["type"]].from_dict(d["mixer"]), None if mlp is None else int(mlp["ff"]))


@dataclass(frozen=True)
class BuzalornConfig:
    vocab_size: int
    width: int
    layers: Tuple[LayerSpec, ...]
    loop_start: int
    loop_stop: int
    loop_times: int
    eps: float
    logit_scale: float

    @classmethod
    def from_dict(cls, d: dict) -> "BuzalornConfig":
        layers = tuple(LayerSpec.from_dict(x) for x in d["layers"])
        loop = d["loop"]
        cfg = cls(int(d["vocab"]), int(d["width"]), layers, int(loop["start"]), int(loop["stop"]), int(loop["times"]),
                  float(d["norm"]["eps"]), float(d["logit_scale"]))
        if not 0 <= cfg.loop_start < cfg.loop_stop <= len(layers) or cfg.loop_times < 1:
            raise ValueError(f"loop {loop} does not fit {len(layers)} layers")
        return cfg

    def runs(self) -> List[Tuple[int, Optional[int]]]:
        """(layer, pass that starts in front of it or None) of every layer run, in order."""
        out: List[Tuple[int, Optional[int]]] = [(i, None) for i in range(self.loop_start)]
        for t in range(self.loop_times):
            out += [(i, t if i == self.loop_start else None) for i in range(self.loop_start, self.loop_stop)]
        return out + [(i, None) for i in range(self.loop_stop, len(self.layers))]


class BuzalornForCausalLM(LayeredDecoder):
    supported_delta_modules = ["qkv_proj", "qkvg_proj", "o_proj", "gate_up_proj", "down_proj"]
    packed_modules_mapping = {"gate_up_proj": ["gate_proj", "up_proj"]}

    def __init__(self, cfg: BuzalornConfig, device="cuda", seed: int = 0, dtype=torch.bfloat16,
                 bias_rows: Union[int, Dict[int, int]] = DEFAULT_BIAS_ROWS):
        """`bias_rows`: rows of the attention layers' distance tables (per layer index when a dict); it
        is a tensor's shape, not a configuration value."""
        super().__init__(cfg, device, seed, dtype)
        f32, w = torch.float32, cfg.width
        self.embed_tokens = self._random(cfg.vocab_size, w, std=1.0)
        self.embed_norm, self.norm = self._random(w, std=0.0, dtype=f32), self._random(w, std=0.0, dtype=f32)
        self.loop_in = self._random(w, 2 * w, std=(2 * w) ** -0.5)
        self.loop_step = self._random(cfg.loop_times, w, std=0.1, dtype=f32)
        self.layers = nn.ModuleList()
        for i, spec in enumerate(cfg.layers):
            if isinstance(spec.mixer, MlstmSpec):
                mixer = Mlstm(spec.mixer, w, cfg.eps, device, dtype)
            else:
                rows = bias_rows[i] if isinstance(bias_rows, dict) else bias_rows
                mixer = WindowAttention(spec.mixer, w, rows, cfg.eps, device, dtype)
            mlp = GatedMLP(w, spec.ff, "gelu_tanh", device, dtype) if spec.ff is not None else None
            self.layers.append(DecoderLayer(mixer, mlp, w, 0.0, device))
        runs = self.plan_cache([i for i, _ in cfg.runs()])
        self.plan = [(self.layers[i], run, first_of_pass) for (i, first_of_pass), run in zip(cfg.runs(), runs)]
        self.finalize()

    # -- weights -----------------------------------------------------------------------
    @classmethod
    def from_tensors(cls, cfg: BuzalornConfig, tensors: Dict[str, torch.Tensor], device="cuda",
                     dtype=torch.bfloat16) -> "BuzalornForCausalLM":
        """Sizes that only a tensor's shape tells come from the checkpoint."""
        rows = {i: tensors[f"l{i}.mix.rel"].shape[0] for i, x in enumerate(cfg.layers)
                if isinstance(x.mixer, WindowAttentionSpec)}
        model = cls(cfg, device=device, dtype=dtype, bias_rows=rows)
        model.load_weights(tensors)
        return model

    def top_weights(self) -> Dict[str, torch.Tensor]:
        return {"embed": self.embed_tokens, "embed.norm": self.embed_norm, "final.norm": self.norm,
                "loop.in": self.loop_in, "loop.step": self.loop_step}

    # -- forward -----------------------------------------------------------------------
    def forward(self, tokens: torch.Tensor, positions: torch.Tensor, cache: PagedKVCache, meta: AttnMeta,
                trace: Optional[list] = None) -> torch.Tensor:
        """tokens [M] (int64); returns the hidden states [M, width] after the final norm.  `positions` are
        implied by `meta` and not read.  `trace`, when a list, receives the residual after every layer
        run."""
        cfg, eps, dt = self.cfg, self.cfg.eps, self.dtype
        m, width = tokens.shape[0], cfg.width
        both = torch.empty((m, 2 * width), dtype=dt, device=tokens.device)         # [x; x0]
        x = ops.embed_norm(tokens, self.embed_tokens, self.embed_norm, eps, NORM_OFFSET, copy=both[:, width:])
        delta = None                                                               # not yet added to x
        for layer, run, first_of_pass in self.plan:
            if first_of_pass is None:
                h = ops.residual_norm(x, delta, layer.norm1, eps, dt, NORM_OFFSET)
            else:
                ops.residual_norm(x, delta, None, eps, dt, out=both[:, :width])
                h = ops.residual_norm(x, ops.matmul_f32(both, self.loop_in), layer.norm1, eps, dt, NORM_OFFSET,
                                      vec=self.loop_step[first_of_pass], replace=True)
            delta = layer.mixer(h, cache, run, meta)
            if layer.mlp is not None:
                h = ops.residual_norm(x, delta, layer.norm2, eps, dt, NORM_OFFSET)
                delta = layer.mlp(h)
            if trace is not None:
                trace.append(x + delta)
        return ops.residual_norm(x, delta, self.norm, eps, dt, NORM_OFFSET)

    # -- sampling ------------------------------------------------------------------------
    def logits(self, hidden: torch.Tensor) -> torch.Tensor:
        """float32 logits; the output matrix is the embedding table."""
        return ops.matmul_f32(hidden, self.embed_tokens) * self.cfg.logit_scale
