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
from .cache import AttnMeta, PagedKVCache, RecurrentStateCache
from .loader import copy_weights
from .mixers import GatedMLP, Mlstm, MlstmSpec, WindowAttention, WindowAttentionSpec
from .parallel_state import get_tensor_model_parallel_world_size

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


class BuzalornLayer(nn.Module):
    def __init__(self, spec: LayerSpec, cfg: BuzalornConfig, bias_rows: int, device, dtype):
        super().__init__()
        if isinstance(spec.mixer, MlstmSpec):
            self.mixer = Mlstm(spec.mixer, cfg.width, cfg.eps, device, dtype)
        else:
            self.mixer = WindowAttention(spec.mixer, cfg.width, bias_rows, cfg.eps, device, dtype)
        norm = lambda: nn.Parameter(torch.zeros(cfg.width, dtype=torch.float32, device=device), requires_grad=False)
        self.norm1 = norm()
        self.mlp = self.norm2 = None
        if spec.ff is not None:
            self.norm2 = norm()
            self.mlp = GatedMLP(cfg.width, spec.ff, "gelu_tanh", device, dtype)


class BuzalornForCausalLM(nn.Module):
    supported_delta_modules = ["qkv_proj", "qkvg_proj", "o_proj", "gate_up_proj", "down_proj"]
    packed_modules_mapping = {"gate_up_proj": ["gate_proj", "up_proj"]}
    supports_portions = True            # a prompt may be continued from the cache and state

    def __init__(self, cfg: BuzalornConfig, device="cuda", seed: int = 0, dtype=torch.bfloat16,
                 bias_rows: Union[int, Dict[int, int]] = DEFAULT_BIAS_ROWS):
        """`bias_rows`: rows of the attention layers' distance tables (per layer index when a dict); it
        is a tensor's shape, not a configuration value."""
        super().__init__()
        if get_tensor_model_parallel_world_size() != 1:
            raise ValueError("this model runs on one rank")
        # 16-bit GEMMs accumulate in 32 bits throughout, 32-bit ones use no reduced-precision mode
        torch.backends.cuda.matmul.allow_bf16_reduced_precision_reduction = False
        torch.backends.cuda.matmul.allow_fp16_reduced_precision_reduction = False
        if dtype == torch.float32:
            torch.backends.cuda.matmul.allow_tf32 = False
        self.cfg, self.dtype = cfg, dtype
        gen = torch.Generator(device=device).manual_seed(seed)
        par = lambda *shape, std, dt=dtype: nn.Parameter(
            torch.empty(shape, dtype=dt, device=device).normal_(0, std, generator=gen), requires_grad=False)
        f32 = torch.float32
        self.embed_tokens = par(cfg.vocab_size, cfg.width, std=1.0)
        self.embed_norm, self.norm = par(cfg.width, std=0.0, dt=f32), par(cfg.width, std=0.0, dt=f32)
        self.loop_in = par(cfg.width, 2 * cfg.width, std=(2 * cfg.width) ** -0.5)
        self.loop_step = par(cfg.loop_times, cfg.width, std=0.1, dt=f32)
        rows = (lambda i: bias_rows[i]) if isinstance(bias_rows, dict) else (lambda i: bias_rows)
        self.layers = nn.ModuleList([
            BuzalornLayer(spec, cfg, rows(i) if isinstance(spec.mixer, WindowAttentionSpec) else 0, device, dtype)
            for i, spec in enumerate(cfg.layers)])
        # cache runs: the n-th key/value pool or state pool belongs to the n-th such layer run
        self.plan, count = [], {"kv": 0, "state": 0}
        self._kv_shapes, self._state_shapes = [], []
        for i, first_of_pass in cfg.runs():
            s, kind = cfg.layers[i].mixer, self.layers[i].mixer.kind
            self.plan.append((self.layers[i], count[kind], first_of_pass))
            count[kind] += 1
            if kind == "kv":
                self._kv_shapes.append((s.kv_heads, s.dim, s.vdim))
            else:
                self._state_shapes.append((s.heads, s.dim, s.vdim))
        windows = [x.mixer.window for x in cfg.layers if isinstance(x.mixer, WindowAttentionSpec)]
        self.window = max(windows, default=0)
        self.kv_heads = max([h for h, _, _ in self._kv_shapes], default=1)
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

    def load_weights(self, tensors: Dict[str, torch.Tensor]) -> None:
        want = {"embed": [self.embed_tokens], "embed.norm": [self.embed_norm], "final.norm": [self.norm],
                "loop.in": [self.loop_in], "loop.step": [self.loop_step]}
        for i, layer in enumerate(self.layers):
            want[f"l{i}.norm1"] = [layer.norm1]
            want.update({f"l{i}.mix.{k}": [v] for k, v in layer.mixer.weight_views().items()})
            if layer.mlp is not None:
                want[f"l{i}.norm2"] = [layer.norm2]
                want.update({f"l{i}.mlp.{k}": [v] for k, v in layer.mlp.weight_views().items()})
        copy_weights(want, tensors)
        self.finalize()

    def finalize(self) -> None:
        for layer in self.layers:
            layer.mixer.prepare()

    # -- cache -------------------------------------------------------------------------
    def make_cache(self, num_blocks: int, block_size: int, max_seqs: int) -> PagedKVCache:
        device = self.embed_tokens.device
        state = RecurrentStateCache(self._state_shapes, max_seqs, device) if self._state_shapes else None
        return PagedKVCache(len(self._kv_shapes), num_blocks, self.kv_heads, block_size, self.dtype, device,
                            layer_shapes=self._kv_shapes, window=self.window, state=state)

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

    def greedy_tokens(self, hidden: torch.Tensor) -> torch.Tensor:
        return self.logits(hidden).argmax(dim=-1)
