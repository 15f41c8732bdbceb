"""Sequence mixers and feed-forwards a decoder layer is put together from, beside the fixed
attention of llama.py: each is a module over the framework's linear layers (so deltas attach to its
projections) that runs on rows of normed hidden states, a PagedKVCache and an AttnMeta.

A mixer reads its sizes and constants from a spec and keeps what it remembers under its own run
number of the cache: a layer that is run several times per token has one run per pass.
`weight_views()` maps the mixer's checkpoint names (without the layer's prefix) to where they go."""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Dict, List

import torch
import torch.nn as nn

from . import layers as L
from . import ops
from .cache import AttnMeta, PagedKVCache


def _padded_rows(rows: int, width: int, dtype: torch.dtype) -> int:
    """Output rows of a stacked projection: filled up to whole 128-row tiles where the tcgen05 GEMM
    can take it (the surplus columns of its result are never read)."""
    tileable = dtype != torch.float32 and width % 64 == 0
    return (rows + 127) // 128 * 128 if tileable else rows


def _stacked(width: int, rows: int, device, dtype) -> L.ColumnParallelLinear:
    """A projection of `rows` rows (plus zero padding) for weights stacked by the caller."""
    total = _padded_rows(rows, width, dtype)
    linear = L.ColumnParallelLinear(width, total, device=device, dtype=dtype)
    with torch.no_grad():
        linear.weight[rows:] = 0
    return linear


def _vector(n: int, device, value: float = 0.0) -> nn.Parameter:
    """Norm weights and biases enter 32-bit arithmetic and are kept in 32 bits."""
    return nn.Parameter(torch.full((n,), value, dtype=torch.float32, device=device), requires_grad=False)


# ---------------------------------------------------------------------------
# sliding-window attention with a learned distance bias
# ---------------------------------------------------------------------------

@dataclass(frozen=True)
class WindowAttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    window: int
    scale: float
    bias_max: int

    @classmethod
    def from_dict(cls, d: dict) -> "WindowAttentionSpec":
        if set(d["mask"]) != {"size"}:
            raise ValueError(f"unknown attention mask {d['mask']}")
        spec = cls(int(d["heads"]), int(d["kv_heads"]), int(d["dim"]), int(d["vdim"]), int(d["mask"]["size"]),
                   float(d["scale"]), int(d["bias_max"]))
        if spec.heads % spec.kv_heads or spec.window < 1:
            raise ValueError("query heads must divide by the key/value heads and the window hold a token")
        return spec


def bucket_edges(rows: int, bias_max: int) -> List[int]:
    """First distance of every bucket of a `rows`-row table: bucket n is distance n up to half the
    rows, the others grow geometrically up to `bias_max`, where the last one is reached at the
    latest.  Distances are compared exactly: with h = rows / 2 and r = rows - h, distance n has
    passed k logarithmic steps when (n / h)^r >= (bias_max / h)^k."""
    half = rows // 2
    if rows < 2 or bias_max <= half:
        raise ValueError(f"a table of {rows} rows cannot be spread up to distance {bias_max}")
    edges, r = list(range(half + 1)), rows - half
    for k in range(1, r):
        goal = bias_max ** k * half ** (r - k)
        n = max(half, int(half * (bias_max / half) ** (k / r)) - 1)
        while n ** r < goal:
            n += 1
        edges.append(n)
    return edges


def distance_bias(rel: torch.Tensor, bias_max: int, window: int) -> torch.Tensor:
    """[heads, distances] bias per distance from a [rows, heads] table, as far as the window looks or
    to the first distance of the last bucket (farther distances repeat the last column)."""
    edges = torch.tensor(bucket_edges(rel.shape[0], bias_max))
    n = torch.arange(min(window, int(edges[-1]) + 1))
    bucket = torch.searchsorted(edges, n, right=True) - 1
    return rel[bucket.to(rel.device)].t().contiguous()


class WindowAttention(nn.Module):
    kind = "kv"

    def __init__(self, spec: WindowAttentionSpec, width: int, bias_rows: int, eps: float, device, dtype):
        super().__init__()
        self.spec, self.eps = spec, eps
        self.q_width, self.k_width = spec.heads * spec.dim, spec.kv_heads * spec.dim
        self.v_width = spec.kv_heads * spec.vdim
        self.qkv_proj = _stacked(width, self.q_width + self.k_width + self.v_width, device, dtype)
        self.o_proj = L.RowParallelLinear(spec.heads * spec.vdim, width, device=device, dtype=dtype)
        self.q_norm, self.k_norm = _vector(self.q_width, device, 1.0), _vector(self.k_width, device, 1.0)
        self.rel = nn.Parameter(torch.zeros((bias_rows, spec.heads), dtype=torch.float32, device=device),
                                requires_grad=False)
        self.bias = None

    def weight_views(self) -> Dict[str, torch.Tensor]:
        q, k, v = self.qkv_proj.weight[: self.q_width + self.k_width + self.v_width].split(
            [self.q_width, self.k_width, self.v_width])
        return {"q": q, "k": k, "v": v, "o": self.o_proj.weight, "q.norm": self.q_norm, "k.norm": self.k_norm,
                "rel": self.rel}

    def prepare(self) -> None:
        """After the weights are final."""
        self.bias = distance_bias(self.rel, self.spec.bias_max, self.spec.window)

    def forward(self, h: torch.Tensor, cache: PagedKVCache, run: int, meta: AttnMeta) -> torch.Tensor:
        s = self.spec
        kc, vc = cache.k[run], cache.v[run]
        qkv = self.qkv_proj(h)[0]
        if meta.decode:
            ops.qk_norm(qkv, self.q_norm, self.k_norm, self.v_width, self.eps, kc, vc, meta.slot_mapping)
        else:
            ops.qk_norm(qkv, self.q_norm, self.k_norm, self.v_width, self.eps)
        att = ops.window_attention(qkv, kc, vc, meta.block_tables, meta.q_starts, meta.ctx_lens, meta.max_query,
                                   meta.decode, s.heads, cache.block_size, s.scale, s.window, self.bias)
        if not meta.decode:
            # only now: the ring may hold exactly one window, which the portion's first rows still read
            ops.kv_append(qkv, self.q_width, kc, vc, meta.slot_mapping)
        return self.o_proj(att)[0]


# ---------------------------------------------------------------------------
# matrix memory with exponential gates
# ---------------------------------------------------------------------------

@dataclass(frozen=True)
class MlstmSpec:
    heads: int
    dim: int
    vdim: int
    gate_cap: float

    @classmethod
    def from_dict(cls, d: dict) -> "MlstmSpec":
        return cls(int(d["heads"]), int(d["dim"]), int(d["vdim"]), float(d["gate_cap"]))


class Mlstm(nn.Module):
    kind = "state"
    # portions up to this many tokens go through the recurrent kernel, longer ones 64 at a time
    RECURRENT_TOKENS = 4

    def __init__(self, spec: MlstmSpec, width: int, eps: float, device, dtype):
        super().__init__()
        self.spec, self.eps = spec, eps
        self.qk, self.vw = spec.heads * spec.dim, spec.heads * spec.vdim
        self.qkvg_proj = _stacked(width, 2 * self.qk + 2 * self.vw, device, dtype)
        self.o_proj = L.RowParallelLinear(self.vw, width, device=device, dtype=dtype)
        self.norm = _vector(self.vw, device, 1.0)
        self.gate_weight = nn.Parameter(torch.zeros((2 * spec.heads, width), dtype=dtype, device=device),
                                        requires_grad=False)
        self.gate_bias = _vector(2 * spec.heads, device)
        self.chunkwise = ops.mlstm_chunk_supported(spec.dim, spec.vdim, dtype)

    def weight_views(self) -> Dict[str, torch.Tensor]:
        q, k, v, g = self.qkvg_proj.weight[: 2 * self.qk + 2 * self.vw].split([self.qk, self.qk, self.vw, self.vw])
        n = self.spec.heads
        return {"q": q, "k": k, "v": v, "g": g, "o": self.o_proj.weight, "norm": self.norm,
                "i": self.gate_weight[:n], "f": self.gate_weight[n:], "i.b": self.gate_bias[:n],
                "f.b": self.gate_bias[n:]}

    def prepare(self) -> None:
        pass

    def forward(self, h: torch.Tensor, cache: PagedKVCache, run: int, meta: AttnMeta) -> torch.Tensor:
        s, st = self.spec, cache.state
        x = self.qkvg_proj(h)[0]
        o = ops.mlstm(x, h, self.gate_weight, self.gate_bias, self.norm, st.S[run], st.n[run], st.m[run],
                      meta.state_slots, meta.q_starts, meta.ctx_lens, s.gate_cap, 1.0 / math.sqrt(s.dim), self.eps,
                      chunkwise=self.chunkwise and meta.max_query > self.RECURRENT_TOKENS)
        return self.o_proj(o)[0]


# ---------------------------------------------------------------------------
# feed-forward
# ---------------------------------------------------------------------------

class GatedMLP(nn.Module):
    """down(act(gate h) * up h)."""

    def __init__(self, width: int, ff: int, activation: str, device, dtype):
        super().__init__()
        self.ff, self.activation = ff, activation
        self.gate_up_proj = L.MergedColumnParallelLinear(width, [ff, ff], device=device, dtype=dtype)
        self.down_proj = L.RowParallelLinear(ff, width, device=device, dtype=dtype)

    def weight_views(self) -> Dict[str, torch.Tensor]:
        gate, up = self.gate_up_proj.weight.split([self.ff, self.ff])
        return {"gate": gate, "up": up, "down": self.down_proj.weight}

    def forward(self, h: torch.Tensor) -> torch.Tensor:
        return self.down_proj(ops.gated_act(self.gate_up_proj(h)[0], self.activation))[0]
