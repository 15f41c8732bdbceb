"""Sequence mixers and feed-forwards a decoder layer is put together from, beside the fixed
attention of llama.py: each is a module over the framework's linear layers (so deltas attach to its
projections) that runs on rows of normed hidden states, a PagedKVCache and an AttnMeta.

A mixer reads its sizes and constants from a spec and keeps what it remembers under its own run
number of the cache: a layer that is run several times per token has one run per pass.  `kind` says
which pools ("kv", with `window`, None for all earlier tokens, and `shares`, the layer whose run it
reads instead of one of its own; or "state"), `cache_shape` their sizes per token or sequence.
`weight_views()` maps the mixer's checkpoint names (without the layer's prefix) to where they go."""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Dict, List, Optional, Tuple

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
    shares = None

    def __init__(self, spec: WindowAttentionSpec, width: int, bias_rows: int, eps: float, device, dtype):
        super().__init__()
        self.spec, self.eps, self.window = spec, eps, spec.window
        self.cache_shape = (spec.kv_heads, spec.dim, spec.vdim)
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
    normalised = True
    # portions up to this many tokens go through the recurrent kernel, longer ones 64 at a time
    RECURRENT_TOKENS = 4

    def __init__(self, spec: MlstmSpec, width: int, eps: float, device, dtype):
        super().__init__()
        self.spec, self.eps = spec, eps
        self.cache_shape = (spec.heads, spec.dim, spec.vdim)
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
# attention over a cached latent
# ---------------------------------------------------------------------------

@dataclass(frozen=True)
class LatentAttentionSpec:
    heads: int
    dim: int                            # query / key components per head without a rotation
    rot_dim: int                        # ... and with one; a key's are shared by all heads
    vdim: int
    kv_rank: int
    scale: float
    rot_base: float
    kv_from: Optional[int] = None       # layer whose latents this one reads instead of its own

    @classmethod
    def from_dict(cls, d: dict) -> "LatentAttentionSpec":
        spec = cls(int(d["heads"]), int(d["dim"]), int(d["rot_dim"]), int(d["vdim"]), int(d["kv_rank"]),
                   float(d["scale"]), float(d["rot"]["base"]), None if d.get("kv_from") is None else int(d["kv_from"]))
        if int(d["rot"]["dims"]) != spec.rot_dim or spec.rot_dim % 2:
            raise ValueError("the rotation covers the rot_dim components, in pairs")
        return spec


@dataclass
class _Rows:
    """Some sequences of a batch and their rows."""
    rows: Optional[torch.Tensor]        # row numbers, None: the slice [first, first + count)
    first: int
    count: int
    max_query: int
    q_starts: torch.Tensor
    ctx_lens: torch.Tensor
    block_tables: torch.Tensor
    kv_starts: Optional[torch.Tensor] = None
    total: int = 0                      # keys of all its sequences
    longest: int = 0

    def take(self, x: torch.Tensor) -> torch.Tensor:
        return x[self.first:self.first + self.count] if self.rows is None else x[self.rows]

    def put(self, out: torch.Tensor, part: torch.Tensor) -> None:
        if self.rows is None:
            out[self.first:self.first + self.count] = part
        else:
            out[self.rows] = part


class LatentAttention(nn.Module):
    """A token is cached as one row [latent | shared rotated key part].  Decoded tokens and short portions
    take the queries to the latent (q W_uk, attention over the rows as they lie, then W_uv); longer portions
    expand the rows of their sequences into keys and values of every head first."""
    kind = "kv"
    window = None
    # portions up to this many tokens work on the latents directly
    LATENT_TOKENS = 16
    # most bytes of expanded keys and values at a time (a single sequence may exceed it)
    EXPANDED_BYTES = 4 << 30

    def __init__(self, spec: LatentAttentionSpec, width: int, eps: float, device, dtype):
        super().__init__()
        self.spec, self.eps, self.shares = spec, eps, spec.kv_from
        self.row = spec.kv_rank + spec.rot_dim
        self.cache_shape = (1, self.row, 0)
        self.head = spec.dim + spec.rot_dim
        self.q_width = spec.heads * self.head
        own = self.shares is None
        self.q_latent_proj = _stacked(width, self.q_width + (self.row if own else 0), device, dtype)
        self.o_proj = L.RowParallelLinear(spec.heads * spec.vdim, width, device=device, dtype=dtype)
        mat = lambda rows: nn.Parameter(torch.empty((rows, spec.kv_rank), dtype=dtype, device=device).normal_(
            0, spec.kv_rank ** -0.5), requires_grad=False)
        self.uk, self.uv = mat(spec.heads * spec.dim), mat(spec.heads * spec.vdim)
        self.latent_norm = _vector(spec.kv_rank, device, 1.0) if own else None
        self.sink = _vector(spec.heads, device)
        self.expand = None

    def weight_views(self) -> Dict[str, torch.Tensor]:
        views = {"q": self.q_latent_proj.weight[: self.q_width], "uk": self.uk, "uv": self.uv, "sink": self.sink,
                 "o": self.o_proj.weight}
        if self.shares is None:
            views["dkv"] = self.q_latent_proj.weight[self.q_width:self.q_width + self.row]
            views["dkv.norm"] = self.latent_norm
        return views

    def prepare(self) -> None:
        """The expansion of a cached row to [keys of all heads | values of all heads] as one matrix: a head's
        key ends with the row's own shared part, which an identity block hands through unchanged."""
        s = self.spec
        w = torch.zeros((self.q_width + s.heads * s.vdim, self.row), dtype=self.uk.dtype, device=self.uk.device)
        keys = w[: self.q_width].view(s.heads, self.head, self.row)
        keys[:, : s.dim, : s.kv_rank] = self.uk.view(s.heads, s.dim, s.kv_rank)
        keys[:, s.dim:, s.kv_rank:] = torch.eye(s.rot_dim, dtype=w.dtype, device=w.device)
        w[self.q_width:, : s.kv_rank] = self.uv
        self.expand = w
        # 64-bit, so that a far position's angle is as good as a near one's
        i = torch.arange(s.rot_dim // 2, dtype=torch.float64)
        self.freq = (s.rot_base ** (-2.0 * i / s.rot_dim)).to(self.uk.device)

    # -- which rows go which way -----------------------------------------------------------
    def _split(self, meta: AttnMeta):
        """(rows for the latent form or None, [groups of rows for the expanded form])."""
        per_row = self.expand.shape[0] * self.expand.element_size()
        most = max(1, self.EXPANDED_BYTES // per_row)
        key = ("latent_attention", most, self.LATENT_TOKENS)
        if key not in meta.shared:
            meta.shared[key] = self._plan(meta, most)
        return meta.shared[key]

    def _plan(self, meta: AttnMeta, most: int):
        dev = meta.q_starts.device
        i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
        if meta.decode:
            n = meta.ctx_lens.shape[0]
            return _Rows(None, 0, n, 1, meta.q_starts, meta.ctx_lens, meta.block_tables), []
        counts, ctx = meta.prompt_lens, meta.host_ctx_lens
        starts = [0]
        for n in counts:
            starts.append(starts[-1] + n)

        def pick(seqs: List[int]) -> _Rows:
            lens, keys = [counts[i] for i in seqs], [ctx[i] + counts[i] for i in seqs]
            first, total = starts[seqs[0]], sum(lens)
            together = seqs == list(range(seqs[0], seqs[0] + len(seqs)))
            rows = None if together else torch.tensor([r for i in seqs for r in range(starts[i], starts[i + 1])], device=dev)
            edges = lambda v: i32([0] + torch.tensor(v).cumsum(0).tolist())
            whole = len(seqs) == len(counts)
            return _Rows(rows, first, total, max(lens), edges(lens), meta.ctx_lens if whole else i32([ctx[i] for i in seqs]),
                         meta.block_tables if whole else meta.block_tables[torch.tensor(seqs, device=dev)], edges(keys),
                         sum(keys), max(keys))

        short = [i for i, n in enumerate(counts) if 0 < n <= self.LATENT_TOKENS]
        groups: List[List[int]] = []
        held = 0
        for i, n in enumerate(counts):
            if n > self.LATENT_TOKENS:
                if not groups or held + ctx[i] + n > most:
                    groups.append([])
                    held = 0
                groups[-1].append(i)
                held += ctx[i] + n
        return (pick(short) if short else None), [pick(g) for g in groups]

    # -- forward ---------------------------------------------------------------------------
    def _latent_form(self, part: _Rows, x: torch.Tensor, q: torch.Tensor, rows: torch.Tensor, block_size: int,
                     out: torch.Tensor) -> None:
        """x: rows with the queries; q [rows, heads, row]: their rotated components are in place."""
        s = self.spec
        plain = x[:, : self.q_width].unflatten(1, (s.heads, self.head))[..., : s.dim]
        torch.bmm(plain.transpose(0, 1), self.uk.view(s.heads, s.dim, s.kv_rank), out=q[..., : s.kv_rank].transpose(0, 1))
        o = ops.latent_attention(q, rows, part.block_tables, part.q_starts, part.ctx_lens, s.kv_rank, block_size, s.scale,
                                 self.sink)
        torch.bmm(o.transpose(0, 1), self.uv.view(s.heads, s.vdim, s.kv_rank).transpose(1, 2),
                  out=out.view(-1, s.heads, s.vdim).transpose(0, 1))

    def forward(self, h: torch.Tensor, cache: PagedKVCache, run: int, meta: AttnMeta) -> torch.Tensor:
        s, rows, m = self.spec, cache.k[run], h.shape[0]
        x = self.q_latent_proj(h)[0]
        latent, groups = self._split(meta)
        own = dict(l_off=self.q_width, norm_weight=self.latent_norm, eps=self.eps, cache=rows,
                   slot_mapping=meta.slot_mapping) if self.shares is None else {}
        q = x.new_empty((m, s.heads, self.row)) if not groups else None
        ops.latent_rows(x, meta.positions, self.freq, s.heads, s.dim, s.rot_dim, s.kv_rank, q_out=q, **own)
        att = x.new_empty((m, s.heads * s.vdim))
        if latent is not None:
            if q is not None:
                self._latent_form(latent, x, q, rows, cache.block_size, att)
            else:
                part = latent.take(x)
                q, o = x.new_empty((part.shape[0], s.heads, self.row)), x.new_empty((part.shape[0], att.shape[1]))
                q[..., s.kv_rank:] = part[:, : self.q_width].unflatten(1, (s.heads, self.head))[..., s.dim:]
                self._latent_form(latent, part, q, rows, cache.block_size, o)
                latent.put(att, o)
        for g in groups:
            kv = ops.latent_gather(rows, g.block_tables, cache.block_size, g.kv_starts, g.total, g.longest)
            kv = ops.base_gemm(kv, self.expand)
            o = ops.rows_attention(g.take(x), kv, g.q_starts, g.ctx_lens, g.kv_starts, g.max_query, s.heads, s.heads,
                                   self.head, s.vdim, s.scale, self.sink)
            if g.count == m:
                att = o
            else:
                g.put(att, o)
        return self.o_proj(att)[0]


# ---------------------------------------------------------------------------
# linear attention with a constant decay
# ---------------------------------------------------------------------------

@dataclass(frozen=True)
class LightningSpec:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]

    @classmethod
    def from_dict(cls, d: dict) -> "LightningSpec":
        decay = d["decay"] if isinstance(d["decay"], (list, tuple)) else [d["decay"]] * int(d["heads"])
        spec = cls(int(d["heads"]), int(d["dim"]), int(d["vdim"]), tuple(float(x) for x in decay))
        if len(spec.decay) != spec.heads:
            raise ValueError("one decay per head")
        return spec


class Lightning(nn.Module):
    kind = "state"
    normalised = False
    # portions up to this many tokens go through the recurrent kernel, longer ones 64 at a time
    RECURRENT_TOKENS = 4

    def __init__(self, spec: LightningSpec, width: int, eps: float, device, dtype):
        super().__init__()
        self.spec, self.eps = spec, eps
        self.cache_shape = (spec.heads, spec.dim, spec.vdim)
        self.qk, self.vw = spec.heads * spec.dim, spec.heads * spec.vdim
        self.qkvg_proj = _stacked(width, 2 * self.qk + 2 * self.vw, device, dtype)
        self.o_proj = L.RowParallelLinear(self.vw, width, device=device, dtype=dtype)
        self.norm = _vector(self.vw, device, 1.0)
        n = torch.arange(ops.LIGHTNING_POWERS, dtype=torch.float64)
        self.powers = (torch.tensor(spec.decay, dtype=torch.float64)[:, None] ** n).float().to(device)
        self.chunkwise = ops.lightning_chunk_supported(spec.dim, spec.vdim, dtype)

    def weight_views(self) -> Dict[str, torch.Tensor]:
        q, k, v, g = self.qkvg_proj.weight[: 2 * self.qk + 2 * self.vw].split([self.qk, self.qk, self.vw, self.vw])
        return {"q": q, "k": k, "v": v, "g": g, "o": self.o_proj.weight, "norm": self.norm}

    def prepare(self) -> None:
        pass

    def forward(self, h: torch.Tensor, cache: PagedKVCache, run: int, meta: AttnMeta) -> torch.Tensor:
        st = cache.state
        x = self.qkvg_proj(h)[0]
        o = ops.lightning(x, self.powers, self.norm, st.S[run], meta.state_slots, meta.q_starts, meta.ctx_lens, self.eps,
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


@dataclass(frozen=True)
class RoutedExpertsSpec:
    experts: int
    top: int
    ff: int
    shared_ff: Optional[int] = None     # width of an expert that every token passes, None: there is none

    @classmethod
    def from_dict(cls, d: dict) -> "RoutedExpertsSpec":
        r, shared = d["router"], d.get("shared")
        spec = cls(int(r["experts"]), int(r["top"]), int(d["expert"]["ff"]), int(shared["ff"]) if shared else None)
        if not 1 <= spec.top <= spec.experts:
            raise ValueError("a token takes between one and all of the experts")
        return spec


class RoutedExperts(nn.Module):
    """Each token through its `top` experts down(act(up(s h))), s = sigmoid of the router's logit -- the score
    scales the expert's input, which the up product's epilogue does to its result -- and, where there is
    one, through a shared expert with scale 1.  Returns the shared expert's output and the routed rows,
    which the next residual step sums."""

    def __init__(self, spec: RoutedExpertsSpec, width: int, activation: str, device, dtype):
        super().__init__()
        self.spec, self.activation = spec, activation
        mat = lambda *shape: nn.Parameter(torch.empty(shape, dtype=dtype, device=device).normal_(0, 0.02),
                                          requires_grad=False)
        self.router = mat(spec.experts, width)
        self.up, self.down = mat(spec.experts, spec.ff, width), mat(spec.experts, width, spec.ff)
        self.up_proj = self.down_proj = None
        if spec.shared_ff is not None:
            self.up_proj = _stacked(width, spec.shared_ff, device, dtype)
            self.down_proj = L.RowParallelLinear(spec.shared_ff, width, device=device, dtype=dtype)

    def weight_views(self) -> Dict[str, torch.Tensor]:
        views = {"router": self.router}
        for e in range(self.spec.experts):
            views[f"e{e}.up"], views[f"e{e}.down"] = self.up[e], self.down[e]
        if self.up_proj is not None:
            views["shared.up"], views["shared.down"] = self.up_proj.weight[: self.spec.shared_ff], self.down_proj.weight
        return views

    def forward(self, h: torch.Tensor) -> ops.Update:
        routing = ops.moe_route(ops.matmul_f32(h, self.router), self.spec.top)
        a = ops.moe_gemm(ops.moe_gather(h, routing), self.up, routing.offsets, routing.sorted_scores, self.activation)
        y = ops.moe_gemm(a, self.down, routing.offsets)
        shared = None
        if self.up_proj is not None:
            shared = self.down_proj(ops.act(self.up_proj(h)[0], self.activation, self.spec.shared_ff))[0]
        return ops.Update(shared, y, routing.place)
