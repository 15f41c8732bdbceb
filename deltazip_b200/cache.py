"""What a sequence leaves behind between steps: paged key/value pools and recurrent state slots,
and the description of a batch that the model's mixers read them through (role of the reference's
block manager + cache engine, serving/vllm/core/block_manager.py,
serving/vllm/worker/cache_engine.py, reduced to what a single process needs)."""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import List, Optional, Sequence, Tuple

import torch


class RecurrentStateCache:
    """Per recurrent layer run the 32-bit pools S [slots, heads, dim, vdim] and, where the run normalises
    (`normalised`, default: all do), n [slots, heads, dim] and m [slots, heads]; a sequence owns one
    slot number, the same in every pool.  Slots are handed out as they are: a sequence without context
    starts from zero without reading its slot."""

    def __init__(self, shapes: Sequence[Tuple[int, int, int]], slots: int, device="cuda",
                 normalised: Optional[Sequence[bool]] = None):
        f32 = dict(dtype=torch.float32, device=device)
        with_n = [True] * len(shapes) if normalised is None else list(normalised)
        self.S = [torch.zeros((slots, h, d, v), **f32) for h, d, v in shapes]
        self.n = [torch.zeros((slots, h, d), **f32) if w else None for (h, d, _), w in zip(shapes, with_n)]
        self.m = [torch.zeros((slots, h), **f32) if w else None for (h, _, _), w in zip(shapes, with_n)]
        self.free: List[int] = list(range(slots - 1, -1, -1))

    def allocate(self) -> int:
        if not self.free:
            raise RuntimeError("out of recurrent state slots")
        return self.free.pop()

    def release(self, slot: int) -> None:
        self.free.append(slot)


class PagedKVCache:
    """Per-layer K and V pools of `num_blocks` blocks of `block_size` tokens, [slots, kv_heads,
    head size] each, with a free list.  `layer_shapes` gives (kv_heads, key size, value size) per
    layer run where layers differ (default: `num_layers` times (kv_heads, 128, 128)); a run that caches
    one row per token for all heads has one key head and value size 0.

    `window`: the largest number of tokens any layer looks back (itself included).  A sequence then
    owns at most ceil(window / block_size) blocks and uses them as a ring: token position t lives in
    block number (t / block_size) modulo the blocks it owns.  `state` holds the recurrent layers'
    slots, where the model has any."""

    def __init__(self, num_layers: int, num_blocks: int, kv_heads: int, block_size: int = 16,
                 dtype=torch.float16, device="cuda",
                 layer_shapes: Optional[Sequence[Tuple[int, int, int]]] = None,
                 window: Optional[int] = None, state: Optional[RecurrentStateCache] = None):
        self.block_size, self.num_blocks, self.kv_heads = block_size, num_blocks, kv_heads
        shapes = [(kv_heads, 128, 128)] * num_layers if layer_shapes is None else list(layer_shapes)
        rows = num_blocks * block_size
        self.k = [torch.empty((rows, h, dk), dtype=dtype, device=device) for h, dk, _ in shapes]
        self.v = [torch.empty((rows, h, dv), dtype=dtype, device=device) for h, _, dv in shapes]
        self.window = window
        self.state = state
        self.free: List[int] = list(range(num_blocks - 1, -1, -1))

    def blocks_for(self, tokens: int) -> int:
        """Blocks a sequence of `tokens` tokens holds at most."""
        if self.window is not None:
            tokens = min(tokens, self.window)
        return (tokens + self.block_size - 1) // self.block_size

    def allocate(self, n_blocks: int) -> List[int]:
        if n_blocks > len(self.free):
            raise RuntimeError("out of KV cache blocks")
        return [self.free.pop() for _ in range(n_blocks)]

    def release(self, blocks: Sequence[int]) -> None:
        self.free.extend(blocks)

    def slots(self, blocks: Sequence[int], start: int, count: int) -> List[int]:
        """Cache slots of token positions [start, start + count) of a sequence owning `blocks`.  Where
        the ring comes round inside the range only its last tokens get a slot (-1: not kept)."""
        bs = self.block_size
        if self.window is None:
            return [blocks[p // bs] * bs + p % bs for p in range(start, start + count)]
        n = len(blocks)
        keep = start + count - n * bs
        return [blocks[p // bs % n] * bs + p % bs if p >= keep else -1 for p in range(start, start + count)]

    # -- whole sequences ---------------------------------------------------------------
    def can_open(self, tokens: int) -> bool:
        return self.blocks_for(tokens) <= len(self.free) and (self.state is None or bool(self.state.free))

    def open(self, seq, tokens: int) -> None:
        """Gives `seq` (an object with `blocks` and `state_slot`) what it needs for `tokens` tokens."""
        seq.blocks = self.allocate(self.blocks_for(tokens))
        if self.state is not None:
            seq.state_slot = self.state.allocate()

    def reserve(self, seq, tokens: int) -> None:
        """Gives an open `seq` the blocks it still lacks for `tokens` tokens.  (A ring has all it will ever
        have: its positions are counted modulo its blocks.)"""
        if self.window is None and len(seq.blocks) < self.blocks_for(tokens):
            seq.blocks = seq.blocks + self.allocate(self.blocks_for(tokens) - len(seq.blocks))

    def close(self, seq) -> None:
        self.release(seq.blocks)
        seq.blocks = []
        if self.state is not None and seq.state_slot >= 0:
            self.state.release(seq.state_slot)
            seq.state_slot = -1


@dataclass
class AttnMeta:
    """How the sequence mixers run in one forward pass; rows are in (sequence, position) order.

    Decode (`prompt_lens` is None): one row per sequence; `block_tables` [B, max_blocks] int32 and
    `seq_lens` [B] int32 (cached length including the current token).
    Prompt portions: `prompt_lens`, the row count of each sequence.

    Models that continue prompts from a cache also read `q_starts` [B + 1] int32 (first row of every
    sequence), `ctx_lens` [B] int32 (tokens before the first row; `host_ctx_lens` the same as numbers, for
    prompt portions) and, with recurrent layers, `state_slots` [B] int32.  `shared` keeps what the layers
    of one pass derive from all this."""
    slot_mapping: Optional[torch.Tensor] = None          # int64 [M] cache slot per token, -1 = none
    block_tables: Optional[torch.Tensor] = None
    seq_lens: Optional[torch.Tensor] = None
    prompt_lens: Optional[List[int]] = None
    splits: int = 1
    q_starts: Optional[torch.Tensor] = None
    ctx_lens: Optional[torch.Tensor] = None
    state_slots: Optional[torch.Tensor] = None
    host_ctx_lens: Optional[List[int]] = None
    positions: Optional[torch.Tensor] = None             # int64 [M], set by models whose mixers read them
    shared: dict = field(default_factory=dict)

    @property
    def decode(self) -> bool:
        return self.prompt_lens is None

    @property
    def max_query(self) -> int:
        return 1 if self.prompt_lens is None else max(self.prompt_lens)
