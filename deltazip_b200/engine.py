"""A small decode engine over the delta layers: sequences, the paged KV cache, delta-aware
admission and the per-step device state.  It stands where the reference's scheduler and model
runner stand around the SBMM path (serving/vllm/core/scheduler.py:359-366,528-535: a batch may
hold at most `max_deltas` distinct deltas and is sorted by delta id, :101-104;
serving/vllm/worker/model_runner.py:919-975: set the active deltas and the mapping, run the
model, sample) -- reduced to greedy sampling and to what the throughput configurations need.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Dict, List, Optional, Tuple

import torch

from . import registry
from .cache import AttnMeta
from .config import DeltaConfig
from .layers import DeltaMapping
from .models import LRUCacheDeltaModelManager


@dataclass
class Sequence:
    seq_id: int
    delta_id: int                       # 0 = base model
    length: int                         # tokens in the cache so far
    max_new: int
    blocks: List[int] = field(default_factory=list)
    state_slot: int = -1                # recurrent models: slot of this sequence's state
    generated: int = 0
    arrival: float = 0.0
    prompt: Optional[torch.Tensor] = None
    first_token_time: Optional[float] = None


class DecodeEngine:
    """Model + slot manager + sequence cache for one tensor-parallel rank.

    The model is built at random from `cfg` or handed in (`model=`, for a loaded checkpoint).
    Without `delta_config` the base model is served alone.  `max_prefill_tokens` bounds the rows of
    one forward pass for models that can continue a prompt from the cache."""

    def __init__(self, cfg, delta_config: Optional[DeltaConfig], max_seqs: int, kv_blocks: int,
                 block_size: int = 16, device="cuda", dtype=None, seed: int = 0, model=None,
                 max_prefill_tokens: int = 8192):
        self.cfg, self.device, self.block_size = cfg, torch.device(device), block_size
        self.model = model if model is not None else registry.build_model(cfg, device=device, seed=seed, dtype=dtype)
        self.manager = None
        if delta_config is not None:
            if self.model.dtype == torch.float32:
                raise ValueError("deltas are applied to 16-bit activations")
            self.manager = LRUCacheDeltaModelManager(self.model, max_seqs,
                                                     max(max_seqs, 2048, max_prefill_tokens
                                                         if self.model.supports_portions else 0),
                                                     cfg.vocab_size, delta_config, device=device)
        self.cache = self.model.make_cache(kv_blocks, block_size, max_seqs)
        self.max_prefill_tokens = max_prefill_tokens
        self.max_seqs = max_seqs
        self.running: List[Sequence] = []
        self._dirty = True
        self._order: List[int] = []
        self.tokens = None
        self.positions = None
        self.block_tables = None
        self.attn_splits = 0            # 0: chosen per step from the batch (see decode_step)
        self.swap_ins = 0

    # -- batch composition -----------------------------------------------------------
    def admit(self, waiting: List[Sequence]) -> List[Sequence]:
        """Delta-aware admission: sequences join while a batch slot, KV blocks for their whole
        life and a GPU slot for their delta are available.  A delta that is not resident takes a
        free slot or evicts the least recently used delta no running sequence needs.  Returns
        the sequences admitted (their deltas are resident and activated)."""
        admitted = []
        mgr = self.manager
        in_use = {s.delta_id for s in self.running if s.delta_id > 0}
        for seq in list(waiting):
            if len(self.running) + len(admitted) >= self.max_seqs:
                break
            tokens = seq.length + seq.max_new
            if not self.cache.can_open(tokens):
                continue
            d = seq.delta_id
            if d > 0 and mgr is None:
                continue                                        # no deltas are served here
            if d > 0 and d not in mgr._active_deltas:
                if mgr.get_delta(d) is None:
                    continue                                    # unknown delta: not servable
                if len(mgr._active_deltas) + len(mgr._loading) >= mgr.delta_slots and d not in mgr._loading:
                    victim = next((x for x in mgr._active_deltas if x not in in_use), None)
                    if victim is None:
                        continue                                # every slot is needed by the batch
                    mgr.deactivate_delta(victim)
                mgr.activate_delta(d)
            elif d > 0:
                mgr._active_deltas.move_to_end(d)
            in_use.add(d)
            self.cache.open(seq, tokens)
            admitted.append(seq)
            waiting.remove(seq)
        if admitted:
            self.running.extend(admitted)
            self._dirty = True
        return admitted

    def admit_overlapped(self, waiting: List[Sequence], ready=None) -> List[Sequence]:
        """Admission that never makes the compute stream wait for a swap-in: a sequence whose
        delta is not resident triggers a prefetch into a free (or evictable) GPU slot -- the
        upload runs on the copy stream while the batch keeps decoding -- and joins in a later
        round, once the upload's event has completed.  `ready(delta_id) -> bool` reports that
        (default: the event's own query; a tensor-parallel caller passes the agreement of all
        ranks so that every rank admits the same sequences)."""
        mgr = self.manager
        if ready is None:
            def ready(d):
                return mgr._slot_ready[mgr._loading[d]].query()
        admitted = []
        in_use = {s.delta_id for s in self.running if s.delta_id > 0}
        wanted = set()
        for seq in list(waiting):
            if len(self.running) + len(admitted) >= self.max_seqs:
                break
            tokens = seq.length + seq.max_new
            if not self.cache.can_open(tokens):
                continue
            d = seq.delta_id
            if d > 0 and mgr is None:
                continue                                        # no deltas are served here
            if d > 0 and d not in mgr._active_deltas:
                if mgr.get_delta(d) is None:
                    continue
                if d in mgr._loading:
                    if not ready(d):
                        continue
                    mgr.activate_delta(d)              # upload finished: no stall
                else:
                    if d in wanted:
                        continue
                    if len(mgr._active_deltas) + len(mgr._loading) >= mgr.delta_slots:
                        victim = next((x for x in mgr._active_deltas if x not in in_use), None)
                        if victim is None:
                            continue
                        mgr.deactivate_delta(victim)
                    mgr.prefetch_delta(d)
                    self.swap_ins += 1
                    wanted.add(d)
                    continue
            elif d > 0:
                mgr._active_deltas.move_to_end(d)
            in_use.add(d)
            self.cache.open(seq, tokens)
            admitted.append(seq)
            waiting.remove(seq)
        if admitted:
            self.running.extend(admitted)
            self._dirty = True
        return admitted

    def retire(self, seq: Sequence) -> None:
        self.cache.close(seq)
        self.running.remove(seq)
        self._dirty = True

    def _slot_of(self, delta_id: int) -> int:
        return self.manager.delta_index_to_id.index(delta_id) if delta_id > 0 else -1

    def _sort_key(self, seq: Sequence):
        return (self._slot_of(seq.delta_id), seq.seq_id)

    def _set_mapping(self, seqs: List[Sequence], counts: List[int]) -> None:
        if self.manager is not None:
            ids = [s.delta_id for s, n in zip(seqs, counts) for _ in range(n)]
            self.manager.set_delta_mapping(DeltaMapping(ids, [s.delta_id for s in seqs]))

    def _block_tables(self, seqs: List[Sequence]) -> torch.Tensor:
        width = max([len(s.blocks) for s in seqs] + [1])
        tab = torch.zeros((max(len(seqs), 1), width), dtype=torch.int32)
        for i, s in enumerate(seqs):
            tab[i, : len(s.blocks)] = torch.tensor(s.blocks, dtype=torch.int32)
        return tab.to(self.device)

    def _int32(self, values) -> torch.Tensor:
        return torch.tensor(values, dtype=torch.int32, device=self.device)

    def _state_slots(self, seqs: List[Sequence]) -> Optional[torch.Tensor]:
        return self._int32([s.state_slot for s in seqs]) if self.cache.state is not None else None

    def _rebuild(self, tokens: Optional[Dict[int, int]] = None) -> None:
        """Device-side state of the running batch, sequences ordered by GPU slot so that the
        token rows reach the SBMM sorted.  `tokens`: seq_id -> next input token."""
        old = {}
        if self.tokens is not None and self._order:
            host = self.tokens.tolist()
            old = {sid: host[i] for i, sid in enumerate(self._order)}
        if tokens:
            old.update(tokens)
        self.running.sort(key=self._sort_key)
        self._order = [s.seq_id for s in self.running]
        dev = self.device
        self.block_tables = self._block_tables(self.running)
        self.positions = torch.tensor([s.length for s in self.running], dtype=torch.int64, device=dev)
        self.tokens = torch.tensor([old.get(s.seq_id, 0) for s in self.running], dtype=torch.int64,
                                   device=dev)
        self.state_slots = self._state_slots(self.running)
        self.q_starts = torch.arange(len(self.running) + 1, dtype=torch.int32, device=dev)
        self._set_mapping(self.running, [1] * len(self.running))
        self._dirty = False

    # -- one decode step ---------------------------------------------------------------
    @torch.inference_mode()
    def decode_step(self) -> torch.Tensor:
        """Feeds every running sequence its latest token (position = its cached length), appends
        the new key/value to the cache and samples the next token greedily.  Device work only
        unless the batch composition changed since the last step."""
        if self._dirty:
            self._rebuild()
        bs = self.block_size
        pos = self.positions
        # the modulus only matters for windowed models, whose sequences use their blocks as a ring
        blk = torch.gather(self.block_tables, 1, (pos // bs % self.block_tables.shape[1]).unsqueeze(1))
        slot = blk.squeeze(1).to(torch.int64) * bs + pos % bs
        lens = (pos + 1).to(torch.int32)
        # one CTA per (sequence, kv head, split): split the keys when the batch alone would leave
        # most SMs without a CTA
        splits = self.attn_splits or max(1, min(8, 296 // max(1, len(self.running) * self.model.kv_heads)))
        h = self.model(self.tokens, pos, self.cache,
                       AttnMeta(slot_mapping=slot, block_tables=self.block_tables, seq_lens=lens,
                                splits=splits, q_starts=self.q_starts, ctx_lens=pos.to(torch.int32),
                                state_slots=self.state_slots))
        self.tokens = self.model.greedy_tokens(h)
        self.positions = pos + 1
        for s in self.running:
            s.length += 1
            s.generated += 1
        return self.tokens

    # -- given tokens --------------------------------------------------------------------
    def _forward_rows(self, work: List[Tuple[Sequence, List[int]]]) -> torch.Tensor:
        """One forward pass over the next tokens of some sequences; returns their hidden states, rows
        in the order of `work` (which is sorted by GPU slot)."""
        seqs, counts = [s for s, _ in work], [len(t) for _, t in work]
        dev = self.device
        decode = all(n == 1 for n in counts) and (self.model.supports_portions or all(s.length for s in seqs))
        if not decode and not self.model.supports_portions and any(s.length for s in seqs):
            raise ValueError("this model cannot continue a prompt from its cache")
        starts = [0]
        for n in counts:
            starts.append(starts[-1] + n)
        meta = AttnMeta(
            slot_mapping=torch.tensor([x for s, n in zip(seqs, counts)
                                       for x in self.cache.slots(s.blocks, s.length, n)],
                                      dtype=torch.int64, device=dev),
            block_tables=self._block_tables(seqs),
            seq_lens=self._int32([s.length + n for s, n in zip(seqs, counts)]),
            prompt_lens=None if decode else counts,
            q_starts=self._int32(starts), ctx_lens=self._int32([s.length for s in seqs]),
            state_slots=self._state_slots(seqs), host_ctx_lens=[s.length for s in seqs])
        toks = torch.tensor([t for _, ts in work for t in ts], dtype=torch.int64).to(dev)
        pos = torch.tensor([s.length + i for s, n in zip(seqs, counts) for i in range(n)], dtype=torch.int64).to(dev)
        self._set_mapping(seqs, counts)
        self._dirty = True                      # the mapping and the lengths are no longer those of a decode step
        h = self.model(toks, pos, self.cache, meta)
        for s, n in zip(seqs, counts):
            s.length += n
        return h

    @torch.inference_mode()
    def extend(self, work: List[Tuple[Sequence, List[int]]]) -> torch.Tensor:
        """Runs the given next tokens of admitted sequences (new prompts, portions of prompts, single
        tokens, in any mixture) from the cache and state that earlier calls left; a sequence that was
        admitted for fewer tokens takes further cache blocks.  Returns the hidden states of all the
        tokens, in the order of `work`.  Models that support it take long work in passes of at most
        `max_prefill_tokens` rows."""
        for s, toks in work:
            self.cache.reserve(s, s.length + len(toks))
        order = sorted(range(len(work)), key=lambda i: self._sort_key(work[i][0]))
        limit = self.max_prefill_tokens if self.model.supports_portions else None
        parts: List[List[torch.Tensor]] = [[] for _ in work]
        done = [0] * len(work)
        while True:
            room, batch = limit, []
            for i in order:
                left = len(work[i][1]) - done[i]
                n = left if room is None else min(left, room)
                if n > 0:
                    batch.append((i, n))
                    room = None if room is None else room - n
            if not batch:
                break
            h = self._forward_rows([(work[i][0], list(work[i][1][done[i]:done[i] + n])) for i, n in batch])
            row = 0
            for i, n in batch:
                parts[i].append(h[row:row + n])
                done[i] += n
                row += n
        rows = [p for ps in parts for p in ps]
        return torch.cat(rows) if rows else torch.empty((0, 0), device=self.device)

    @torch.inference_mode()
    def prefill(self, seqs: List[Sequence]) -> None:
        """Runs the prompts of newly admitted sequences (all tokens of all prompts in one pass where
        they fit, rows sorted by GPU slot), fills their cache blocks and leaves their first generated
        token as the next decode input."""
        if not seqs:
            return
        seqs = sorted(seqs, key=self._sort_key)
        for s in seqs:
            s.length = 0
        h = self.extend([(s, s.prompt.tolist()) for s in seqs])
        last = torch.tensor([int(s.prompt.numel()) for s in seqs], device=self.device).cumsum(0) - 1
        nxt = self.model.greedy_tokens(h[last]).tolist()
        first = {s.seq_id: nxt[i] for i, s in enumerate(seqs)}
        for s in seqs:
            s.generated = 1
        self._rebuild(first)

    # -- whole requests ------------------------------------------------------------------
    def generate(self, prompts: List[List[int]], max_new: int, delta_ids: Optional[List[int]] = None,
                 stop_id: Optional[int] = None) -> List[List[int]]:
        """Greedy generation for a list of prompts through admission, prefill and decode steps: sequences
        join as batch slots, cache and deltas allow and leave when they have `max_new` tokens or
        produced `stop_id`."""
        if self.running:
            raise RuntimeError("sequences are already running")
        if max_new < 1 or any(not p for p in prompts):
            raise ValueError("prompts hold at least a token, and at least one token is generated")
        waiting = [Sequence(i, delta_ids[i] if delta_ids else 0, len(p), max_new,
                            prompt=torch.tensor(p, dtype=torch.int64)) for i, p in enumerate(prompts)]
        out: List[List[int]] = [[] for _ in prompts]

        def take(tokens: List[int], order: List[int], fresh) -> None:
            for sid, tok in zip(order, tokens):
                if sid in fresh:
                    out[sid].append(tok)
            for s in list(self.running):
                if s.seq_id in fresh and (s.generated >= max_new or out[s.seq_id][-1] == stop_id):
                    self.retire(s)

        while waiting or self.running:
            admitted = self.admit(waiting)
            if admitted:
                self.prefill(admitted)
                take(self.tokens.tolist(), self._order, {s.seq_id for s in admitted})
            elif not self.running:
                raise RuntimeError("a waiting request fits neither the cache nor the resident deltas")
            if self.running:
                toks = self.decode_step().tolist()
                take(toks, self._order, set(self._order))
        return out
