"""Host-side parts of the Buzalorn model without a GPU: configuration, registry, distance buckets, the
ring cache and state slots, the loader, and the oracle's own consistency (a second way to compute
each recurrence, so that a slip in the oracle does not go unnoticed)."""
import numpy as np
import pytest
import torch

from deltazip_b200 import registry
from deltazip_b200.cache import PagedKVCache, RecurrentStateCache
from deltazip_b200.engine import DecodeEngine, Sequence
from deltazip_b200.loader import copy_weights, read_config, read_tensors
from deltazip_b200.mixers import bucket_edges, distance_bias
from oracle import buzalorn_oracle as O
from tests import buzalorn_util as U


def test_config_registry_and_layer_runs():
    config = U.make_config()
    entry = registry.lookup(config)
    cfg = entry.config_class.from_dict(config)
    assert entry.name == "Buzalorn" and registry.entry_for(cfg) is entry
    assert [i for i, _ in cfg.runs()] == [0, 1, 2, 1, 2, 1, 2, 3]
    assert [p for _, p in cfg.runs()] == [None, 0, None, 1, None, 2, None, None]
    assert [i for i, _ in cfg.runs()] == [i for i, _ in O.layer_runs(config)]
    assert cfg.layers[2].ff is None and cfg.layers[3].ff == 80
    assert registry.lookup({"architectures": ["LlamaForCausalLM"]}).name == "LlamaForCausalLM"
    with pytest.raises(ValueError, match="no model"):
        registry.lookup({"architecture": "Nonesuch"})
    for broken in ({"type": "conv"}, {"mlp": {"kind": "sparse", "ff": 8}}):
        bad = U.make_config()
        bad["layers"][0].update(broken)
        with pytest.raises(ValueError):
            entry.config_class.from_dict(bad)
    with pytest.raises(ValueError):
        entry.config_class.from_dict(U.make_config(loop=(2, 5, 2)))


@pytest.mark.parametrize("rows,bias_max", [(12, 50), (32, 100), (4, 1000), (2, 9), (8, 64), (10, 7)])
def test_distance_buckets(rows, bias_max):
    edges = bucket_edges(rows, bias_max)
    assert edges[: rows // 2 + 1] == list(range(rows // 2 + 1)) and len(edges) == rows
    rel = torch.arange(rows, dtype=torch.float32)[:, None] * torch.tensor([1.0, -1.0])
    for window in (3, rows, bias_max // 2 + 1, 3 * bias_max):
        table = distance_bias(rel, bias_max, window)
        for n in range(window):
            want = O.distance_bucket(n, rows, bias_max)
            assert table[0, min(n, table.shape[1] - 1)] == want and table[1, min(n, table.shape[1] - 1)] == -want


def test_bucket_edges_are_exact_at_powers():
    # the last bucket starts where the logarithm reaches it, also where that falls on an integer
    assert bucket_edges(8, 64)[4:] == [4, 8, 16, 32]
    assert bucket_edges(6, 81)[3:] == [3, 9, 27]


def test_ring_cache_slots():
    c = PagedKVCache(0, 10, 1, 4, torch.float32, "cpu", layer_shapes=[(1, 2, 3)], window=10)
    assert c.k[0].shape == (40, 1, 2) and c.v[0].shape == (40, 1, 3)
    assert [c.blocks_for(n) for n in (1, 4, 5, 10, 11, 1000)] == [1, 1, 2, 3, 3, 3]
    blocks = [7, 2, 5]
    assert c.slots(blocks, 0, 5) == [28, 29, 30, 31, 8]
    assert c.slots(blocks, 11, 3) == [23, 28, 29]                      # the ring comes round at 12
    assert c.slots(blocks, 0, 14) == [-1, -1] + c.slots(blocks, 2, 12)  # only a ring's worth is kept
    live = {}
    for p in range(50):                                                # every window is intact at any time
        live[c.slots(blocks, p, 1)[0]] = p
        assert set(range(max(0, p - 9), p + 1)) <= set(live.values())


def test_admission_opens_and_returns_blocks_and_state_slots():
    eng = DecodeEngine.__new__(DecodeEngine)
    eng.block_size, eng.max_seqs, eng.manager = 4, 8, None
    state = RecurrentStateCache([(2, 3, 5)], 2, "cpu")
    assert state.S[0].shape == (2, 2, 3, 5) and state.n[0].shape == (2, 2, 3) and state.m[0].shape == (2, 2)
    eng.cache = PagedKVCache(0, 7, 1, 4, torch.float32, "cpu", layer_shapes=[], window=12, state=state)
    eng.running, eng._dirty = [], False
    waiting = [Sequence(i, 0, 100, 20) for i in range(3)]
    got = eng.admit(waiting)
    assert [s.seq_id for s in got] == [0, 1] and len(waiting) == 1        # no third state slot
    assert sorted(s.state_slot for s in got) == [0, 1] and all(len(s.blocks) == 3 for s in got)
    slot, blocks = got[0].state_slot, list(got[0].blocks)
    eng.retire(got[0])
    assert got[0].state_slot == -1 and got[0].blocks == []
    again = eng.admit(waiting)
    assert again[0].state_slot == slot and sorted(again[0].blocks) == sorted(blocks)
    assert eng.admit([Sequence(9, 4, 1, 1)]) == []                        # a delta cannot be served here


def test_checkpoint_reader_and_weight_copy(tmp_path):
    config = U.make_config()
    tensors = U.make_tensors(config)
    U.write_checkpoint(str(tmp_path), config, tensors)
    assert read_config(str(tmp_path)) == config
    back = read_tensors(str(tmp_path))
    assert set(back) == set(tensors) and all(torch.equal(back[k], tensors[k]) for k in back)
    dst = torch.zeros(3, 2)
    copy_weights({"a": [dst[:2], dst[1:]]}, {"a": torch.ones(2, 2)})
    assert dst.sum() == 6
    for tensors in ({}, {"a": torch.ones(2, 3)}, {"a": torch.ones(2, 2), "b": torch.ones(1)}):
        with pytest.raises(ValueError):
            copy_weights({"a": [dst[:2]]}, tensors)


# -- the oracle against itself -------------------------------------------------------------------

def test_oracle_recurrence_against_its_unstabilised_sum():
    """o = sum_s w_ts (q.k_s) v_s over the denominator, with w_ts = exp(i_s + sum_{s < r <= t} f_r)."""
    rng = np.random.default_rng(0)
    t, dim, vdim = 9, 4, 3
    q, k, v = rng.normal(size=(t, dim)), rng.normal(size=(t, dim)), rng.normal(size=(t, vdim))
    i, f = rng.normal(size=t) * 3, O.log_sigmoid(rng.normal(size=t))
    got = O.mlstm_recurrence(q, k, v, i, f)
    m = 0.0
    for a in range(t):
        m = max(m + f[a], i[a])
        w = np.array([np.exp(i[s] + f[s + 1:a + 1].sum()) for s in range(a + 1)])
        s = w * (k[:a + 1] @ q[a])
        den = max(abs(s.sum()), 1.0) + 1e-6 * np.exp(m)
        assert np.allclose(got[a], s @ v[:a + 1] / den, rtol=1e-9)


def test_oracle_attention_window_and_far_key():
    """A key that dominates every score is returned inside the window and invisible one step outside."""
    t, window = 40, 7
    q = np.ones((t, 1, 2)) * 10
    k = np.zeros((t, 1, 2))
    k[5] = 10
    v = np.arange(t, dtype=float).reshape(t, 1, 1)
    out = O.attention_core(q, k, v, 1.0, window)[:, 0, 0]
    assert np.allclose(out[5:5 + window], 5) and abs(out[5 + window] - 5) > 1
    rel = np.zeros((4, 1))
    rel[3] = 50.0                                        # the last bucket: distances from its edge on
    edge = bucket_edges(4, 9)[3]
    out = O.attention_core(q * 0, k, v, 1.0, 30, rel, 9)[:, 0, 0]
    assert np.allclose(out[edge], 0) and not np.allclose(out[edge - 1], 0)


def test_oracle_forward_is_causal():
    config = U.make_config()
    tensors = U.make_tensors(config)
    toks = [3, 7, 100, 7, 55]
    a, b = U.oracle_logits(config, tensors, toks), U.oracle_logits(config, tensors, toks[:3])
    assert np.allclose(a[:3], b)
