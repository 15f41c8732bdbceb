"""Host-side parts of the Movarax model without a GPU: configuration, registry, cache runs, which rows of
a batch go which way, and the oracle's own consistency (a second way to compute what it computes, so that
a slip in it does not go unnoticed)."""
import copy

import numpy as np
import pytest
import torch

from deltazip_b200 import registry
from deltazip_b200.cache import AttnMeta, PagedKVCache, RecurrentStateCache
from deltazip_b200.mixers import LatentAttention, LatentAttentionSpec, LightningSpec, RoutedExpertsSpec
from oracle import movarax_oracle as O
from tests import movarax_util as U


def model_of(config, dtype=torch.float32):
    entry = registry.lookup(config)
    cfg = entry.config_class.from_dict(config)
    return entry, cfg, entry.model_class(cfg, device="cpu", dtype=dtype)


def test_config_and_registry():
    config = U.make_config()
    entry = registry.lookup(config)
    cfg = entry.config_class.from_dict(config)
    assert entry.name == "Movarax" and registry.entry_for(cfg) is entry
    assert cfg.embed_scale == 1.7 and cfg.eps == 1e-5 and cfg.vocab_size == 203
    assert cfg.layers[0].mlp == 96 and cfg.layers[3].mlp is None
    assert cfg.layers[1].mlp == RoutedExpertsSpec(6, 2, 40, 72) and cfg.layers[2].mlp == RoutedExpertsSpec(6, 1, 40, None)
    assert cfg.layers[2].mixer.kv_from == 0 and cfg.layers[0].mixer.kv_from is None
    assert cfg.layers[3].mixer == LightningSpec(2, 32, 24, (0.5, 0.97))


@pytest.mark.parametrize("change", [
    lambda c: c["layers"][0].update(type="conv"),
    lambda c: c["layers"][0]["mlp"].update(kind="sparse"),
    lambda c: c["layers"][0]["mixer"]["rot"].update(dims=6),
    lambda c: c["layers"][1]["mlp"]["router"].update(top=7),
    lambda c: c["layers"][1]["mixer"].update(decay=[0.5]),
    lambda c: c["layers"][2]["mixer"].update(kv_from=1),          # a layer without latents
    lambda c: c["layers"][2]["mixer"].update(kv_from=4),          # a later layer
    lambda c: c["layers"][2]["mixer"].update(kv_rank=64),         # rows of another size
    lambda c: c["layers"][4]["mixer"].update(kv_from=2),          # a layer that has none of its own
])
def test_config_errors(change):
    config = copy.deepcopy(U.make_config())
    change(config)
    with pytest.raises(ValueError):
        registry.lookup(config).config_class.from_dict(config)


def test_cache_runs_and_weights():
    config = U.make_config()
    tensors = U.make_tensors(config)
    entry, cfg, _ = model_of(config)
    model = entry.from_tensors(cfg, tensors, "cpu", torch.float32)
    assert [run for _, run in model.plan] == [0, 0, 0, 1, 1]             # layer 2 reads the rows of layer 0
    assert model.window is None and model.kv_heads == 1
    cache = model.make_cache(5, 4, 3)
    assert [tuple(k.shape) for k in cache.k] == [(20, 1, 64)] * 2 and all(v.numel() == 0 for v in cache.v)
    assert [tuple(s.shape) for s in cache.state.S] == [(3, 3, 16, 40), (3, 2, 32, 24)]
    assert cache.state.n == [None, None] and cache.blocks_for(17) == 5
    assert torch.equal(model.layers[1].mlp.up[3], tensors["l1.mlp.e3.up"].float())
    w = model.layers[4].mixer.expand                                     # rows to keys and values of all heads
    row = torch.randn(64)
    got = w @ row
    assert torch.allclose(got[:96].view(3, 32)[:, :24].reshape(-1), tensors["l4.mix.uk"].float() @ row[:56], atol=1e-5)
    assert torch.equal(got[:96].view(3, 32)[:, 24:], row[56:].expand(3, 8))
    assert torch.allclose(got[96:], tensors["l4.mix.uv"].float() @ row[:56], atol=1e-5)
    for broken in ({"l0.mix.sink"}, set()):
        t = {k: v for k, v in tensors.items() if k not in broken}
        if not broken:
            t["l2.mix.dkv"] = tensors["l0.mix.dkv"]                      # a reading layer has none
        with pytest.raises(ValueError):
            entry.from_tensors(cfg, t, "cpu", torch.float32)


def test_powers_of_the_decay():
    _, _, model = model_of(U.make_config(layers=[U.lightning_layer(decay=(0.0, 1.0, 0.3))]))
    p = model.layers[0].mixer.powers
    assert model.window == 0 and p.shape == (3, 65)
    assert p[0].tolist() == [1.0] + [0.0] * 64 and p[1].eq(1).all() and torch.isclose(p[2, 5], torch.tensor(0.3 ** 5))


def test_rows_of_a_batch_by_portion_length():
    layer = LatentAttention(LatentAttentionSpec(2, 8, 4, 8, 12, 0.3, 100.0), 32, 1e-5, "cpu", torch.float32)
    layer.prepare()
    counts, ctx = [20, 1, 16, 0, 17, 40], [0, 9, 3, 5, 100, 7]
    starts = torch.tensor([0, 20, 21, 37, 37, 54, 94], dtype=torch.int32)
    meta = AttnMeta(block_tables=torch.arange(6, dtype=torch.int32)[:, None], prompt_lens=counts, q_starts=starts,
                    ctx_lens=torch.tensor(ctx, dtype=torch.int32), host_ctx_lens=ctx)
    short, groups = layer._plan(meta, 10 ** 9)
    assert (short.rows, short.first, short.count) == (None, 20, 17) and short.q_starts.tolist() == [0, 1, 17]
    assert short.ctx_lens.tolist() == [9, 3] and short.block_tables.tolist() == [[1], [2]]
    assert len(groups) == 1
    g = groups[0]
    assert g.rows.tolist() == list(range(20)) + list(range(37, 94)) and g.q_starts.tolist() == [0, 20, 37, 77]
    assert g.kv_starts.tolist() == [0, 20, 137, 184] and (g.total, g.longest, g.max_query) == (184, 117, 40)
    x = torch.arange(94.0)[:, None]
    out = torch.zeros(94, 1)
    for part in (short, g):
        part.put(out, part.take(x) + 1)
    assert torch.equal(out, x + 1)
    _, groups = layer._plan(meta, 130)                                   # no more rows at a time than this
    assert [g.kv_starts.tolist() for g in groups] == [[0, 20], [0, 117], [0, 47]]
    assert [(g.first, g.count) for g in groups] == [(0, 20), (37, 17), (54, 40)]
    meta = AttnMeta(block_tables=torch.zeros(2, 1), q_starts=starts[:3], ctx_lens=torch.tensor([4, 4]))
    short, groups = layer._plan(meta, 1)
    assert groups == [] and short.count == 2


def test_state_pools_without_a_normaliser():
    s = RecurrentStateCache([(2, 3, 4), (1, 5, 6)], 7, "cpu", [False, True])
    assert s.n[0] is None and s.m[0] is None and s.n[1].shape == (7, 1, 5)
    c = PagedKVCache(1, 3, 1, 4, torch.float32, "cpu", layer_shapes=[(1, 9, 0)], state=s)
    assert c.k[0].shape == (12, 1, 9) and c.v[0].shape == (12, 1, 0)


# -- the oracle against itself -------------------------------------------------------------------

def test_oracle_rotation_keeps_relative_positions():
    rng = np.random.default_rng(0)
    q, k = rng.normal(size=(1, 6)), rng.normal(size=(1, 6))
    dot = lambda a, b: float(O.rotate_pairs(q, np.array([a]), 50.0)[0] @ O.rotate_pairs(k, np.array([b]), 50.0)[0])
    assert np.isclose(dot(9, 4), dot(105, 100)) and not np.isclose(dot(9, 4), dot(9, 5))
    z = (q[0, 0::2] + 1j * q[0, 1::2]) * np.exp(1j * 7 * 50.0 ** (-np.arange(3) / 3.0))
    got = O.rotate_pairs(q, np.array([7]), 50.0)[0]
    assert np.allclose(got[0::2] + 1j * got[1::2], z)


def test_oracle_sink_takes_weight_but_has_no_value():
    s = np.array([[0.3, -1.0, -np.inf]])
    got = O.softmax_with_sink(s, 0.7)
    e = np.exp([0.3, -1.0, 0.7])
    assert np.allclose(got, [[e[0] / e.sum(), e[1] / e.sum(), 0.0]])
    assert np.allclose(O.softmax_with_sink(s, 900.0), 0) and np.allclose(O.softmax_with_sink(s, -900.0).sum(), 1)


def test_oracle_latent_form_equals_expanded_form():
    rng = np.random.default_rng(1)
    mix = {"dim": 3, "rot": {"base": 20.0}, "scale": 0.4}
    q, c, r = rng.normal(size=(5, 2, 7)), rng.normal(size=(5, 6)), rng.normal(size=(5, 4))
    uk, uv, sink = rng.normal(size=(2, 3, 6)), rng.normal(size=(2, 5, 6)), np.array([0.5, -0.2])
    want = O.latent_attention_core(q, c, r, uk, uv, mix, sink)
    turned = O.rotate_pairs(q[..., 3:], np.arange(5), 20.0)
    for a in range(2):
        lat = np.concatenate([q[:, a, :3] @ uk[a], turned[:, a]], 1)
        s = lat @ np.concatenate([c, r], 1).T * 0.4
        p = O.softmax_with_sink(np.where(np.tri(5, dtype=bool), s, -np.inf), sink[a])
        assert np.allclose(p @ c @ uv[a].T, want[:, a])


def test_oracle_decayed_sum_in_closed_form():
    rng = np.random.default_rng(2)
    q, k, v = rng.normal(size=(9, 4)), rng.normal(size=(9, 4)), rng.normal(size=(9, 3))
    n = np.arange(9)[:, None] - np.arange(9)[None, :]
    w = np.where(n >= 0, 0.8 ** np.maximum(n, 0), 0.0)
    assert np.allclose(O.decayed_sum(q, k, v, 0.8), (w * (q @ k.T)) @ v)


def test_oracle_mixture_token_by_token():
    rng = np.random.default_rng(3)
    mlp = U.moe(experts=4, top=2, ff=5, shared=3)
    w = {f"e{e}.up": rng.normal(size=(5, 6)) for e in range(4)} | {f"e{e}.down": rng.normal(size=(6, 5)) for e in range(4)}
    w |= {"shared.up": rng.normal(size=(3, 6)), "shared.down": rng.normal(size=(6, 3)), "router": rng.normal(size=(4, 6))}
    h = rng.normal(size=(7, 6))
    got = O.mixture(h, w, mlp)
    for t in range(7):
        s = 1 / (1 + np.exp(-w["router"] @ h[t]))
        want = w["shared.down"] @ np.maximum(w["shared.up"] @ h[t], 0) ** 2
        for e in sorted(range(4), key=lambda e: -s[e])[:2]:
            want = want + s[e] ** 2 * (w[f"e{e}.down"] @ np.maximum(w[f"e{e}.up"] @ h[t], 0) ** 2)
        assert np.allclose(got[t], want)


def test_oracle_forward_is_causal_and_reads_the_other_layers_latents():
    config = U.make_config()
    tensors = U.make_tensors(config)
    toks = [3, 7, 100, 7, 55]
    a, b = U.oracle_logits(config, tensors, toks), U.oracle_logits(config, tensors, toks[:3])
    assert np.allclose(a[:3], b)
    changed = dict(tensors)
    changed["l0.mix.dkv"] = tensors["l0.mix.dkv"].flip(0)
    config2 = U.make_config(layers=config["layers"][:3])
    keep = {k: v for k, v in tensors.items() if not k.startswith(("l3.", "l4."))}
    x = [U.oracle_logits(config2, {**keep, **{k: changed[k] for k in keep}}, toks), U.oracle_logits(config2, keep, toks)]
    assert not np.allclose(*x)
