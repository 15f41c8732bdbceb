"""Movarax on the GPU against the plain numpy oracle: every mechanism alone, then whole models through the
engine -- prompts, portions, decoding, batches, reused pages and slots, generation, the command line and
deltas on top."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from oracle import movarax_oracle as O
from tests import movarax_util as U

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F32, BF16, F16 = torch.float32, torch.bfloat16, torch.float16
EXACT = {F32: 2e-5, F16: 4e-3, BF16: 2e-2}


def rel(got, want):
    got, want = np.asarray(got, dtype=np.float64), np.asarray(want, dtype=np.float64)
    return np.abs(got - want).max() / max(np.abs(want).max(), 1e-30)


def host(t):
    return t.double().cpu().numpy()


def dev(a, dtype=F32):
    return torch.tensor(np.asarray(a), device="cuda").to(dtype)


def i32(x):
    return torch.tensor(np.asarray(x), dtype=torch.int32, device="cuda")


def tokens_of(n, vocab, seed):
    return np.random.default_rng(seed).integers(0, vocab, size=n).tolist()


# -- element-wise steps ----------------------------------------------------------------------------

@pytest.mark.parametrize("width", [64, 77, 4096])
@pytest.mark.parametrize("dtype", [F32, F16, BF16])
def test_residual_sums_routed_rows_and_scaled_embedding(width, dtype):
    from deltazip_b200 import ops
    rng = np.random.default_rng(width)
    m, eps = 5, 1e-3
    rows, w = dev(rng.normal(size=(9, width)), dtype), dev(rng.normal(size=width))
    index = i32([[0, 8], [-1, 3], [3, 3], [-1, -1], [7, 2]])
    picked = np.stack([sum((host(rows)[j] for j in r if j >= 0), np.zeros(width)) for r in index.cpu().numpy()])
    for d in (None, dev(rng.normal(size=(m, width)), dtype)):
        x = dev(rng.normal(size=(m, width)))
        want = host(x) + picked + (0 if d is None else host(d))
        update = ops.Update(d, rows, index)
        assert rel(host(update.dense()), want - host(x)) < 1e-6
        out = ops.residual_norm(x, update, w, eps, dtype)
        assert rel(host(x), want) < 1e-6
        assert rel(host(out), O.rms_norm(want, host(w), eps)) < EXACT[dtype]
    table, toks = dev(rng.normal(size=(11, width)), dtype), torch.tensor([3, 10, 0], device="cuda")
    r = ops.embed_norm(toks, table, None, eps, scale=2.7)
    assert r.dtype == F32 and rel(host(r), 2.7 * host(table)[[3, 10, 0]]) < 1e-6
    r = ops.embed_norm(toks, table, w, eps, scale=0.01)
    assert rel(host(r), O.rms_norm(0.01 * host(table)[[3, 10, 0]], host(w), eps)) < 2e-6


@pytest.mark.parametrize("inter", [8, 100, 2000])
@pytest.mark.parametrize("dtype", [F32, F16, BF16])
def test_activations(inter, dtype):
    from deltazip_b200 import ops
    x = (torch.randn((7, 2 * inter + 8), device="cuda") * 3).to(dtype)
    z, u = host(x)[:, :inter], host(x)[:, inter:2 * inter]
    assert rel(host(ops.act(x, "relu2", inter)), O.squared_relu(z)) < EXACT[dtype]
    assert rel(host(ops.act(x, "silu", inter)), O.silu(z)) < EXACT[dtype]
    assert rel(host(ops.gated_act(x, "relu2", inter)), O.squared_relu(z) * u) < EXACT[dtype]


# -- latent rows -----------------------------------------------------------------------------------

@pytest.mark.parametrize("sizes", [(3, 24, 8, 56), (2, 5, 2, 9), (4, 128, 64, 512), (1, 0, 6, 16)])
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_rotation_norm_and_append(sizes, dtype):
    from deltazip_b200 import ops
    heads, dim, rot, rank = sizes
    rng = np.random.default_rng(rank)
    base, m, qw = 5e5, 6, heads * (dim + rot)
    pos = np.array([0, 1, 2, 1000, 131071, 2 ** 22 + 1])
    x = dev(rng.normal(size=(m, qw + rank + rot + 6)), dtype)
    x0, w = host(x), dev(rng.normal(size=rank) + 1)
    freq = torch.tensor(base ** (-2.0 * np.arange(rot // 2) / rot), device="cuda", dtype=torch.float64)
    positions = torch.tensor(pos, device="cuda")
    cache = torch.zeros((9, 1, rank + rot), dtype=dtype, device="cuda")
    slots = torch.tensor([8, -1, 0, 3, 5, 7], device="cuda")
    q_out = torch.zeros((m, heads, rank + rot), dtype=dtype, device="cuda")
    ops.latent_rows(x, positions, freq, heads, dim, rot, rank, q_out, qw, w, 1e-4, cache, slots)
    assert np.array_equal(host(x), x0)
    want = O.rotate_pairs(x0[:, :qw].reshape(m, heads, dim + rot)[..., dim:], pos, base)
    assert rel(host(q_out)[..., rank:], want) < EXACT[dtype] and not q_out[..., :rank].any()
    c, r = O.rms_norm(x0[:, qw:qw + rank], host(w), 1e-4), O.rotate_pairs(x0[:, qw + rank:qw + rank + rot], pos, base)
    for row, s in enumerate([8, None, 0, 3, 5, 7]):
        if s is not None:
            assert rel(host(cache)[s, 0, :rank], c[row]) < EXACT[dtype] and rel(host(cache)[s, 0, rank:], r[row]) < EXACT[dtype]
    assert not cache[[1, 2, 4, 6]].any()
    ops.latent_rows(x, positions, freq, heads, dim, rot, rank)           # in place, queries only
    y = host(x)
    assert rel(y[:, :qw].reshape(m, heads, -1)[..., dim:], want) < EXACT[dtype]
    assert np.array_equal(y[:, :qw].reshape(m, heads, -1)[..., :dim], x0[:, :qw].reshape(m, heads, -1)[..., :dim])
    assert np.array_equal(y[:, qw:], x0[:, qw:])


class LatentRun:
    """Given queries against given rows [latent | shared part] in the cache, both forms."""

    def __init__(self, heads, rank, rot, t, dtype, seed=0, block=8, scale=0.3, sink=None, rows=None, q=None):
        rng = np.random.default_rng(seed)
        d = rank + rot
        self.q = dev(rng.normal(size=(t, heads, d)) * (3 / d ** 0.5) if q is None else q, dtype)
        self.rows = dev(rng.normal(size=(t, d)) if rows is None else rows, dtype)
        self.sink = None if sink is None else dev(sink)
        self.scale, self.rank, self.heads, self.t, self.block, self.dtype = scale, rank, heads, t, block, dtype
        n = -(-t // block)
        self.table = rng.permutation(n + 3)[:n]
        self.cache = torch.full(((n + 3) * block, 1, d), float("nan"), dtype=dtype, device="cuda")
        slots = np.concatenate([b * block + np.arange(block) for b in self.table])[:t]
        self.cache[torch.tensor(slots, device="cuda"), 0] = self.rows
        qh, rh = host(self.q), host(self.rows)
        hidden = np.triu(np.ones((t, t), dtype=bool), 1)
        self.want = np.empty((t, heads, rank))
        for a in range(heads):
            s = np.where(hidden, -np.inf, qh[:, a] @ rh.T * scale)
            p = O.softmax_with_sink(s, -1e30 if sink is None else host(self.sink)[a])
            self.want[:, a] = p @ rh[:, :rank]

    def run(self, lo, hi, splits=0):
        """Rows [lo, hi) as one portion."""
        from deltazip_b200 import ops
        return host(ops.latent_attention(self.q[lo:hi].contiguous(), self.cache, i32([self.table]), i32([0, hi - lo]), i32([lo]),
                                         self.rank, self.block, self.scale, self.sink, splits))


SHAPES = [(3, 56, 8), (7, 104, 24), (16, 512, 64), (20, 64, 24), (40, 128, 8), (1, 8, 8), (2, 9, 2), (33, 24, 6), (5, 528, 16)]


@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("dtype", [F32, F16, BF16])
def test_latent_attention_kernels(shape, dtype):
    from deltazip_b200 import ops
    heads, rank, rot = shape
    t = 300 if heads * rank < 3000 else 140
    r = LatentRun(heads, rank, rot, t, dtype, seed=rank, sink=np.random.default_rng(1).normal(size=heads))
    for lo, hi in ((t - 1, t), (0, 1), (63, 65), (100, 116), (0, 40)):
        for splits in (0, 1, 3, 16):
            assert rel(r.run(lo, hi, splits), r.want[lo:hi]) < EXACT[dtype], (lo, hi, splits)
    # without a sink, other page sizes (those that are not a multiple of eight have a kernel of their own)
    for block in (12, 16, 24, 64, 128):
        r = LatentRun(heads, rank, rot, 90, dtype, seed=block, block=block)
        assert rel(r.run(70, 90), r.want[70:]) < EXACT[dtype], block
    assert ops.read_status() == 0


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_latent_attention_far_key_and_sink(dtype):
    """One key stands out from hundreds, at and around page and tile borders: every later row returns its
    latent, no earlier one does; a large sink takes the weight away, and with it the length of the output."""
    t, rank, rot, heads = 260, 16, 8, 3
    rng = np.random.default_rng(5)
    for far in (0, 1, 7, 8, 63, 64, 65, 128, 200):
        q, rows = np.zeros((t, heads, rank + rot)), rng.normal(size=(t, rank + rot)) * 0.1
        q[..., 0], rows[far, 0], rows[far, 1:rank] = 8, 8, 3          # a score of 32, the others within 2 of zero
        r = LatentRun(heads, rank, rot, t, dtype, scale=0.5, sink=[0.0, 32.0, 60.0], rows=rows, q=q)
        got = np.concatenate([r.run(0, max(far, 1)), r.run(max(far, 1), t - 1), r.run(t - 1, t, 4)])
        assert rel(got, r.want) < EXACT[dtype]
        assert np.abs(got[far:, 0, 1:] - 3).max() < 0.05 and np.abs(got[far:, 1, 1:] - 1.5).max() < 0.02
        assert np.abs(got[far:, 2]).max() < 0.01
        if far:
            assert np.abs(got[:far, 0, 1:]).max() < 0.5


def test_split_launches_of_changing_batch_size_share_a_workspace():
    """Large, small, large: what a launch keeps in the workspace is not where a larger one looks for its tickets."""
    from deltazip_b200 import ops
    g = torch.Generator(device="cuda").manual_seed(0)
    rnd = lambda *s: torch.randn(s, generator=g, device="cuda").to(BF16)
    t, bs, most = 200, 8, 96
    table, q1 = i32(np.arange(25)[None].repeat(most, 0)), torch.arange(most + 1, dtype=torch.int32, device="cuda")
    ctx = i32([t - 1] * most)
    lat, ql = rnd(200, 1, 48), rnd(most, 4, 48)
    k, v, x = rnd(200, 2, 128), rnd(200, 2, 128), rnd(most, 8 * 128)
    calls = {"latent": lambda n, s: ops.latent_attention(ql[:n], lat, table[:n], q1[:n + 1], ctx[:n], 32, bs, 0.2, None, s),
             "window": lambda n, s: ops.window_attention(x[:n], k, v, table[:n], q1[:n + 1], ctx[:n], 1, True, 4, bs, 0.1, 0,
                                                         None, s),
             "paged": lambda n, s: ops.paged_attention_decode(x[:n], k, v, table[:n], ctx[:n] + 1, 4, 2, bs, 0.1, s)}
    for name, call in calls.items():
        want = call(most, 1)
        for n in (most, 1, most, 2, 3, most):
            assert rel(host(call(n, 4)), host(want[:n])) < 1e-2, (name, n)


@pytest.mark.parametrize("grow", [False, True])
def test_latent_attention_with_scores_that_grow_along_the_keys(grow):
    """The running maximum moves by far more than rounding allows to ignore, in every tile or in none, also
    where the largest score comes first."""
    t, heads, rank, rot = 700, 20, 136, 24
    rng = np.random.default_rng(6)
    rows, q = rng.normal(size=(t, rank + rot)) * 0.2, np.zeros((t, heads, rank + rot))
    rows[:, 0] = np.linspace(0, 60, t)[::1 if grow else -1]
    q[..., 0], q[..., 1:] = 2.0, rng.normal(size=(t, heads, rank + rot - 1)) * 0.1
    r = LatentRun(heads, rank, rot, t, F16, scale=0.8, rows=rows, q=q, sink=rng.normal(size=heads) * 20)
    for splits in (1, 4):
        assert rel(r.run(t - 2, t, splits), r.want[t - 2:]) < EXACT[F16]


def test_first_tokens_see_themselves_and_the_sink():
    r = LatentRun(2, 16, 8, 4, F32, sink=[0.4, -1.0])
    s = (host(r.q)[0] @ host(r.rows)[0]) * r.scale
    want = (np.exp(s) / (np.exp(s) + np.exp(host(r.sink))))[:, None] * host(r.rows)[0, :16]
    assert rel(r.run(0, 1)[0], want) < 1e-5


@pytest.mark.parametrize("shape", [(2, 80, 64), (3, 32, 40), (2, 192, 128), (1, 136, 24), (2, 9, 5), (1, 200, 72)])
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_expanded_attention_with_sinks(shape, dtype):
    """Keys and values in rows of their own, several sequences with and without context, every portion size
    (the tcgen05 kernel takes the long ones)."""
    from deltazip_b200 import ops
    heads, dim, vdim = shape
    rng = np.random.default_rng(dim)
    ctx, new = [0, 300, 17, 64], [270, 200, 1, 65]
    for cut in (slice(0, 4), slice(1, 3), slice(2, 4)):
        c, n = ctx[cut], new[cut]
        starts, kv_starts = np.concatenate([[0], np.cumsum(n)]), np.concatenate([[0], np.cumsum(np.add(c, n))])
        pad = 8 - heads * dim % 8 if dim % 8 == 0 else 3
        q = dev(rng.normal(size=(starts[-1], heads * dim + pad)), dtype)
        kv = dev(rng.normal(size=(kv_starts[-1], heads * (dim + vdim))) * np.linspace(0.3, 2.0, kv_starts[-1])[:, None], dtype)
        sink = dev(rng.normal(size=heads) + 2)
        scale = 1.4 * dim ** -0.5
        got = host(ops.rows_attention(q, kv, i32(starts), i32(c), i32(kv_starts), max(n), heads, heads, dim, vdim, scale, sink))
        for i in range(len(c)):
            qi = host(q)[starts[i]:starts[i + 1], :heads * dim].reshape(n[i], heads, dim)
            rows = host(kv)[kv_starts[i]:kv_starts[i + 1]]
            hidden = np.arange(c[i] + n[i])[None, :] > c[i] + np.arange(n[i])[:, None]
            for a in range(heads):
                s = qi[:, a] @ rows[:, a * dim:(a + 1) * dim].T * scale
                p = O.softmax_with_sink(np.where(hidden, -np.inf, s), host(sink)[a])
                want = p @ rows[:, heads * dim + a * vdim:heads * dim + (a + 1) * vdim]
                assert rel(got[starts[i]:starts[i + 1], a * vdim:(a + 1) * vdim], want) < EXACT[dtype]
    assert ops.read_status() == 0


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_window_attention_takes_a_sink_too(dtype):
    from deltazip_b200 import ops
    from deltazip_b200.cache import PagedKVCache
    rng = np.random.default_rng(2)
    heads, kvh, dim, vdim, window, t = 4, 2, 32, 40, 21, 150
    x = dev(rng.normal(size=(t, heads * dim + kvh * (dim + vdim))), dtype)
    sink = dev(rng.normal(size=heads) + 1)
    cache = PagedKVCache(1, 8, kvh, 4, dtype, "cuda", layer_shapes=[(kvh, dim, vdim)], window=window)
    blocks = cache.allocate(cache.blocks_for(t))
    q, k, v = np.split(host(x), [heads * dim, (heads + kvh) * dim], axis=1)
    q, k, v = q.reshape(t, heads, dim), k.reshape(t, kvh, dim), v.reshape(t, kvh, vdim)
    n = np.arange(t)[:, None] - np.arange(t)[None, :]
    want = np.concatenate([O.softmax_with_sink(np.where((n >= 0) & (n < window), q[:, a] @ k[:, a // 2].T * 0.2, -np.inf),
                                               host(sink)[a]) @ v[:, a // 2] for a in range(heads)], axis=1)
    at, got = 0, []
    for size in [80, 30, 3] + [1] * 37:
        part = x[at:at + size].clone()
        slots = torch.tensor(cache.slots(blocks, at, size), device="cuda")
        if size == 1:
            ops.kv_append(part, heads * dim, cache.k[0], cache.v[0], slots)
        got.append(host(ops.window_attention(part, cache.k[0], cache.v[0], i32([blocks]), i32([0, size]), i32([at]), size,
                                             size == 1, heads, 4, 0.2, window, None, at % 3, sink)))
        if size > 1:
            ops.kv_append(part, heads * dim, cache.k[0], cache.v[0], slots)
        at += size
    assert rel(np.concatenate(got), want) < EXACT[dtype]


# -- linear attention ------------------------------------------------------------------------------

class LightningRun:
    def __init__(self, heads, dim, vdim, t, dtype, seed=0, decay=None):
        from deltazip_b200 import ops
        rng = np.random.default_rng(seed)
        self.decay = np.asarray(decay if decay is not None else 1 - 0.6 ** (1 + 3 * np.arange(heads)))
        self.powers = dev(self.decay[:, None] ** np.arange(ops.LIGHTNING_POWERS))
        self.heads, self.t, self.eps = heads, t, 1e-3
        qk, vw = heads * dim, heads * vdim
        self.x = dev(rng.normal(size=(t, 2 * (qk + vw) + 8)) * 1.5, dtype)
        self.norm = dev(rng.normal(size=vw) + 1)
        q, k, v, g = np.split(host(self.x)[:, :2 * (qk + vw)], np.cumsum([qk, qk, vw]), axis=1)
        q, k, v = (O.silu(a).reshape(t, heads, -1) for a in (q, k, v))
        o = np.stack([O.decayed_sum(q[:, a], k[:, a], v[:, a], self.decay[a]) for a in range(heads)], 1)
        self.want = O.rms_norm(o.reshape(t, vw), host(self.norm), self.eps) * O.sigmoid(g)
        self.S = torch.full((3, heads, dim, vdim), float("nan"), device="cuda")

    def run(self, cuts, slot=1, chunk=lambda n: n > 4):
        from deltazip_b200 import ops
        out, at = [], 0
        for n in list(cuts) + [1] * (self.t - sum(cuts)):
            out.append(host(ops.lightning(self.x[at:at + n], self.powers, self.norm, self.S, i32([slot]), i32([0, n]), i32([at]),
                                          self.eps, chunk(n))))
            at += n
        return np.concatenate(out)


LIGHTNING_SHAPES = [(3, 16, 40), (1, 24, 24), (2, 64, 128), (4, 128, 72), (2, 256, 64), (5, 8, 8), (1, 320, 200), (5, 72, 48)]


@pytest.mark.parametrize("shape", LIGHTNING_SHAPES + [(2, 20, 12), (1, 7, 5), (2, 33, 130)])
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_lightning_recurrent(shape, dtype):
    r = LightningRun(*shape, 40, dtype)
    for cuts in ([40], [1], [2, 17]):
        assert rel(r.run(cuts, chunk=lambda n: False), r.want) < EXACT[dtype], cuts
    assert torch.isnan(r.S[0]).all() and torch.isnan(r.S[2]).all()


@pytest.mark.parametrize("shape", LIGHTNING_SHAPES)
@pytest.mark.parametrize("dtype", [BF16, F16])
def test_lightning_chunkwise(shape, dtype):
    from deltazip_b200 import ops
    assert ops.lightning_chunk_supported(shape[1], shape[2], dtype)
    assert not ops.lightning_chunk_supported(shape[1], shape[2], F32)
    r = LightningRun(*shape, 330, dtype)
    for cuts in ([330], [64, 64, 202], [63, 2, 1, 65, 199], [5, 100]):
        always = cuts != [5, 100]
        assert rel(r.run(cuts, chunk=lambda n: always or n > 4), r.want) < EXACT[dtype], cuts
    assert torch.isnan(r.S[0]).all() and torch.isnan(r.S[2]).all()


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_lightning_decays_at_their_ends_and_a_far_token(dtype):
    """Decay 0 (only the token itself), 1 (nothing is forgotten) and 0.999: one key stands out, and is read
    back exactly as far as its decay carries it, across chunk borders and in decoding."""
    t, dim, vdim, heads = 400, 16, 24, 3
    r = LightningRun(heads, dim, vdim, t, dtype, decay=[0.0, 1.0, 0.999])
    for far in (0, 62, 63, 64, 65, 130):
        x = r.x.clone()
        x[:, :2 * heads * dim] = -30.0                       # SiLU(-30) is about zero
        x[far:, [0, dim, 2 * dim]] = 4.0                     # every later query reads component 0 ...
        x[far, [heads * dim, heads * dim + dim, heads * dim + 2 * dim]] = 4.0      # ... which one key holds
        r.x = x
        qk, vw = heads * dim, heads * vdim
        q, k, v, g = np.split(host(x)[:, :2 * (qk + vw)], np.cumsum([qk, qk, vw]), axis=1)
        q, k, v = (O.silu(a).reshape(t, heads, -1) for a in (q, k, v))
        o = np.stack([O.decayed_sum(q[:, a], k[:, a], v[:, a], r.decay[a]) for a in range(heads)], 1)
        assert np.abs(o[far + 1:, 0]).max() < 1e-6 and np.allclose(o[far:, 1], o[far, 1], atol=1e-6)
        assert np.allclose(o[-1, 2], o[far, 2] * 0.999 ** (t - 1 - far), atol=1e-6)
        r.want = O.rms_norm(o.reshape(t, vw), host(r.norm), r.eps) * O.sigmoid(g)
        for cuts in ([t], [far + 1, 2, 70], [64, 64]):
            assert rel(r.run(cuts, chunk=lambda n: dtype != F32 and n > 4), r.want) < EXACT[dtype], (far, cuts)


def test_lightning_batch_of_unequal_sequences():
    from deltazip_b200 import ops
    runs = [LightningRun(2, 16, 24, t, BF16, seed=t) for t in (90, 3, 64)]
    p, norm, eps = runs[0].powers, runs[0].norm, runs[0].eps
    S = torch.zeros(4, 2, 16, 24, device="cuda")
    got = ops.lightning(torch.cat([r.x for r in runs]), p, norm, S, i32([3, 0, 2]), i32([0, 90, 93, 157]), i32([0, 0, 0]), eps, True)
    at = 0
    for r, slot in zip(runs, (3, 0, 2)):
        alone_S = torch.zeros_like(S)
        alone = ops.lightning(r.x, p, norm, alone_S, i32([1]), i32([0, r.t]), i32([0]), eps, True)
        assert torch.equal(alone, got[at:at + r.t]) and torch.equal(alone_S[1], S[slot])
        at += r.t
    x1 = torch.cat([r.x[:1] for r in runs])                  # decoding all three continues each from its own slot
    both = ops.lightning(x1, p, norm, S.clone(), i32([3, 0, 2]), i32([0, 1, 2, 3]), i32([90, 3, 64]), eps, False)
    for j, slot in enumerate((3, 0, 2)):
        one = ops.lightning(x1[j:j + 1], p, norm, S.clone(), i32([slot]), i32([0, 1]), i32([9]), eps, False)
        assert torch.equal(one, both[j:j + 1])


# -- routed experts --------------------------------------------------------------------------------

@pytest.mark.parametrize("m,experts,top", [(1, 1, 1), (7, 5, 5), (64, 6, 2), (1000, 130, 8), (5000, 40, 3), (3, 700, 1)])
def test_routing_and_sorting(m, experts, top):
    from deltazip_b200 import ops
    z = torch.randn((m, experts), device="cuda")
    z[m // 2] = 0.25                                         # a tie goes to the lower number
    if experts > 4:
        z[:, 3] = -50                                        # an expert without tokens (unless all are taken)
    r = ops.moe_route(z, top)
    zh = host(z)
    want = np.argsort(-zh, axis=-1, kind="stable")[:, :top]
    assert np.array_equal(r.ids.cpu().numpy(), want)
    assert rel(host(r.scores), O.sigmoid(np.take_along_axis(zh, want, -1))) < 1e-6
    flat = want.reshape(-1)
    order = np.argsort(flat, kind="stable")
    assert np.array_equal(r.order.cpu().numpy(), order)
    assert np.array_equal(r.offsets.cpu().numpy(), np.searchsorted(flat[order], np.arange(experts + 1)))
    assert np.array_equal(r.place.cpu().numpy().reshape(-1)[order], np.arange(m * top))
    assert torch.equal(r.sorted_scores.cpu(), r.scores.cpu().reshape(-1)[torch.tensor(order)])
    x = torch.randn((m, 24), device="cuda").to(BF16)
    assert torch.equal(ops.moe_gather(x, r).cpu(), x.cpu()[torch.tensor(order // top)])
    bad = z.clone()
    bad[0] = float("nan")                                    # no choice: the entries are left out
    r = ops.moe_route(bad, top)
    assert (r.place[0] == -1).all() and int(r.offsets[-1]) == (m - 1) * top and (r.order[(m - 1) * top:] == -1).all()


@pytest.mark.parametrize("counts,n,k", [([3, 0, 17, 1], 40, 72), ([5], 128, 64), ([0, 300, 1, 0, 700], 200, 136), ([2, 1], 9, 11),
                                        ([1] * 50, 384, 256), ([129, 257, 16, 15], 256, 512), ([0, 0, 4], 130, 24)])
@pytest.mark.parametrize("dtype", [F32, F16, BF16])
def test_grouped_gemm(counts, n, k, dtype):
    from deltazip_b200 import ops
    rng = np.random.default_rng(n)
    rows, e = sum(counts), len(counts)
    x, w = dev(rng.normal(size=(rows + 5, k)), dtype)[:rows], dev(rng.normal(size=(e, n, k)) * k ** -0.5, dtype)
    scale, offsets = dev(rng.uniform(size=rows)), i32(np.concatenate([[0], np.cumsum(counts)]))
    of = np.repeat(np.arange(e), counts)
    plain = np.einsum("rk,rnk->rn", host(x), host(w)[of])
    assert rel(host(ops.moe_gemm(x, w, offsets)), plain) < EXACT[dtype]
    got = ops.moe_gemm(x, w, offsets, scale, "relu2")
    assert rel(host(got), O.squared_relu(plain * host(scale)[:, None])) < EXACT[dtype]
    # a row does not depend on its company
    last = [i for i, c in enumerate(counts) if c][-1]
    alone = ops.moe_gemm(x[rows - 1:].contiguous(), w, i32([0] * (last + 1) + [1] * (e - last)), scale[rows - 1:].contiguous(), "relu2")
    assert rel(host(alone), host(got[rows - 1:])) < EXACT[dtype]
    assert ops.read_status() == 0


@pytest.mark.parametrize("shared", [None, 40])
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_routed_experts_module(shared, dtype):
    from deltazip_b200.mixers import RoutedExperts, RoutedExpertsSpec
    rng = np.random.default_rng(8)
    mlp = U.moe(experts=5, top=3, ff=24, shared=shared)
    mod = RoutedExperts(RoutedExpertsSpec.from_dict(mlp), 48, "relu2", "cuda", dtype)
    w = {}
    for name, view in mod.weight_views().items():
        view.data.copy_(dev(rng.normal(size=view.shape) * view.shape[1] ** -0.5 * 1.5, dtype))
        w[name] = host(view)
    h = dev(rng.normal(size=(200, 48)), dtype)
    z = np.sort(host(h) @ w["router"].T, axis=-1)
    clear = z[:, 2] - z[:, 1] > 1e-3                         # the third and the fourth choice are not as good as equal
    got, want = host(mod(h).dense()), O.mixture(host(h), w, mlp)
    assert clear.sum() > 190 and rel(got[clear], want[clear]) < EXACT[dtype]


# -- whole models through the engine ---------------------------------------------------------------

CONFIGS = {
    "mixed": U.make_config(),
    "equal sizes": U.make_config(layers=[U.latent_layer(U.moe(experts=2, top=1, ff=32, shared=32), heads=2, dim=32, rot_dim=32,
                                                        vdim=32, kv_rank=32),
                                         U.lightning_layer(U.dense(64), heads=2, dim=32, vdim=32, decay=(0.9, 0.9))], scale=1.0),
    "odd sizes": U.make_config(layers=[U.lightning_layer(U.moe(experts=3, top=2, ff=21, shared=13), heads=1, dim=9, vdim=14),
                                       U.latent_layer(U.dense(33), heads=3, dim=5, rot_dim=6, vdim=7, kv_rank=11),
                                       U.latent_layer(U.moe(experts=7, top=7, ff=10, shared=None), heads=1, dim=10, rot_dim=6, vdim=3,
                                                      kv_rank=11, kv_from=1)], vocab=101, width=77, scale=0.6),
    "attention only": U.make_config(layers=[U.latent_layer(U.dense(), heads=20, dim=64, rot_dim=16, vdim=64, kv_rank=128, scale=0.1),
                                            U.latent_layer(None, heads=2, rot_dim=16, kv_rank=128, kv_from=0),
                                            U.latent_layer(None, heads=4, rot_dim=16, kv_rank=128, kv_from=0)]),
    "recurrent only": U.make_config(layers=[U.lightning_layer(U.moe()), U.lightning_layer(None, dim=64, vdim=64, kind="lightning_2")]),
}


@pytest.mark.parametrize("name", list(CONFIGS))
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_model_prompts_portions_and_decoding(name, dtype):
    config = CONFIGS[name]
    tensors = U.make_tensors(config, seed=len(name))
    eng = U.make_engine(config, tensors, dtype)
    toks = tokens_of(151, config["vocab"], 1)
    want = U.oracle_logits(config, tensors, toks)
    # the sequence is opened anew each time: its pages and state slot are those just given back
    for cuts in ([151], [120], [1], [64, 2, 2, 3, 31], [2] * 75, [33, 17, 96], [16, 17, 16, 70]):
        seq = U.open_sequence(eng, 5, 160)
        U.assert_logits(U.run_cuts(eng, seq, toks, cuts), want, dtype, cuts[:5])
        eng.retire(seq)
    assert len(eng.cache.free) == 64 and not eng.running
    # a prompt that is taken in several passes of at most 40 rows
    eng.max_prefill_tokens = 40
    seq = U.open_sequence(eng, 6, 160)
    U.assert_logits(U.run_cuts(eng, seq, toks, [140]), want, dtype)


def test_residual_after_every_layer():
    config = CONFIGS["mixed"]
    tensors = U.make_tensors(config, seed=2)
    eng = U.make_engine(config, tensors, F32)
    toks = tokens_of(50, config["vocab"], 3)
    want, got = [], []
    U.oracle_logits(config, tensors, toks, want)
    forward = eng.model.forward
    eng.model.forward = lambda t, p, c, meta: forward(t, p, c, meta, trace=got)
    eng.extend([(U.open_sequence(eng, 0, 60), toks)])
    assert len(got) == len(want) == 5
    for a, b in zip(got, want):
        assert rel(host(a), b) < 1e-4


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_mixed_batches_equal_each_alone(dtype):
    config = CONFIGS["mixed"]
    tensors = U.make_tensors(config, seed=4)
    prompts = [tokens_of(n, config["vocab"], n) for n in (90, 1, 34, 2, 60)]
    want = [U.oracle_logits(config, tensors, p) for p in prompts]
    eng = U.make_engine(config, tensors, dtype, kv_blocks=70)
    for layer in eng.model.layers:
        if hasattr(layer.mixer, "EXPANDED_BYTES"):           # two groups of sequences in the expanded form
            layer.mixer.EXPANDED_BYTES = 70 * layer.mixer.expand.shape[0] * layer.mixer.expand.element_size()
    seqs = [U.open_sequence(eng, i, 100) for i in range(5)]
    at, got = [0] * 5, [[] for _ in prompts]
    # every step another mixture of long portions, short ones and single tokens; 3 also ends and restarts
    plan = [[60, 1, 2, 0, 7], [1, 0, 1, 2, 1], [5, 0, 20, 0, 40], [1, 0, 1, 0, 1], [23, 0, 10, 0, 11]]
    for step in plan:
        work = [(i, prompts[i][at[i]:at[i] + n]) for i, n in enumerate(step) if n]
        work = work[::-1]
        with torch.inference_mode():
            out = eng.model.logits(eng.extend([(seqs[i], t) for i, t in work])).double().cpu().numpy()
        row = 0
        for i, t in work:
            got[i].append(out[row:row + len(t)])
            at[i] += len(t)
            row += len(t)
        if at[3] == 2 and seqs[3] in eng.running:
            eng.retire(seqs[3])
    assert at == [len(p) for p in prompts]
    for i in range(5):
        U.assert_logits(np.concatenate(got[i]), want[i], dtype, i)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_long_decoding_stays_on_the_oracle(dtype):
    config = CONFIGS["mixed"]
    tensors = U.make_tensors(config, seed=6)
    toks = tokens_of(400, config["vocab"], 7)
    eng = U.make_engine(config, tensors, dtype)
    got = U.run_cuts(eng, U.open_sequence(eng, 0, 400), toks, [3])
    U.assert_logits(got, U.oracle_logits(config, tensors, toks), dtype)


def greedy_oracle(config, tensors, prompt, steps):
    toks, margin = list(prompt), []
    for _ in range(steps):
        y = U.oracle_logits(config, tensors, toks)[-1]
        top = np.sort(y)[-2:]
        margin.append((top[1] - top[0]) / y.std())
        toks.append(int(y.argmax()))
    return toks[len(prompt):], margin


def test_generation_through_the_scheduler():
    """More requests than batch slots, unequal prompts, greedy: every request equals the oracle alone."""
    config = CONFIGS["mixed"]
    tensors = U.make_tensors(config, seed=8)
    prompts = [tokens_of(n, config["vocab"], n) for n in (40, 3, 17, 1, 70, 9)]
    eng = U.make_engine(config, tensors, F32, max_seqs=3, kv_blocks=24, max_prefill=32)
    got = eng.generate(prompts, 12)
    for p, g in zip(prompts, got):
        want, margin = greedy_oracle(config, tensors, p, 12)
        same = next((i for i in range(12) if g[i] != want[i]), 12)
        assert same == 12 or margin[same] < 1e-3, (same, margin[same])
    assert not eng.running and len(eng.cache.free) == 24 and len(eng.cache.state.free) == 3
    again = eng.generate(prompts[::-1], 12)                  # other slots, other company
    assert again[::-1] == got
    stop = got[1][4]
    assert eng.generate([prompts[1]], 12, stop_id=stop) == [got[1][:got[1].index(stop) + 1]]
    # the 16-bit engine agrees wherever the oracle's choice is clear
    half = U.make_engine(config, tensors, BF16, max_seqs=3, kv_blocks=24).generate(prompts, 12)
    for p, g in zip(prompts, half):
        want, margin = greedy_oracle(config, tensors, p, 12)
        same = next((i for i in range(12) if g[i] != want[i]), 12)
        assert same == 12 or margin[same] < 0.3, (same, margin[same])


def test_command_line_and_replay(tmp_path):
    config = CONFIGS["mixed"]
    tensors = U.make_tensors(config, seed=9)
    U.write_checkpoint(str(tmp_path), config, tensors)
    prompt = [5, 9, 200, 31]
    run = subprocess.run([sys.executable, "-m", "deltazip_b200", "generate", "--model", str(tmp_path), "--prompt",
                          " ".join(map(str, prompt)), "--max-new", "5", "--dtype", "float32"], cwd=ROOT,
                         capture_output=True, text=True, timeout=300)
    assert run.returncode == 0, run.stderr[-2000:]
    want, margin = greedy_oracle(config, tensors, prompt, 5)
    if min(margin) > 1e-3:
        assert json.loads(run.stdout.splitlines()[-1]) == want
    toks = tokens_of(30, config["vocab"], 1)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:20], "want": [0, 19]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": toks[20:22], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": toks[22:23], "want": [0]},
                                     {"id": "y", "tokens": toks[:9], "want": [8]}], "end": ["x", "y"]},
             {"step": 3, "entries": [{"id": "x", "tokens": toks[:7], "want": [6]}], "end": ["x"]}]
    run = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32",
                          "--out", str(tmp_path), "--max-tokens", "64"], input="\n".join(map(json.dumps, steps)),
                         cwd="/", capture_output=True, text=True, timeout=300)
    assert run.returncode == 0, run.stderr[-2000:]
    assert [x for x in run.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
    want = U.oracle_logits(config, tensors, toks)
    for i, rows in ((0, [0, 19]), (2, [22, 8]), (3, [6])):
        got = np.fromfile(tmp_path / f"{i}.f32", dtype="<f4").reshape(len(rows), config["vocab"])
        U.assert_logits(got.astype(np.float64), want[rows], F32)
    assert not (tmp_path / "1.f32").exists()


def test_deltas_on_top_of_the_model():
    """The model's projections are ordinary delta layers: a batch in which every request selects its own
    compressed delta equals, request by request, the model with that delta added to its weights."""
    from deltazip_b200 import ops, synth
    from deltazip_b200.config import DeltaConfig
    from deltazip_b200.engine import Sequence
    from deltazip_b200.models import DeltaModel
    layers = [U.latent_layer(U.dense(128), heads=4, dim=24, rot_dim=8, vdim=32, kv_rank=56),
              U.lightning_layer(U.moe(experts=4, top=2, shared=128), heads=2, dim=64, vdim=64)]
    config = U.make_config(layers=layers, width=128, vocab=256)
    tensors = U.make_tensors(config, seed=10)
    eng = U.make_engine(config, tensors, BF16, deltas=DeltaConfig(max_deltas=2, max_bitwidth=4))
    mgr = eng.manager
    assert sorted(n.split(".")[-1] for n in mgr.modules) == sorted(
        ["q_latent_proj", "o_proj", "gate_up_proj", "down_proj", "qkvg_proj", "o_proj", "up_proj", "down_proj"])
    g = torch.Generator(device="cuda").manual_seed(1)
    dense = {}
    for did in (1, 2):
        parts = {}
        for name, mod in mgr.modules.items():
            n, k = mod.weight.shape
            w = torch.randn((n, k), generator=g, device="cuda") * 0.04
            if name.split(".")[-1] in ("o_proj", "down_proj"):
                w[:6] = 0                                    # the routers' own coordinates, as in the model
            parts[name] = synth.compress_delta_gptq(w, 4)
        dm = DeltaModel.from_gptq_tensors(did, 4, parts)
        mgr.add_delta(dm)
        dense[did] = {name: ops.unpack(w.qweight.cuda(), w.meta.cuda(), w.scales.cuda(), *mgr.modules[name].weight.shape,
                                       4).double().cpu() for name, w in dm.deltas.items()}
    prompts = [tokens_of(n, 256, n) for n in (30, 9, 17)]
    seqs = [Sequence(i, d, 0, 40) for i, d in enumerate((2, 0, 1))]
    assert len(eng.admit(list(seqs))) == 3
    got = [[] for _ in seqs]
    for lo, hi in ((0, 8), (8, 9), (9, 40)):
        work = [(i, p[lo:hi]) for i, p in enumerate(prompts) if p[lo:hi]]
        with torch.inference_mode():
            out = eng.model.logits(eng.extend([(seqs[i], t) for i, t in work])).double().cpu().numpy()
        row = 0
        for i, t in work:
            got[i].append(out[row:row + len(t)])
            row += len(t)
    base = [U.oracle_logits(config, tensors, p) for p in prompts]
    for i, d in enumerate((2, 0, 1)):
        t = {k: v.double() for k, v in tensors.items()}
        for name, delta in dense.get(d, {}).items():
            li, leaf = name.split(".")[1], name.split(".")[-1]
            down = ["mlp.down"] if f"l{li}.mlp.down" in t else ["mlp.shared.down"]
            parts = {"q_latent_proj": ["mix.q", "mix.dkv"], "qkvg_proj": ["mix.q", "mix.k", "mix.v", "mix.g"],
                     "o_proj": ["mix.o"], "gate_up_proj": ["mlp.gate", "mlp.up"], "down_proj": down,
                     "up_proj": ["mlp.shared.up"]}[leaf]
            row = 0
            for p in parts:
                key = f"l{li}.{p}"
                t[key] = t[key] + delta[row:row + t[key].shape[0]]
                row += t[key].shape[0]
        want = U.oracle_logits(config, t, prompts[i])
        U.assert_logits(np.concatenate(got[i]), want, BF16)
        assert d == 0 or U.logit_errors(base[i], want).mean() > 0.2
