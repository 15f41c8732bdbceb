"""Buzalorn on the GPU against the plain numpy oracle: every mechanism alone, then whole models through
the engine -- prompts, portions, decoding, batches, reused pages and slots, generation, the command
line and deltas on top."""
import io
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from oracle import buzalorn_oracle as O
from tests import buzalorn_util as U

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F32, BF16, F16 = torch.float32, torch.bfloat16, torch.float16
EXACT = {F32: 2e-5, F16: 4e-3, BF16: 2e-2}


def rel(got, want):
    got, want = np.asarray(got, dtype=np.float64), np.asarray(want, dtype=np.float64)
    return np.abs(got - want).max() / max(np.abs(want).max(), 1e-30)


def host(t):
    return t.double().cpu().numpy()


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device="cuda")


# -- element-wise steps ----------------------------------------------------------------------------

@pytest.mark.parametrize("width", [64, 72, 77, 4096])
@pytest.mark.parametrize("dtype", [F32, F16, BF16])
def test_residual_norm_and_embedding(width, dtype):
    from deltazip_b200 import ops
    g = torch.Generator(device="cuda").manual_seed(width)
    rnd = lambda *s: torch.randn(s, generator=g, device="cuda")
    m, eps = 5, 1e-3
    w, vec = rnd(width), rnd(width)
    for offset in (0.0, 1.0):
        for d in (None, rnd(m, width).to(dtype), rnd(m, width)):
            for replace in (False, True):
                if replace and d is None:
                    continue
                x = rnd(m, width)
                want = (0 if replace else host(x)) + (0 if d is None else host(d)) + host(vec)
                out = ops.residual_norm(x, d, w, eps, dtype, offset, vec=vec, replace=replace)
                assert rel(host(x), want) < 1e-6
                assert rel(host(out), O.rms_norm(want, eps) * (offset + host(w))) < EXACT[dtype]
    wide = torch.full((m, 2 * width), 9.0, dtype=dtype, device="cuda")      # cast only, into a slice
    ops.residual_norm(x, None, None, eps, dtype, out=wide[:, :width])
    assert rel(host(wide[:, :width]), host(x)) < EXACT[dtype] and bool((wide[:, width:] == 9).all())
    table = rnd(11, width).to(dtype)
    toks = torch.tensor([3, 10, 0], device="cuda")
    cp = torch.zeros((3, 2 * width), dtype=dtype, device="cuda")
    r = ops.embed_norm(toks, table, w, eps, 1.0, copy=cp[:, width:])
    want = O.norm_one_plus(host(table)[[3, 10, 0]], host(w), eps)
    assert r.dtype == F32 and rel(host(r), want) < 2e-6 and rel(host(cp[:, width:]), want) < EXACT[dtype]
    assert bool((cp[:, :width] == 0).all())


@pytest.mark.parametrize("inter", [8, 100, 2000])
@pytest.mark.parametrize("dtype", [F32, F16, BF16])
def test_gated_activation(inter, dtype):
    from deltazip_b200 import ops
    x = (torch.randn((7, 2 * inter), device="cuda") * 3).to(dtype)
    z, u = host(x)[:, :inter], host(x)[:, inter:]
    assert rel(host(ops.gated_act(x, "gelu_tanh")), O.gelu_tanh(z) * u) < EXACT[dtype]
    assert rel(host(ops.gated_act(x, "silu")), z * O.sigmoid(z) * u) < EXACT[dtype]
    big = torch.tensor([[-200.0, 200.0, 1.0, 1.0]], device="cuda").to(dtype)
    assert torch.isfinite(ops.gated_act(big, "gelu_tanh")).all()


@pytest.mark.parametrize("widths", [(96, 48, 40), (30, 15, 21), (4096, 1024, 1024)])
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_query_key_norm_and_append(widths, dtype):
    from deltazip_b200 import ops
    qn, kn, vn = widths
    x = torch.randn((4, qn + kn + vn + 8), device="cuda").to(dtype)
    x0 = host(x)
    wq, wk = torch.randn(qn, device="cuda"), torch.randn(kn, device="cuda")
    kc = torch.zeros((6, 1, kn), dtype=dtype, device="cuda")
    vc = torch.zeros((6, 1, vn), dtype=dtype, device="cuda")
    slots = torch.tensor([5, -1, 0, 2], device="cuda")
    ops.qk_norm(x, wq, wk, vn, 1e-4, kc, vc, slots)
    assert rel(host(x)[:, :qn], O.rms_norm(x0[:, :qn], 1e-4) * host(wq)) < EXACT[dtype]
    assert rel(host(x)[:, qn:qn + kn], O.rms_norm(x0[:, qn:qn + kn], 1e-4) * host(wk)) < EXACT[dtype]
    assert np.array_equal(host(x)[:, qn + kn:], x0[:, qn + kn:])
    for row, s in ((0, 5), (2, 0), (3, 2)):
        assert torch.equal(kc[s, 0], x[row, qn:qn + kn]) and torch.equal(vc[s, 0], x[row, qn + kn:qn + kn + vn])
    assert not kc[[1, 3, 4]].any()
    kc2, vc2 = torch.zeros_like(kc), torch.zeros_like(vc)
    ops.kv_append(x, qn, kc2, vc2, slots)
    assert torch.equal(kc, kc2) and torch.equal(vc, vc2)


# -- attention -------------------------------------------------------------------------------------

class AttentionRun:
    """One sequence's q, k, v through the cache ring in portions, each portion through the kernels
    the model uses for it."""

    def __init__(self, q, k, v, dtype, window, scale, rel_table=None, bias_max=None, block=8, spare=3):
        from deltazip_b200.cache import PagedKVCache
        from deltazip_b200.mixers import distance_bias
        t, self.heads, dim = q.shape
        kvh, vdim = k.shape[1], v.shape[2]
        self.rows = torch.tensor(np.concatenate([q.reshape(t, -1), k.reshape(t, -1), v.reshape(t, -1)], 1),
                                 device="cuda").to(dtype)
        self.parts = (self.heads * dim, kvh * dim, kvh * vdim)
        cut = np.split(host(self.rows), np.cumsum(self.parts)[:2], axis=1)
        self.want = O.attention_core(cut[0].reshape(q.shape), cut[1].reshape(k.shape), cut[2].reshape(v.shape),
                                     scale, window, rel_table, bias_max)
        self.cache = PagedKVCache(1, 70, kvh, block, dtype, "cuda", layer_shapes=[(kvh, dim, vdim)], window=window)
        self.cache.k[0].fill_(float("nan"))             # nothing may be read that was not written
        self.cache.v[0].fill_(float("nan"))
        self.cache.allocate(spare)
        self.blocks = self.cache.allocate(self.cache.blocks_for(t))[::-1]
        self.bias = distance_bias(torch.tensor(rel_table, dtype=F32), bias_max, window).cuda() \
            if rel_table is not None else None
        self.window, self.scale, self.shape = window, scale, (self.heads, vdim)

    def run(self, cuts, splits=0, decode_single=True):
        from deltazip_b200 import ops
        out, at, t = [], 0, self.rows.shape[0]
        table = i32([self.blocks])
        kc, vc = self.cache.k[0], self.cache.v[0]
        for n in list(cuts) + [1] * (t - sum(cuts)):
            x = self.rows[at:at + n].clone()
            slots = torch.tensor(self.cache.slots(self.blocks, at, n), device="cuda")
            decode = n == 1 and decode_single
            if decode:
                ops.kv_append(x, self.parts[0], kc, vc, slots)
            o = ops.window_attention(x, kc, vc, table, i32([0, n]), i32([at]), n, decode, self.heads,
                                     self.cache.block_size, self.scale, self.window, self.bias, splits)
            if not decode:
                ops.kv_append(x, self.parts[0], kc, vc, slots)
            out.append(host(o))
            at += n
        return np.concatenate(out).reshape(t, *self.shape)


SHAPES = [(4, 2, 24, 40), (3, 3, 64, 64), (8, 1, 128, 96), (6, 2, 40, 136), (2, 2, 20, 12), (1, 1, 7, 5), (5, 1, 16, 256),
          (2, 1, 264, 272)]


@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_attention_kernels(shape, dtype):
    heads, kvh, dim, vdim = shape
    rng = np.random.default_rng(dim)
    t, window = 150, 37
    q, k = rng.normal(size=(t, heads, dim)), rng.normal(size=(t, kvh, dim))
    v = rng.normal(size=(t, kvh, vdim))
    r = AttentionRun(q, k, v, dtype, window, 1.3 * dim ** -0.5, rng.normal(size=(10, heads)), 30)
    for cuts in ([t], [1], [64, 2, 3, 33], [100, 17]):
        for splits in (0, 3):
            assert rel(r.run(cuts, splits), r.want) < EXACT[dtype], (cuts, splits)
    assert rel(r.run([70, 1, 1, 30], decode_single=False), r.want) < EXACT[dtype]


@pytest.mark.parametrize("shape", [(2, 1, 128, 128), (2, 2, 64, 64), (3, 1, 72, 104), (1, 1, 40, 200)])
@pytest.mark.parametrize("window", [129, 300, 5000])
@pytest.mark.parametrize("dtype", [F16, BF16])
def test_attention_long_portions(shape, window, dtype):
    """Several 256-row blocks of the tcgen05 kernel, with and without context, running maxima that grow
    along the keys, and a table longer than a key tile."""
    heads, kvh, dim, vdim = shape
    rng = np.random.default_rng(window + dim)
    t = 900
    q, k, v = (rng.normal(size=(t, n, d)) for n, d in ((heads, dim), (kvh, dim), (kvh, vdim)))
    k *= np.linspace(0.2, 3.0, t)[:, None, None]
    r = AttentionRun(q, k, v, dtype, window, 1.5 * dim ** -0.5, rng.normal(size=(32, heads)) * 2, 200, block=16)
    for cuts in ([t], [257, 643], [100, 65, 300, 128, 307]):
        assert rel(r.run(cuts), r.want) < EXACT[dtype], cuts
    from deltazip_b200 import ops
    assert ops.read_status() == 0


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("window", [1, 2, 16, 24, 65, 500])
def test_attention_far_key_at_the_window_edge(window, dtype):
    """One key stands out from hundreds; it must be returned by exactly the rows whose window holds it,
    in prompts and in decoding, at and around page borders and tile borders."""
    t, dim, block = 220, 16, 8
    rng = np.random.default_rng(window)
    for far in (0, 7, 8, 63, 64, 100):
        q = rng.normal(size=(t, 2, dim)) * 0.1
        q[:, :, 0] = 8
        k = rng.normal(size=(t, 1, dim)) * 0.1
        k[far, 0, 0] = 8
        v = rng.normal(size=(t, 1, 24)) * 0.1
        v[far] = 3
        r = AttentionRun(q, k, v, dtype, window, 0.5, block=block)
        for cuts in ([t], [far + 1], [max(1, far - 1), 3, 40]):
            got = r.run(cuts)
            assert rel(got, r.want) < EXACT[dtype]
            inside = got[far:far + window]
            assert np.abs(inside - 3).max() < 0.05
            if far + window < t:
                assert np.abs(got[far + window]).max() < 0.6


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_distance_bias_steps(dtype):
    """Constant scores, a table with one large entry: the output jumps exactly where that bucket starts."""
    t, rows, bias_max = 130, 12, 50
    from deltazip_b200.mixers import bucket_edges
    edges = bucket_edges(rows, bias_max) + [10 ** 9]
    v = np.arange(t, dtype=float).reshape(t, 1, 1).repeat(8, 2) / t
    for b in (0, 3, 6, 9, rows - 1):
        table = np.zeros((rows, 2))
        table[b, 1] = 12.0
        r = AttentionRun(np.zeros((t, 2, 8)), np.zeros((t, 1, 8)), v, dtype, 100, 1.0, table, bias_max)
        for cuts in ([t], [60], [33, 2, 2, 50]):
            assert rel(r.run(cuts), r.want) < EXACT[dtype]
        if edges[b] > 0:
            mean = host(r.rows)[:, -1][: edges[b]].mean()                # the bucket is not reached yet
            assert abs(r.want[edges[b] - 1, 1, 0] - mean) < 1e-9


def test_attention_ragged_batch_equals_each_alone():
    from deltazip_b200 import ops
    from deltazip_b200.cache import PagedKVCache
    rng = np.random.default_rng(3)
    heads, kvh, dim, vdim, window, block = 4, 2, 32, 40, 21, 4
    ctx, new = [0, 5, 40, 0, 100], [70, 1, 2, 3, 65]
    cache = PagedKVCache(1, 64, kvh, block, BF16, "cuda", layer_shapes=[(kvh, dim, vdim)], window=window)
    width = heads * dim + kvh * (dim + vdim)
    seqs = [(torch.tensor(rng.normal(size=(c + n, width)), device="cuda").to(BF16), c, n) for c, n in zip(ctx, new)]
    blocks = [cache.allocate(cache.blocks_for(window)) for _ in seqs]
    for (rows, c, n), b in zip(seqs, blocks):
        if c:
            ops.kv_append(rows[:c], heads * dim, cache.k[0], cache.v[0],
                          torch.tensor(cache.slots(b, 0, c), device="cuda"))
    x = torch.cat([rows[c:] for rows, c, _ in seqs])
    starts = np.concatenate([[0], np.cumsum(new)])
    call = lambda x, b, st, cx, mq: ops.window_attention(x, cache.k[0], cache.v[0], i32(b), i32(st), i32(cx), mq, False,
                                                         heads, block, 0.2, window, None)
    got = call(x, blocks, starts, ctx, max(new))
    for i, (rows, c, n) in enumerate(seqs):
        alone = call(rows[c:].contiguous(), [blocks[i]], [0, n], [c], n)
        assert rel(host(got[starts[i]:starts[i + 1]]), host(alone)) < 1e-2        # kernels differ with the largest portion
        h = host(rows)
        want = O.attention_core(h[:, :heads * dim].reshape(-1, heads, dim),
                                h[:, heads * dim:(heads + kvh) * dim].reshape(-1, kvh, dim),
                                h[:, (heads + kvh) * dim:].reshape(-1, kvh, vdim), 0.2, window)[c:]
        assert rel(host(alone), want.reshape(n, -1)) < EXACT[BF16]


# -- matrix memory -----------------------------------------------------------------------------------

class MlstmRun:
    def __init__(self, heads, dim, vdim, t, dtype, seed=0, width=48, cap=6.0, i_std=2.0, f_mean=2.0, gate_scale=1.0):
        rng = np.random.default_rng(seed)
        dev = lambda a, d=dtype: torch.tensor(np.asarray(a), device="cuda").to(d)
        self.heads, self.dim, self.vdim, self.t, self.cap, self.eps = heads, dim, vdim, t, cap, 1e-5
        self.h = dev(rng.normal(size=(t, width)))
        self.w = dev(rng.normal(size=(2 * heads, width)) * i_std * width ** -0.5 * gate_scale)
        b = rng.normal(size=2 * heads)
        b[heads:] += f_mean
        self.b = dev(b, F32)
        self.norm = dev(rng.normal(size=heads * vdim) + 1, F32)
        self.x = dev(rng.normal(size=(t, 2 * heads * (dim + vdim) + 8)))
        self.scale = dim ** -0.5
        hh, w, x = host(self.h), host(self.w), host(self.x)
        pre = hh @ w.T + host(self.b)
        gi, gf = O.mlstm_gates(pre[:, :heads], pre[:, heads:], cap)
        qk, vw = heads * dim, heads * vdim
        q, k, v, g = np.split(x[:, :2 * (qk + vw)], np.cumsum([qk, qk, vw]), axis=1)
        q, k, v = (a.reshape(t, heads, -1) for a in (q * self.scale, k, v))
        self.raw = np.stack([O.mlstm_recurrence(q[:, a], k[:, a], v[:, a], gi[:, a], gf[:, a])
                             for a in range(heads)], 1)
        self.want = O.head_norm_gate(self.raw, host(self.norm), g, self.eps)
        nan = lambda *s: torch.full(s, float("nan"), device="cuda")
        self.S, self.n, self.m = nan(3, heads, dim, vdim), nan(3, heads, dim), nan(3, heads)

    def run(self, cuts, slot=1, chunk=lambda n: n > 4):
        from deltazip_b200 import ops
        out, at = [], 0
        for n in list(cuts) + [1] * (self.t - sum(cuts)):
            o = ops.mlstm(self.x[at:at + n], self.h[at:at + n], self.w, self.b, self.norm, self.S, self.n, self.m,
                          i32([slot]), i32([0, n]), i32([at]), self.cap, self.scale, self.eps, chunk(n))
            out.append(host(o))
            at += n
        return np.concatenate(out)


MLSTM_SHAPES = [(3, 16, 40), (1, 24, 24), (2, 64, 128), (4, 128, 72), (2, 256, 64), (5, 8, 8), (1, 320, 200)]


@pytest.mark.parametrize("shape", MLSTM_SHAPES + [(2, 20, 12), (1, 7, 5), (2, 33, 130)])
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_mlstm_recurrent(shape, dtype):
    r = MlstmRun(*shape, 40, dtype)
    never = lambda n: False
    for cuts in ([40], [1], [2, 17]):
        assert rel(r.run(cuts, chunk=never), r.want) < EXACT[dtype], cuts
    assert torch.isnan(r.S[0]).all() and torch.isnan(r.S[2]).all() and torch.isnan(r.m[[0, 2]]).all()


@pytest.mark.parametrize("shape", MLSTM_SHAPES)
@pytest.mark.parametrize("dtype", [BF16, F16])
def test_mlstm_chunkwise(shape, dtype):
    from deltazip_b200 import ops
    assert ops.mlstm_chunk_supported(shape[1], shape[2], dtype)
    assert not ops.mlstm_chunk_supported(shape[1], shape[2], F32)
    r = MlstmRun(*shape, 200, dtype)
    always = lambda n: True
    for cuts in ([200], [64, 64, 72], [63, 2, 1, 65, 69], [5, 100]):
        assert rel(r.run(cuts, chunk=always if cuts != [5, 100] else (lambda n: n > 4)), r.want) < EXACT[dtype], cuts


@pytest.mark.parametrize("case", ["forgets", "remembers", "denominator", "strong"])
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_mlstm_gate_extremes(case, dtype):
    """Gates at the cap both ways, m far from its start at zero, |n.q| below exp(-m) and the 1e-6 beside a
    small exp(-m)."""
    kw = {"forgets": dict(f_mean=-30.0, cap=12.0), "remembers": dict(f_mean=30.0, cap=14.0),
          "denominator": dict(i_std=0.1, f_mean=-2.0, cap=9.0), "strong": dict(i_std=40.0, cap=13.0)}[case]
    r = MlstmRun(2, 32, 40, 130, dtype, seed=5, **kw)
    if case == "denominator":
        r.b[:2] = -8.0
        hh = host(r.h) @ host(r.w).T + host(r.b)
        gi, gf = O.mlstm_gates(hh[:, :2], hh[:, 2:], r.cap)
        x = host(r.x)
        q, k, v, g = np.split(x[:, :2 * 2 * 72], np.cumsum([64, 64, 80]), axis=1)
        q, k, v = (a.reshape(r.t, 2, -1) for a in (q * r.scale, k, v))
        raw = np.stack([O.mlstm_recurrence(q[:, a], k[:, a], v[:, a], gi[:, a], gf[:, a]) for a in range(2)], 1)
        r.want = O.head_norm_gate(raw, host(r.norm), g, r.eps)
    for cuts in ([130], [1], [70, 3]):
        got = r.run(cuts, chunk=lambda n: dtype != F32 and n > 4)
        assert rel(got, r.want) < EXACT[dtype] * (5 if dtype == F32 else 1.5), cuts


def test_mlstm_batch_of_unequal_sequences():
    from deltazip_b200 import ops
    runs = [MlstmRun(2, 16, 24, t, BF16, seed=t) for t in (90, 3, 64)]
    w, b, norm = runs[0].w, runs[0].b, runs[0].norm
    S, n, m = torch.zeros(4, 2, 16, 24, device="cuda"), torch.zeros(4, 2, 16, device="cuda"), torch.zeros(4, 2, device="cuda")
    x, h = torch.cat([r.x for r in runs]), torch.cat([r.h for r in runs])
    args = (runs[0].cap, runs[0].scale, runs[0].eps)
    got = ops.mlstm(x, h, w, b, norm, S, n, m, i32([3, 0, 2]), i32([0, 90, 93, 157]), i32([0, 0, 0]), *args, True)
    at = 0
    for r, slot in zip(runs, (3, 0, 2)):
        s1, n1, m1 = torch.zeros_like(S), torch.zeros_like(n), torch.zeros_like(m)
        alone = ops.mlstm(r.x, r.h, w, b, norm, s1, n1, m1, i32([1]), i32([0, r.t]), i32([0]), *args, True)
        assert torch.equal(alone, got[at:at + r.t]) and torch.equal(s1[1], S[slot]) and torch.equal(m1[1], m[slot])
        at += r.t
    # decoding all three at once continues each from its own slot
    x1, h1 = torch.cat([r.x[:1] for r in runs]), torch.cat([r.h[:1] for r in runs])
    both = ops.mlstm(x1, h1, w, b, norm, S.clone(), n.clone(), m.clone(), i32([3, 0, 2]), i32([0, 1, 2, 3]),
                     i32([90, 3, 64]), *args, False)
    for j, slot in enumerate((3, 0, 2)):
        one = ops.mlstm(x1[j:j + 1], h1[j:j + 1], w, b, norm, S.clone(), n.clone(), m.clone(), i32([slot]),
                        i32([0, 1]), i32([9]), *args, False)
        assert torch.equal(one, both[j:j + 1])


# -- whole models through the engine ---------------------------------------------------------------

def tokens_of(n, vocab, seed):
    return np.random.default_rng(seed).integers(0, vocab, size=n).tolist()


CONFIGS = {
    "mixed": U.make_config(),
    "equal sizes": U.make_config(layers=[U.attention_layer(heads=2, kv_heads=2, dim=32, vdim=32),
                                         U.mlstm_layer(heads=2, dim=32, vdim=32, ff=64)],
                                 loop=(0, 2, 1), logit_scale=1.0),
    "loop of one, odd sizes": U.make_config(layers=[U.mlstm_layer(heads=1, dim=9, vdim=14, ff=70),
                                                    U.attention_layer(heads=3, kv_heads=1, dim=10, vdim=6, ff=33)],
                                            loop=(0, 1, 4), vocab=101, width=77),
    "attention only": U.make_config(layers=[U.attention_layer(window=64, dim=64, vdim=128),
                                            U.attention_layer(window=5, ff=None, heads=6, kv_heads=1)], loop=(0, 2, 2)),
    "memory only": U.make_config(layers=[U.mlstm_layer(), U.mlstm_layer(dim=64, vdim=64, ff=128)], loop=(1, 2, 2)),
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
    for cuts in ([151], [120], [1], [64, 2, 2, 3, 31], [2] * 75, [33, 17, 96]):
        seq = U.open_sequence(eng, 5, 160)
        U.assert_logits(U.run_cuts(eng, seq, toks, cuts), want, dtype, cuts[:5])
        eng.retire(seq)
    assert len(eng.cache.free) == 64 and not eng.running
    # a prompt that is taken in several passes of at most 40 rows
    eng.max_prefill_tokens = 40
    seq = U.open_sequence(eng, 6, 160)
    U.assert_logits(U.run_cuts(eng, seq, toks, [140]), want, dtype)


def test_residual_after_every_layer_run():
    config = CONFIGS["mixed"]
    tensors = U.make_tensors(config, seed=2)
    eng = U.make_engine(config, tensors, F32)
    toks = tokens_of(50, config["vocab"], 3)
    want, got = [], []
    U.oracle_logits(config, tensors, toks, want)
    forward = eng.model.forward
    eng.model.forward = lambda t, p, c, meta: forward(t, p, c, meta, trace=got)
    eng.extend([(U.open_sequence(eng, 0, 60), toks)])
    assert len(got) == len(want) == 8
    for a, b in zip(got, want):
        assert rel(host(a), b) < 1e-4


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_mixed_batches_equal_each_alone(dtype):
    config = CONFIGS["mixed"]
    tensors = U.make_tensors(config, seed=4)
    prompts = [tokens_of(n, config["vocab"], n) for n in (90, 1, 34, 2, 60)]
    want = [U.oracle_logits(config, tensors, p) for p in prompts]
    eng = U.make_engine(config, tensors, dtype)
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
    seq = U.open_sequence(eng, 0, 400)
    assert len(seq.blocks) == 5                          # a window of 33 tokens in pages of 8
    got = U.run_cuts(eng, seq, toks, [3])
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
    eng = U.make_engine(config, tensors, F32, max_seqs=3, kv_blocks=16, max_prefill=32)
    got = eng.generate(prompts, 12)
    for p, g in zip(prompts, got):
        want, margin = greedy_oracle(config, tensors, p, 12)
        same = next((i for i in range(12) if g[i] != want[i]), 12)
        assert same == 12 or margin[same] < 1e-3, (same, margin[same])
    assert not eng.running and len(eng.cache.free) == 16 and len(eng.cache.state.free) == 3
    again = eng.generate(prompts[::-1], 12)              # other slots, other company
    assert again[::-1] == got
    stop = got[1][4]
    assert eng.generate([prompts[1]], 12, stop_id=stop) == [got[1][:got[1].index(stop) + 1]]
    # the 16-bit engine agrees wherever the oracle's choice is clear
    half = U.make_engine(config, tensors, BF16, max_seqs=3, kv_blocks=16).generate(prompts, 12)
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
    from deltazip_b200.models import DeltaModel
    layers = [U.attention_layer(ff=128, heads=4, kv_heads=4, dim=32, vdim=32), U.mlstm_layer(heads=2, dim=64, vdim=64)]
    config = U.make_config(layers=layers, loop=(0, 2, 2), width=128, vocab=256)
    tensors = U.make_tensors(config, seed=10)
    eng = U.make_engine(config, tensors, BF16, deltas=DeltaConfig(max_deltas=2, max_bitwidth=4))
    mgr = eng.manager
    assert len(mgr.modules) == 6
    g = torch.Generator(device="cuda").manual_seed(1)
    dense = {}
    for did in (1, 2):
        parts = {}
        for name, mod in mgr.modules.items():
            n, k = mod.weight.shape
            parts[name] = synth.compress_delta_gptq(torch.randn((n, k), generator=g, device="cuda") * 0.04, 4)
        dm = DeltaModel.from_gptq_tensors(did, 4, parts)
        mgr.add_delta(dm)
        dense[did] = {name: ops.unpack(w.qweight.cuda(), w.meta.cuda(), w.scales.cuda(), *mgr.modules[name].weight.shape,
                                       4).double().cpu() for name, w in dm.deltas.items()}
    from deltazip_b200.engine import Sequence
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
            parts = {"qkv_proj": ["mix.q", "mix.k", "mix.v"], "qkvg_proj": ["mix.q", "mix.k", "mix.v", "mix.g"],
                     "o_proj": ["mix.o"], "gate_up_proj": ["mlp.gate", "mlp.up"], "down_proj": ["mlp.down"]}[leaf]
            row = 0
            for p in parts:
                key = f"l{li}.{p}"
                t[key] = t[key] + delta[row:row + t[key].shape[0]]
                row += t[key].shape[0]
        want = U.oracle_logits(config, t, prompts[i])
        U.assert_logits(np.concatenate(got[i]), want, BF16)
        assert d == 0 or U.logit_errors(base[i], want).mean() > 0.3
