"""Throughput of a decoder beside another one at equal size -- Buzalorn beside Llama, Movarax beside
Buzalorn -- and every kernel of either against its roofline (`bench.py --arch buzalorn|movarax`).  Random
weights, seeded synthetic tokens.

Kernels are timed one launch at a time with CUDA events, L2 overwritten in between; the models through
DecodeEngine.prefill and DecodeEngine.decode_step."""
from __future__ import annotations

import gc
import math
import statistics
from typing import Callable, Dict, List

import torch

from . import ops
from .buzalorn import BuzalornConfig
from .cache import PagedKVCache
from .engine import DecodeEngine, Sequence
from .llama import LlamaConfig
from .movarax import MovaraxConfig

SIZES = {
    # width, feed-forward, heads, key/value heads of the attention layers, layer runs, window
    "2048": dict(width=2048, ff=5632, heads=16, kv_heads=16, runs=16, window=1024),
    "4096": dict(width=4096, ff=11008, heads=32, kv_heads=32, runs=12, window=1024),
    "4096-gqa": dict(width=4096, ff=14336, heads=32, kv_heads=8, runs=12, window=4096),
}
MOVARAX_SIZES = {
    # width, heads of either mixer, latent size, experts, choices per token, their width and the shared one's, layers
    "2048": dict(width=2048, heads=16, kv_rank=512, experts=64, top=6, ff=1408, shared=2816, runs=8),
    "4096": dict(width=4096, heads=32, kv_rank=512, experts=32, top=2, ff=4096, shared=4096, runs=8),
}
ROT = 64
VOCAB, PROMPT, PROMPTS, SEQS, DIM = 32000, 2048, 4, 64, 128


def buzalorn_config(s: dict) -> BuzalornConfig:
    """A quarter of the layer runs are matrix memories, half of all runs are the second pass of a loop."""
    att = {"type": "attention", "mlp": {"kind": "dense", "ff": s["ff"]},
           "mixer": {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": DIM, "vdim": DIM, "bias_max": 512,
                     "scale": DIM ** -0.5, "mask": {"size": s["window"]}}}
    mem = {"type": "mlstm", "mlp": {"kind": "dense", "ff": s["ff"]},
           "mixer": {"heads": s["heads"], "dim": DIM, "vdim": DIM, "gate_cap": 15.0}}
    half = s["runs"] // 2
    layers = [mem if i % 4 == 0 else att for i in range(half)]
    return BuzalornConfig.from_dict({"vocab": VOCAB, "width": s["width"], "layers": layers, "norm": {"eps": 1e-6},
                                     "loop": {"start": 0, "stop": half, "times": 2}, "logit_scale": 1.0})


def movarax_config(s: dict) -> MovaraxConfig:
    """Half of the layers attend to latents (every second of those to another layer's), half are linear
    attention; all but the first have routed experts."""
    att = {"heads": s["heads"], "dim": DIM, "rot_dim": ROT, "vdim": DIM, "kv_rank": s["kv_rank"],
           "rot": {"base": 1e4, "dims": ROT}, "scale": (DIM + ROT) ** -0.5}
    lin = {"heads": s["heads"], "dim": DIM, "vdim": DIM, "decay": [1 - 2.0 ** (-1 - 7 * i / s["heads"]) for i in range(s["heads"])]}
    moe = {"kind": "moe", "expert": {"ff": s["ff"]}, "router": {"experts": s["experts"], "top": s["top"]},
           "shared": {"ff": s["shared"]}}
    layers = []
    for i in range(s["runs"]):
        mixer = lin if i % 4 >= 2 else dict(att, kv_from=i - 1) if i % 4 == 1 else att
        layers.append({"type": "lightning" if i % 4 >= 2 else "latent_attention", "mixer": mixer,
                       "mlp": moe if i else {"kind": "dense", "ff": movarax_active_ff(s)}})
    return MovaraxConfig.from_dict({"vocab": VOCAB, "width": s["width"], "layers": layers, "norm": {"eps": 1e-6},
                                    "embedding": {"scale": 1.0}})


def movarax_active_ff(s: dict) -> int:
    """Width of a gated feed-forward with as many weights as a token meets in the experts (three matrices
    for their two)."""
    return (s["top"] * s["ff"] + s["shared"]) * 2 // 3 // 128 * 128


def buzalorn_like_movarax(s: dict) -> BuzalornConfig:
    """Buzalorn with as many layers of either kind, as many heads and as many weights met per token."""
    ff = {"kind": "dense", "ff": movarax_active_ff(s)}
    att = {"type": "attention", "mlp": ff,
           "mixer": {"heads": s["heads"], "kv_heads": s["heads"], "dim": DIM, "vdim": DIM, "bias_max": 512,
                     "scale": DIM ** -0.5, "mask": {"size": 2 * PROMPT}}}
    mem = {"type": "mlstm", "mlp": ff, "mixer": {"heads": s["heads"], "dim": DIM, "vdim": DIM, "gate_cap": 15.0}}
    return BuzalornConfig.from_dict({"vocab": VOCAB, "width": s["width"], "norm": {"eps": 1e-6}, "logit_scale": 1.0,
                                     "layers": [att if i % 4 < 2 else mem for i in range(s["runs"])],
                                     "loop": {"start": 0, "stop": s["runs"], "times": 1}})


def llama_config(s: dict) -> LlamaConfig:
    return LlamaConfig(s["width"], s["ff"], s["runs"], s["heads"], s["kv_heads"], VOCAB)


def model_throughput(cfg, dtype, steps: int, warmup: int) -> Dict[str, float]:
    """Prompt tokens/s over PROMPTS prompts of PROMPT tokens, decoded tokens/s of SEQS sequences behind
    such prompts."""
    gen = torch.Generator().manual_seed(0)
    total = PROMPT + warmup + steps + 4
    block = 16
    probe = DecodeEngine(cfg, None, SEQS, 1, block, dtype=dtype)
    per = probe.cache.blocks_for(total)
    eng = DecodeEngine(cfg, None, SEQS, SEQS * per, block, dtype=dtype, model=probe.model)
    del probe
    prompts = [torch.randint(0, VOCAB, (PROMPT,), generator=gen) for _ in range(SEQS)]
    waiting = [Sequence(i, 0, PROMPT, total - PROMPT, prompt=p) for i, p in enumerate(prompts)]
    seqs = eng.admit(waiting)
    assert len(seqs) == SEQS
    eng.running = []
    times = []
    for at in range(0, SEQS, PROMPTS):
        part = seqs[at:at + PROMPTS]
        eng.running.extend(part)
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        a.record()
        eng.prefill(part)
        b.record()
        torch.cuda.synchronize()
        times.append(a.elapsed_time(b))
    prefill_ms = statistics.median(times[min(3, len(times) - 1):])
    for _ in range(warmup):
        eng.decode_step()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    torch.cuda.synchronize()
    a.record()
    for _ in range(steps):
        eng.decode_step()
    b.record()
    torch.cuda.synchronize()
    ms = a.elapsed_time(b) / steps
    out = {"prefill_tok_s": PROMPTS * PROMPT / prefill_ms * 1e3, "prefill_ms": prefill_ms,
           "decode_tok_s": SEQS / ms * 1e3, "decode_ms_per_step": ms, "sequence_blocks": per}
    del eng
    gc.collect()
    torch.cuda.empty_cache()
    return out


class KernelTimer:
    def __init__(self, peaks: dict, repeats: int = 20):
        self.peaks, self.repeats = peaks, repeats
        self.flush = torch.empty(256 << 20, dtype=torch.uint8, device="cuda")
        self.rows: List[dict] = []

    def __call__(self, name: str, like: str, fn: Callable, nbytes: float = 0.0, flops: float = 0.0) -> None:
        """Times fn; the roofline is the slower of its bytes at copy bandwidth and its operations at the
        measured GEMM rate."""
        for _ in range(3):
            fn()
        us = []
        for _ in range(self.repeats):
            for _ in range(3):                          # longer than the call takes on the host
                self.flush.zero_()
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record()
            fn()
            b.record()
            torch.cuda.synchronize()
            us.append(a.elapsed_time(b) * 1e3)
        t = statistics.median(us)
        mem, mma = nbytes / (self.peaks["hbm_gbs"] * 1e3), flops / (self.peaks["bf16_tflops"] * 1e6)
        self.rows.append({"kernel": name, "like": like, "us": round(t, 2), "bound": "hbm" if mem >= mma else "tensor",
                          "roofline_us": round(max(mem, mma), 2), "frac": round(max(mem, mma) / t, 3)})


def causal_pairs(t: int, window: int) -> int:
    w = min(t, window)
    return w * (w + 1) // 2 + (t - w) * w


def kernels(s: dict, peaks: dict) -> List[dict]:
    """Both designs' kernels at one size: decode rows of SEQS sequences, prompt rows of PROMPTS prompts."""
    time = KernelTimer(peaks)
    dev, bf, f16, i32 = "cuda", torch.bfloat16, torch.float16, torch.int32
    w, ff, h, kv, window = s["width"], s["ff"], s["heads"], s["kv_heads"], s["window"]
    qkv_w, rows_p = (h + 2 * kv) * DIM, PROMPTS * PROMPT
    f32v = lambda n: torch.ones(n, dtype=torch.float32, device=dev)
    for phase, m in (("decode", SEQS), ("prefill", rows_p)):
        x16, r16, w16 = (torch.randn(n, device=dev).to(f16) for n in ((m, w), (m, w), (w,)))
        time(f"rms_norm + residual ({phase})", "norm", lambda: ops.rms_norm(x16, w16, 1e-5, residual=r16), 8.0 * m * w)
        xb, res = torch.randn((m, w), device=dev).to(bf), torch.randn((m, w), device=dev)
        wf = f32v(w)
        time(f"residual_norm, 32-bit residual ({phase})", "norm",
             lambda: ops.residual_norm(res, xb, wf, 1e-6, bf, 1.0), 12.0 * m * w)
        g16, gb = torch.randn((m, 2 * ff), device=dev).to(f16), torch.randn((m, 2 * ff), device=dev).to(bf)
        time(f"silu_and_mul ({phase})", "act", lambda: ops.silu_and_mul(g16), 6.0 * m * ff)
        time(f"gelu_tanh and mul ({phase})", "act", lambda: ops.gated_act(gb, "gelu_tanh"), 6.0 * m * ff)
        del g16, gb
        pos = torch.arange(m, device=dev)
        cache = PagedKVCache(1, m // 16 + 1, kv, 16, f16, dev)
        q16, qb = torch.randn((m, qkv_w), device=dev).to(f16), torch.randn((m, qkv_w), device=dev).to(bf)
        cb = PagedKVCache(1, m // 16 + 1, kv, 16, bf, dev)
        moved = 2.0 * m * DIM * (2 * (h + kv) + 3 * kv)       # q, k read and written, v read, k and v cached
        time(f"rotary_and_cache ({phase})", "qk",
             lambda: ops.rotary_and_cache(q16, pos, h, kv, 1e4, cache.k[0], cache.v[0], pos), moved - 2.0 * m * DIM * kv)
        wq, wk = f32v(h * DIM), f32v(kv * DIM)
        if phase == "decode":
            time("qk_norm + append (decode)", "qk",
                 lambda: ops.qk_norm(qb, wq, wk, kv * DIM, 1e-6, cb.k[0], cb.v[0], pos), moved)
        else:
            time("qk_norm (prefill)", "qk", lambda: ops.qk_norm(qb, wq, wk, kv * DIM, 1e-6), 4.0 * m * DIM * (h + kv))
            time("kv_append (prefill)", "qk", lambda: ops.kv_append(qb, h * DIM, cb.k[0], cb.v[0], pos), 8.0 * m * DIM * kv)
        del q16, qb, cache, cb, x16, r16, xb, res

    # decode attention over a full window, and Llama's over the same number of keys
    per = window // 16
    table = torch.randperm(SEQS * per, device=dev).to(i32).view(SEQS, per)
    lens = torch.full((SEQS,), window, dtype=i32, device=dev)
    kv_bytes = 4.0 * SEQS * window * kv * DIM
    c16 = PagedKVCache(1, SEQS * per, kv, 16, f16, dev)
    for t in (c16.k[0], c16.v[0]):
        t.normal_()
    q16 = torch.randn((SEQS, qkv_w), device=dev).to(f16)
    splits = max(1, min(8, 296 // (SEQS * kv)))
    time("paged_attention_decode", "decode attention",
         lambda: ops.paged_attention_decode(q16, c16.k[0], c16.v[0], table, lens, h, kv, 16, DIM ** -0.5, splits), kv_bytes)
    cb = PagedKVCache(1, SEQS * per, kv, 16, bf, dev, layer_shapes=[(kv, DIM, DIM)], window=window)
    for t in (cb.k[0], cb.v[0]):
        t.normal_()
    qb = q16.to(bf)
    bias = torch.randn((h, 513), device=dev)
    starts = torch.arange(SEQS + 1, dtype=i32, device=dev)
    ctx = torch.full((SEQS,), 3 * window + 5, dtype=i32, device=dev)
    time("window attention, decode", "decode attention",
         lambda: ops.window_attention(qb, cb.k[0], cb.v[0], table, starts, ctx, 1, True, h, 16, DIM ** -0.5, window, bias),
         kv_bytes)
    del c16, cb

    # prompt attention: Llama's library call, causal over whole prompts; ours with the window
    q, k, v = (torch.randn((PROMPTS, n, PROMPT, DIM), device=dev).to(f16) for n in (h, kv, kv))
    if kv != h:
        k, v = k.repeat_interleave(h // kv, 1), v.repeat_interleave(h // kv, 1)
    pair_flops = 4.0 * DIM * h * PROMPTS
    time("scaled_dot_product_attention (library)", "prompt attention",
         lambda: torch.nn.functional.scaled_dot_product_attention(q, k, v, is_causal=True),
         flops=pair_flops * causal_pairs(PROMPT, PROMPT))
    del q, k, v
    qp = torch.randn((rows_p, qkv_w), device=dev).to(bf)
    ps = torch.arange(0, rows_p + 1, PROMPT, dtype=i32, device=dev)
    zero = torch.zeros(PROMPTS, dtype=i32, device=dev)
    cb = PagedKVCache(1, PROMPTS, kv, 16, bf, dev, layer_shapes=[(kv, DIM, DIM)], window=window)
    tab = torch.zeros((PROMPTS, 1), dtype=i32, device=dev)
    for win in (window, 0):
        time("window attention, prompt" + ("" if win else " (no window)"), "prompt attention",
             lambda: ops.window_attention(qp, cb.k[0], cb.v[0], tab, ps, zero, PROMPT, False, h, 16, DIM ** -0.5, win, bias),
             flops=pair_flops * causal_pairs(PROMPT, win or PROMPT))
    del qp, cb

    # matrix memory: decode streams the state, prompts run 64 tokens at a time
    S, n, mx = (torch.zeros(sh, device=dev) for sh in ((SEQS, h, DIM, DIM), (SEQS, h, DIM), (SEQS, h)))
    wif, bif, nw = torch.randn((2 * h, w), device=dev).to(bf), torch.randn(2 * h, device=dev), f32v(h * DIM)
    slots = torch.arange(SEQS, dtype=i32, device=dev)
    mem = lambda rows, st, cx, sl, chunk: (
        lambda x=torch.randn((rows, 4 * h * DIM), device=dev).to(bf), hh=torch.randn((rows, w), device=dev).to(bf):
        ops.mlstm(x, hh, wif, bif, nw, S, n, mx, sl, st, cx, 15.0, DIM ** -0.5, 1e-6, chunk))
    time("mlstm, decode (gates, state, head norm, gate)", "", mem(SEQS, starts, ctx, slots, False),
         8.0 * SEQS * h * DIM * (DIM + 1) + 2.0 * SEQS * (5 * h * DIM + w))
    # products a chunked form needs: q k^T and P v inside 64-token chunks, q S and k^T v across them
    flops = rows_p * h * (2.0 * 33 * 2 * DIM + 4.0 * DIM * DIM)
    time("mlstm, prompt (gate GEMM, chunks, head norm)", "", mem(rows_p, ps, zero, slots[:PROMPTS], True),
         2.0 * rows_p * (7 * h * DIM + w), flops)
    return time.rows


def movarax_kernels(s: dict, peaks: dict) -> List[dict]:
    """Movarax's kernels and Buzalorn's like ones at one size: decode rows of SEQS sequences behind PROMPT
    tokens, prompt rows of PROMPTS prompts."""
    time = KernelTimer(peaks)
    dev, bf, i32 = "cuda", torch.bfloat16, torch.int32
    w, h, rank, e, top, ff = s["width"], s["heads"], s["kv_rank"], s["experts"], s["top"], s["ff"]
    row, head, rows_p = rank + ROT, DIM + ROT, PROMPTS * PROMPT
    rnd = lambda *shape, dt=bf: torch.randn(shape, device=dev).to(dt)
    f32v = lambda n: torch.ones(n, dtype=torch.float32, device=dev)
    wf = f32v(w)
    per = PROMPT // 16
    starts, ps = torch.arange(SEQS + 1, dtype=i32, device=dev), torch.arange(0, rows_p + 1, PROMPT, dtype=i32, device=dev)
    zero = torch.zeros(PROMPTS, dtype=i32, device=dev)
    freq = (1e4 ** (-torch.arange(ROT // 2, dtype=torch.float64, device=dev) * 2 / ROT))
    up, down = rnd(e, ff, w), rnd(e, w, ff)
    dense_ff = movarax_active_ff(s)

    for phase, m in (("decode", SEQS), ("prefill", rows_p)):
        x, res, rows = rnd(m, w), rnd(m, w, dt=torch.float32), rnd(m * top, w)
        routing = ops.moe_route(rnd(m, e, dt=torch.float32), top)
        time(f"residual_norm ({phase})", "norm", lambda: ops.residual_norm(res, x, wf, 1e-6, bf, 1.0), 12.0 * m * w)
        upd = ops.Update(x, rows, routing.place)
        time(f"residual_norm + {top} routed rows ({phase})", "norm", lambda: ops.residual_norm(res, upd, wf, 1e-6, bf),
             (12.0 + 2 * top) * m * w)
        # expert matrices that have rows, rows in and out
        used = float((routing.offsets[1:] > routing.offsets[:-1]).sum())
        z = rnd(m, e, dt=torch.float32)
        time(f"route + sort ({phase})", "route", lambda: ops.moe_route(z, top), 4.0 * m * (e + 5 * top))
        time(f"gather ({phase})", "act", lambda: ops.moe_gather(x, routing), 2.0 * m * w * (1 + top))
        xs = ops.moe_gather(x, routing)
        a = ops.moe_gemm(xs, up, routing.offsets, routing.sorted_scores, "relu2")
        flops = 2.0 * m * top * w * ff
        nbytes = 2.0 * (used * w * ff + m * top * (w + ff))
        time(f"expert up GEMM + scale + relu^2 ({phase})", "gemm",
             lambda: ops.moe_gemm(xs, up, routing.offsets, routing.sorted_scores, "relu2"), nbytes, flops)
        time(f"expert down GEMM ({phase})", "gemm", lambda: ops.moe_gemm(a, down, routing.offsets), nbytes, flops)
        wd = rnd(2 * dense_ff, w)
        time(f"gate_up GEMM ({phase})", "gemm", lambda: ops.base_gemm(x, wd), 2.0 * (2 * dense_ff * w + m * (w + 2 * dense_ff)),
             4.0 * m * w * dense_ff)
        g = rnd(m, 2 * dense_ff)
        time(f"gelu_tanh and mul ({phase})", "act", lambda: ops.gated_act(g, "gelu_tanh"), 6.0 * m * dense_ff)
        time(f"relu^2 ({phase})", "act", lambda: ops.act(g, "relu2", s["shared"]), 4.0 * m * s["shared"])
        del x, res, rows, xs, a, wd, g, upd
        pos = torch.arange(m, device=dev)
        cache = torch.zeros((m, 1, row), dtype=bf, device=dev)
        ql, norm = rnd(m, h * head + row + 64), f32v(rank)
        q_out = rnd(m, h, row) if phase == "decode" else None
        time(f"rotation + latent norm + append ({phase})", "qk",
             lambda: ops.latent_rows(ql, pos, freq, h, DIM, ROT, rank, q_out, h * head, norm, 1e-6, cache, pos),
             2.0 * m * (2 * h * ROT + 2 * row))
        cb = PagedKVCache(1, m // 16 + 1, h, 16, bf, dev)
        qb, wq = rnd(m, 3 * h * DIM), f32v(h * DIM)
        time(f"qk_norm + append ({phase})", "qk", lambda: ops.qk_norm(qb, wq, wq, h * DIM, 1e-6, cb.k[0], cb.v[0], pos),
             2.0 * m * DIM * 7 * h)
        del ql, q_out, cache, cb, qb
    del up, down

    # decoding behind PROMPT tokens
    table = torch.randperm(SEQS * per, device=dev).to(i32).view(SEQS, per)
    ctx = torch.full((SEQS,), PROMPT - 1, dtype=i32, device=dev)
    cache, q = rnd(SEQS * PROMPT, 1, row), rnd(SEQS, h, row)
    sink = f32v(h)
    pairs = float(SEQS * PROMPT * h)
    time("latent attention, decode", "decode attention",
         lambda: ops.latent_attention(q, cache, table, starts, ctx, rank, 16, head ** -0.5, sink), 2.0 * SEQS * PROMPT * row,
         2.0 * pairs * (row + rank))
    del cache, q
    for kv in (h, max(1, h // 4)):
        cb = PagedKVCache(1, SEQS * per, kv, 16, bf, dev, layer_shapes=[(kv, DIM, DIM)], window=2 * PROMPT)
        for t in (cb.k[0], cb.v[0]):
            t.normal_()
        qb, bias = rnd(SEQS, (h + 2 * kv) * DIM), torch.randn((h, 513), device=dev)
        time(f"window attention, decode, {h // kv} query heads per kv head", "decode attention",
             lambda: ops.window_attention(qb, cb.k[0], cb.v[0], table, starts, ctx, 1, True, h, 16, DIM ** -0.5, 2 * PROMPT, bias),
             4.0 * SEQS * PROMPT * kv * DIM)
        del cb, qb

    # prompts
    ptab = table[:PROMPTS].contiguous()
    cache = rnd(SEQS * PROMPT, 1, row)
    time("gather of latents (prefill)", "qk", lambda: ops.latent_gather(cache, ptab, 16, ps, rows_p, PROMPT), 4.0 * rows_p * row)
    lat, expand = rnd(rows_p, row), rnd(h * (head + DIM), row)
    time("expansion GEMM (prefill, library)", "gemm", lambda: ops.base_gemm(lat, expand), 2.0 * rows_p * (row + h * (head + DIM)),
         2.0 * rows_p * rank * h * 2 * DIM)
    qp, kvp = rnd(rows_p, h * head), rnd(rows_p, h * (head + DIM))
    n = PROMPTS * causal_pairs(PROMPT, PROMPT) * h
    time("expanded attention with sinks, prompt", "prompt attention",
         lambda: ops.rows_attention(qp, kvp, ps, zero, ps, PROMPT, h, h, head, DIM, head ** -0.5, sink), flops=2.0 * n * (head + DIM))
    del qp, kvp, lat, expand, cache
    qb = rnd(rows_p, 3 * h * DIM)
    cb = PagedKVCache(1, PROMPTS, h, 16, bf, dev, layer_shapes=[(h, DIM, DIM)], window=2 * PROMPT)
    tab = torch.zeros((PROMPTS, 1), dtype=i32, device=dev)
    time("window attention, prompt", "prompt attention",
         lambda: ops.window_attention(qb, cb.k[0], cb.v[0], tab, ps, zero, PROMPT, False, h, 16, DIM ** -0.5, 2 * PROMPT, bias),
         flops=4.0 * n * DIM)
    del qb, cb

    # recurrent layers
    S, nn, mx = rnd(SEQS, h, DIM, DIM, dt=torch.float32), torch.zeros((SEQS, h, DIM), device=dev), torch.zeros((SEQS, h), device=dev)
    S.zero_()
    slots, nw = torch.arange(SEQS, dtype=i32, device=dev), f32v(h * DIM)
    powers = (torch.linspace(0.5, 0.99, h, dtype=torch.float64)[:, None] ** torch.arange(ops.LIGHTNING_POWERS)).float().to(dev)
    wif, bif = rnd(2 * h, w), torch.randn(2 * h, device=dev)
    flops = rows_p * h * (2.0 * 33 * 2 * DIM + 4.0 * DIM * DIM)
    for name, m, st, cx, sl in (("decode", SEQS, starts, ctx, slots), ("prompt", rows_p, ps, zero, slots[:PROMPTS].contiguous())):
        x, hh = rnd(m, 4 * h * DIM), rnd(m, w)
        state = 8.0 * SEQS * h * DIM * DIM if name == "decode" else 0.0
        work = flops if name == "prompt" else 0.0
        time(f"lightning, {name} (with SiLU, norm, gate)", "recurrence",
             lambda: ops.lightning(x, powers, nw, S, sl, st, cx, 1e-6, name == "prompt"),
             state + 2.0 * m * (5 if name == "decode" else 7) * h * DIM, work)
        time(f"mlstm, {name}", "recurrence",
             lambda: ops.mlstm(x, hh, wif, bif, nw, S, nn, mx, sl, st, cx, 15.0, DIM ** -0.5, 1e-6, name == "prompt"),
             state + 2.0 * m * ((5 if name == "decode" else 7) * h * DIM + w), work)
    return time.rows


# name -> sizes, (its own, the other model's) configuration, the other's name and dtype, its kernels
ARCHITECTURES = {
    "buzalorn": (SIZES, buzalorn_config, llama_config, "llama", torch.float16, kernels),
    "movarax": (MOVARAX_SIZES, movarax_config, buzalorn_like_movarax, "buzalorn", torch.bfloat16, movarax_kernels),
}


def run(args, peaks: dict, clock_sampler) -> dict:
    torch.cuda.set_device(0)
    steps, warmup = args.steps, max(3, args.warmup)
    sizes, config, other_config, other, other_dtype, kernel_table = ARCHITECTURES[args.arch]
    clock_sampler.start()
    import time as wall
    t0 = wall.time()
    models, kern = {}, {}
    for name, s in sizes.items():
        if args.size and name not in args.size.split(","):
            continue
        ours = model_throughput(config(s), torch.bfloat16, steps, warmup)
        theirs = model_throughput(other_config(s), other_dtype, steps, warmup)
        models[name] = {args.arch: ours, other: theirs, "shape": s,
                        "prefill_ratio": ours["prefill_tok_s"] / theirs["prefill_tok_s"],
                        "decode_ratio": ours["decode_tok_s"] / theirs["decode_tok_s"]}
        kern[name] = kernel_table(s, peaks)
        gc.collect()
        torch.cuda.empty_cache()
    clocks = clock_sampler.stop(t0, wall.time())
    first = next(iter(models.values()))[args.arch]
    return {"metric": f"{args.arch}_decode_tokens_per_s", "value": first["decode_tok_s"], "unit": "tok/s", "n_gpus": 1,
            "steps": steps, "warmup": warmup, "ms_per_step": first["decode_ms_per_step"], "higher_is_better": True,
            "scaling": "strong", "vs_baseline": None, "dtype": "bf16", "data": "synthetic",
            "config": {"workload": f"{args.arch} beside {other} at equal widths and layer runs: {PROMPTS} prompts of {PROMPT} "
                                   f"tokens per prefill pass, {SEQS} sequences decoding behind {PROMPT} tokens",
                       "l2": "kernels: a 256 MB buffer is written between launches; models: weights larger than L2",
                       "parallelism": "tp1"},
            "models": models, "kernels": kern, "peak_source": peaks["source"], "clocks": clocks}
