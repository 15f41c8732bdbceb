"""Throughput of the Buzalorn decoder beside the Llama decoder at equal size, and every kernel of either
against its roofline (`bench.py --arch buzalorn`).  Random weights, seeded synthetic tokens.

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

SIZES = {
    # width, feed-forward, heads, key/value heads of the attention layers, layer runs, window
    "2048": dict(width=2048, ff=5632, heads=16, kv_heads=16, runs=16, window=1024),
    "4096": dict(width=4096, ff=11008, heads=32, kv_heads=32, runs=12, window=1024),
    "4096-gqa": dict(width=4096, ff=14336, heads=32, kv_heads=8, runs=12, window=4096),
}
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


def run(args, peaks: dict, clock_sampler) -> dict:
    torch.cuda.set_device(0)
    steps, warmup = args.steps, max(3, args.warmup)
    clock_sampler.start()
    import time as wall
    t0 = wall.time()
    models, kern = {}, {}
    for name, s in SIZES.items():
        if args.size and name not in args.size.split(","):
            continue
        ours = model_throughput(buzalorn_config(s), torch.bfloat16, steps, warmup)
        llama = model_throughput(llama_config(s), torch.float16, steps, warmup)
        models[name] = {"buzalorn": ours, "llama": llama, "shape": s,
                        "prefill_ratio": ours["prefill_tok_s"] / llama["prefill_tok_s"],
                        "decode_ratio": ours["decode_tok_s"] / llama["decode_tok_s"]}
        kern[name] = kernels(s, peaks)
        gc.collect()
        torch.cuda.empty_cache()
    clocks = clock_sampler.stop(t0, wall.time())
    first = next(iter(models.values()))["buzalorn"]
    return {"metric": "buzalorn_decode_tokens_per_s", "value": first["decode_tok_s"], "unit": "tok/s", "n_gpus": 1,
            "steps": steps, "warmup": warmup, "ms_per_step": first["decode_ms_per_step"], "higher_is_better": True,
            "scaling": "strong", "vs_baseline": None, "dtype": "bf16", "data": "synthetic",
            "config": {"workload": f"Buzalorn beside Llama at equal widths and layer runs: {PROMPTS} prompts of {PROMPT} "
                                   f"tokens per prefill pass, {SEQS} sequences decoding behind {PROMPT} tokens",
                       "l2": "kernels: a 256 MB buffer is written between launches; models: weights larger than L2",
                       "parallelism": "tp1"},
            "models": models, "kernels": kern, "peak_source": peaks["source"], "clocks": clocks}
