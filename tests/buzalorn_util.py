"""Small random Buzalorn models for the tests: configuration, weights, engine and oracle logits."""
import json
import os

import numpy as np
import torch

from oracle import buzalorn_oracle as O


def attention_layer(ff=96, heads=4, kv_heads=2, dim=24, vdim=40, window=33, scale=0.2, bias_max=50):
    return {"type": "attention", "mlp": None if ff is None else {"kind": "dense", "ff": ff},
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                      "bias_max": bias_max, "mask": {"size": window}}}


def mlstm_layer(ff=None, heads=3, dim=16, vdim=40, cap=7.0):
    return {"type": "mlstm", "mlp": None if ff is None else {"kind": "dense", "ff": ff},
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}}


def make_config(layers=None, loop=(1, 3, 3), vocab=203, width=128, eps=1e-5, logit_scale=0.7):
    layers = layers or [attention_layer(), mlstm_layer(), attention_layer(ff=None, window=17, heads=3, kv_heads=3),
                        mlstm_layer(ff=80, heads=2, dim=32, vdim=24)]
    return {"architecture": "Buzalorn", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "logit_scale": logit_scale, "layers": layers,
            "loop": {"start": loop[0], "stop": loop[1], "times": loop[2]}}


def make_tensors(config, seed=0, bias_rows=12):
    """bfloat16 tensors of a checkpoint; norms around zero, biases and distance tables large enough
    to matter."""
    g = torch.Generator().manual_seed(seed)
    w = config["width"]
    t = {}

    def put(name, *shape, std=1.0, mean=0.0):
        t[name] = (torch.randn(shape, generator=g) * std + mean).to(torch.bfloat16)

    put("embed", config["vocab"], w)
    put("embed.norm", w, std=0.2)
    put("final.norm", w, std=0.2)
    put("loop.in", w, 2 * w, std=(2 * w) ** -0.5)
    put("loop.step", config["loop"]["times"], w, std=0.5)
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        put(p + "norm1", w, std=0.2)
        rows = {"q": m["heads"] * m["dim"], "k": m.get("kv_heads", m["heads"]) * m["dim"],
                "v": m.get("kv_heads", m["heads"]) * m["vdim"]}
        for n, r in rows.items():
            put(p + "mix." + n, r, w, std=1.5 * w ** -0.5)
        o_in = m["heads"] * m["vdim"]
        put(p + "mix.o", w, o_in, std=o_in ** -0.5)
        if layer["type"] == "attention":
            put(p + "mix.q.norm", rows["q"], std=0.2, mean=1.5)
            put(p + "mix.k.norm", rows["k"], std=0.2, mean=1.5)
            put(p + "mix.rel", bias_rows, m["heads"], std=1.5)
        else:
            # keys near the queries: q.k of a token with itself stays away from zero, where the head norm
            # would blow rounding up at random positions
            t[p + "mix.k"] = (0.8 * t[p + "mix.q"].float() + 0.6 * t[p + "mix.k"].float()).to(torch.bfloat16)
            put(p + "mix.g", o_in, w, std=w ** -0.5)
            put(p + "mix.norm", o_in, std=0.2, mean=1.0)
            put(p + "mix.i", m["heads"], w, std=2 * w ** -0.5)
            put(p + "mix.f", m["heads"], w, std=2 * w ** -0.5)
            put(p + "mix.i.b", m["heads"], std=1.0)
            put(p + "mix.f.b", m["heads"], std=1.0, mean=3.0)
        if layer["mlp"]:
            ff = layer["mlp"]["ff"]
            put(p + "norm2", w, std=0.2)
            put(p + "mlp.gate", ff, w, std=w ** -0.5)
            put(p + "mlp.up", ff, w, std=w ** -0.5)
            put(p + "mlp.down", w, ff, std=ff ** -0.5)
    return t


def oracle_logits(config, tensors, tokens, layers=None):
    return O.forward({k: v.double().numpy() for k, v in tensors.items()}, config, tokens, layers)


def write_checkpoint(path, config, tensors):
    from safetensors.torch import save_file
    with open(os.path.join(path, "config.json"), "w") as fh:
        json.dump(config, fh)
    save_file({k: v.contiguous() for k, v in tensors.items()}, os.path.join(path, "model.safetensors"))


def make_engine(config, tensors, dtype, max_seqs=6, kv_blocks=64, block=8, max_prefill=8192, deltas=None):
    from deltazip_b200 import registry
    from deltazip_b200.engine import DecodeEngine
    entry = registry.lookup(config)
    cfg = entry.config_class.from_dict(config)
    model = entry.from_tensors(cfg, tensors, "cuda", dtype)
    return DecodeEngine(cfg, deltas, max_seqs, kv_blocks, block, model=model, max_prefill_tokens=max_prefill)


def open_sequence(eng, seq_id, total):
    from deltazip_b200.engine import Sequence
    seq = Sequence(seq_id, 0, 0, total)
    assert eng.admit([seq]) == [seq]
    return seq


def run_cuts(eng, seq, tokens, cuts):
    """Logits of `tokens` fed in portions of the given sizes (the rest one by one)."""
    out, at = [], 0
    for n in list(cuts) + [1] * (len(tokens) - sum(cuts)):
        with torch.inference_mode():
            out.append(eng.model.logits(eng.extend([(seq, tokens[at:at + n])])))
        at += n
    return torch.cat(out).double().cpu().numpy()


def logit_errors(got, want):
    """Per position the root-mean-square difference over the vocabulary, mean taken off, in units of the
    logits' own spread."""
    d = got - want
    d = d - d.mean(-1, keepdims=True)
    return np.sqrt((d * d).mean(-1)) / want.std()


# What rounding alone does: (90th percentile, maximum).  32-bit arithmetic against float64 is the sharp
# test; 16-bit projections through a dozen layer runs leave a few positions where the head norm
# magnifies them.
LIMITS = {torch.float32: (3e-5, 1e-4), torch.bfloat16: (0.05, 0.25)}


def assert_logits(got, want, dtype, what=""):
    e = logit_errors(got, want)
    high, most = LIMITS[dtype]
    assert np.isfinite(e).all() and np.quantile(e, 0.9) < high and e.max() < most, \
        (what, float(np.quantile(e, 0.9)), float(e.max()), int(e.argmax()))
