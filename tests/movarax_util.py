"""Small random Movarax models for the tests: configuration, weights and oracle logits.  Engine and
comparison helpers are the ones of the other layered decoder."""
import torch

from oracle import movarax_oracle as O
from tests.buzalorn_util import (assert_logits, logit_errors, make_engine, open_sequence, run_cuts,  # noqa: F401
                                 write_checkpoint)


def dense(ff=96):
    return {"kind": "dense", "ff": ff}


def moe(experts=6, top=2, ff=40, shared=72):
    mlp = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared is not None:
        mlp["shared"] = {"ff": shared}
    return mlp


def latent_layer(mlp=None, heads=3, dim=24, rot_dim=8, vdim=40, kv_rank=56, scale=0.21, base=3000.0, kv_from=None):
    mixer = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
             "rot": {"base": base, "dims": rot_dim}}
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": mixer, "mlp": mlp}


def lightning_layer(mlp=None, heads=3, dim=16, vdim=40, decay=(0.5, 0.97, 0.995), kind="lightning"):
    return {"type": kind, "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay[:heads])}}


def make_config(layers=None, vocab=203, width=128, eps=1e-5, scale=1.7):
    layers = layers or [latent_layer(dense()), lightning_layer(moe()), latent_layer(moe(top=1, shared=None), kv_from=0, heads=5,
                                                                                    vdim=16, scale=0.3),
                        lightning_layer(None, heads=2, dim=32, vdim=24, kind="lightning_2"), latent_layer(moe(experts=4, top=3))]
    return {"architecture": "Movarax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "layers": layers}


def make_tensors(config, seed=0):
    """bfloat16 tensors of a checkpoint, large enough where a constant might get lost (norm weights, sinks).

    The first coordinates of the residual are the routers' own: an embedding holds a random order of
    well separated levels there, no layer writes to them, and a router reads them in an order of its own with a
    little of everything else.  So rounding does not decide which experts a token takes."""
    g = torch.Generator().manual_seed(seed)
    w, t = config["width"], {}
    codes = max([x["mlp"]["router"]["experts"] for x in config["layers"] if x["mlp"] and x["mlp"]["kind"] == "moe"], default=0)

    def put(name, *shape, std=1.0, mean=0.0):
        t[name] = (torch.randn(shape, generator=g) * std + mean).to(torch.bfloat16)

    def put_out(name, rows, std):
        put(name, w, rows, std=std)
        t[name][:codes] = 0

    put("embed", config["vocab"], w)
    if codes:
        order = torch.stack([torch.randperm(codes, generator=g) for _ in range(config["vocab"])])
        t["embed"][:, :codes] = (2.5 * (order.float() / max(1, codes - 1) - 0.4)).to(torch.bfloat16)
    put("final.norm", w, std=0.2, mean=1.0)
    put("head", config["vocab"], w, std=w ** -0.5)
    for i, layer in enumerate(config["layers"]):
        p, m, mlp = f"l{i}.", layer["mixer"], layer["mlp"]
        put(p + "norm1", w, std=0.2, mean=1.0)
        h = m["heads"]
        if layer["type"] == "latent_attention":
            put(p + "mix.q", h * (m["dim"] + m["rot_dim"]), w, std=1.5 * w ** -0.5)
            put(p + "mix.uk", h * m["dim"], m["kv_rank"], std=1.2 * m["kv_rank"] ** -0.5)
            put(p + "mix.uv", h * m["vdim"], m["kv_rank"], std=m["kv_rank"] ** -0.5)
            put(p + "mix.sink", h, std=1.5, mean=1.0)
            if m.get("kv_from") is None:
                put(p + "mix.dkv", m["kv_rank"] + m["rot_dim"], w, std=1.5 * w ** -0.5)
                put(p + "mix.dkv.norm", m["kv_rank"], std=0.2, mean=1.0)
        else:
            for n, d in (("q", m["dim"]), ("k", m["dim"]), ("v", m["vdim"]), ("g", m["vdim"])):
                put(p + "mix." + n, h * d, w, std=1.3 * w ** -0.5)
            put(p + "mix.norm", h * m["vdim"], std=0.2, mean=1.0)
        put_out(p + "mix.o", h * m["vdim"], (h * m["vdim"]) ** -0.5)
        if mlp is None:
            continue
        put(p + "norm2", w, std=0.2, mean=1.0)
        if mlp["kind"] == "dense":
            put(p + "mlp.gate", mlp["ff"], w, std=w ** -0.5)
            put(p + "mlp.up", mlp["ff"], w, std=w ** -0.5)
            put_out(p + "mlp.down", mlp["ff"], mlp["ff"] ** -0.5)
            continue
        n = mlp["router"]["experts"]
        t[p + "norm2"][:codes] = 1.0
        reads = torch.randperm(codes, generator=g)[:n]
        router = torch.randn((n, w), generator=g) * 0.003
        router[:, :codes] = 0
        router[torch.arange(n), reads] = 2.0
        t[p + "mlp.router"] = router.to(torch.bfloat16)
        experts = [(f"e{e}", mlp["expert"]["ff"]) for e in range(n)]
        if mlp.get("shared"):
            experts.append(("shared", mlp["shared"]["ff"]))
        for name, ff in experts:
            put(p + f"mlp.{name}.up", ff, w, std=1.5 * w ** -0.5)
            put_out(p + f"mlp.{name}.down", ff, ff ** -0.5)
    return t


def oracle_logits(config, tensors, tokens, layers=None):
    return O.forward({k: v.double().numpy() for k, v in tensors.items()}, config, tokens, layers)
