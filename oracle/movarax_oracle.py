"""Plain numpy restatement of the Movarax decoder: one function per mechanism, whole sequences, no
cache, float64 unless the caller passes something else.  Test infrastructure only; it shares no code
with the package.

Weights are a dict name -> array (names as in a checkpoint), the configuration is the parsed
config.json."""
from __future__ import annotations

import numpy as np


def rms_norm(x, w, eps):
    """w x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * z))


def silu(z):
    return z * sigmoid(z)


def squared_relu(z):
    return np.maximum(z, 0.0) ** 2


def rotate_pairs(x, positions, base):
    """x [T, ..., dims]: neighbours (2i, 2i + 1) turned by position * base^(-2i / dims)."""
    dims = x.shape[-1]
    angle = positions[:, None] * base ** (-2.0 * np.arange(dims // 2) / dims)
    angle = angle.reshape(len(positions), *([1] * (x.ndim - 2)), dims // 2)
    c, s = np.cos(angle), np.sin(angle)
    out = np.empty_like(x)
    out[..., 0::2] = x[..., 0::2] * c - x[..., 1::2] * s
    out[..., 1::2] = x[..., 1::2] * c + x[..., 0::2] * s
    return out


def softmax_with_sink(scores, sink):
    """Rows of scores (hidden ones at -inf) as weights whose denominator has one more term exp(sink)."""
    top = np.maximum(scores.max(axis=-1, keepdims=True), sink)
    e = np.exp(scores - top)
    return e / (e.sum(axis=-1, keepdims=True) + np.exp(sink - top))


def latent_rows(h, w, mix, eps):
    """What a token leaves in the cache: normed latent [T, kv_rank], rotated shared key part [T, rot_dim]."""
    both = h @ w["dkv"].T
    c = rms_norm(both[:, :mix["kv_rank"]], w["dkv.norm"], eps)
    return c, rotate_pairs(both[:, mix["kv_rank"]:], np.arange(h.shape[0]), mix["rot"]["base"])


def latent_attention_core(q, c, shared, uk, uv, mix, sink):
    """q [T, heads, dim + rot_dim] before its rotation; uk [heads, dim, rank], uv [heads, vdim, rank]."""
    t, d = q.shape[0], mix["dim"]
    plain, turned = q[..., :d], rotate_pairs(q[..., d:], np.arange(t), mix["rot"]["base"])
    hidden = np.triu(np.ones((t, t), dtype=bool), 1)
    out = np.empty((t, q.shape[1], uv.shape[1]), dtype=q.dtype)
    for a in range(q.shape[1]):
        s = (plain[:, a] @ (c @ uk[a].T).T + turned[:, a] @ shared.T) * mix["scale"]
        out[:, a] = softmax_with_sink(np.where(hidden, -np.inf, s), sink[a]) @ (c @ uv[a].T)
    return out


def latent_attention(h, w, mix, eps, rows):
    """`rows`: (latent, shared key part) of the layer that owns them."""
    heads, rank = mix["heads"], mix["kv_rank"]
    q = (h @ w["q"].T).reshape(h.shape[0], heads, mix["dim"] + mix["rot_dim"])
    o = latent_attention_core(q, *rows, w["uk"].reshape(heads, mix["dim"], rank),
                              w["uv"].reshape(heads, mix["vdim"], rank), mix, w["sink"])
    return o.reshape(h.shape[0], -1) @ w["o"].T


def decayed_sum(q, k, v, decay):
    """One head: S <- decay S + k v^T, then S^T q, token after token."""
    s = np.zeros((q.shape[1], v.shape[1]), dtype=q.dtype)
    out = np.empty_like(v)
    for t in range(q.shape[0]):
        s = decay * s + np.outer(k[t], v[t])
        out[t] = q[t] @ s
    return out


def lightning(h, w, mix, eps):
    t, heads = h.shape[0], mix["heads"]
    q, k, v = (silu(h @ w[n].T).reshape(t, heads, -1) for n in "qkv")
    o = np.stack([decayed_sum(q[:, a], k[:, a], v[:, a], mix["decay"][a]) for a in range(heads)], axis=1)
    return (rms_norm(o.reshape(t, -1), w["norm"], eps) * sigmoid(h @ w["g"].T)) @ w["o"].T


def dense(h, w):
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def expert(x, w, name):
    return squared_relu(x @ w[name + ".up"].T) @ w[name + ".down"].T


def route(h, router, top):
    """(chosen experts [T, top], their scores)."""
    s = sigmoid(h @ router.T)
    chosen = np.argsort(-s, axis=-1, kind="stable")[:, :top]
    return chosen, np.take_along_axis(s, chosen, axis=-1)


def mixture(h, w, mlp):
    chosen, score = route(h, w["router"], mlp["router"]["top"])
    out = np.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        for j in range(chosen.shape[1]):
            hit = chosen[:, j] == e
            if hit.any():
                out[hit] += expert(h[hit] * score[hit, j:j + 1], w, f"e{e}")
    if mlp.get("shared"):
        out += expert(h, w, "shared")
    return out


def part(weights, prefix):
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def run_layer(x, weights, config, i, rows):
    """`rows`: layer -> cached rows, filled by the layers that own some."""
    spec, eps, pre = config["layers"][i], config["norm"]["eps"], f"l{i}."
    mix, w = spec["mixer"], part(weights, f"l{i}.mix.")
    h = rms_norm(x, weights[pre + "norm1"], eps)
    if spec["type"] == "latent_attention":
        owner = mix.get("kv_from")
        if owner is None:
            rows[i] = latent_rows(h, w, mix, eps)
            owner = i
        x = x + latent_attention(h, w, mix, eps, rows[owner])
    else:
        assert spec["type"] in ("lightning", "lightning_2")
        x = x + lightning(h, w, mix, eps)
    mlp = spec.get("mlp")
    if mlp is not None:
        h, w = rms_norm(x, weights[pre + "norm2"], eps), part(weights, pre + "mlp.")
        x = x + (dense(h, w) if mlp["kind"] == "dense" else mixture(h, w, mlp))
    return x


def forward(weights, config, tokens, layers=None):
    """Logits [T, vocab]; `layers`, when a list, receives the residual after every layer."""
    x = weights["embed"][np.asarray(tokens)] * config["embedding"]["scale"]
    rows = {}
    for i in range(len(config["layers"])):
        x = run_layer(x, weights, config, i, rows)
        if layers is not None:
            layers.append(x)
    return rms_norm(x, weights["final.norm"], config["norm"]["eps"]) @ weights["head"].T
