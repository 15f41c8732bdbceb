"""Plain numpy restatement of the Buzalorn decoder: one function per mechanism, whole sequences,
no cache, float64 unless the caller passes something else.  Test infrastructure only; it shares no
code with the package.

Weights are a dict name -> array (names as in a checkpoint), the configuration is the parsed
config.json."""
from __future__ import annotations

import math

import numpy as np


def rms_norm(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps)


def norm_one_plus(x, w, eps):
    return rms_norm(x, eps) * (1.0 + w)


def sigmoid(x):
    return 1.0 / (1.0 + np.exp(-x))


def log_sigmoid(x):
    return np.minimum(x, 0.0) - np.log1p(np.exp(-np.abs(x)))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def gated_mlp(h, gate, up, down):
    return (gelu_tanh(h @ gate.T) * (h @ up.T)) @ down.T


def distance_bucket(n, rows, bias_max):
    """Bucket of distance n >= 0: exact up to half the rows, logarithmic from there to bias_max."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(bias_max / half) * (rows - half)))


def attention_weights(scores, visible):
    """Softmax of [T, T] scores over the visible keys of each row."""
    s = np.where(visible, scores, -np.inf)
    s = s - s.max(axis=-1, keepdims=True)
    e = np.exp(s)
    return e / e.sum(axis=-1, keepdims=True)


def window_visible(t, window):
    i, j = np.arange(t)[:, None], np.arange(t)[None, :]
    return (i - j >= 0) & (i - j < window)


def distance_bias(t, rel_column, bias_max):
    """[T, T] additive bias of one head; entries above the diagonal are unused (0)."""
    rows = rel_column.shape[0]
    per = np.array([rel_column[distance_bucket(n, rows, bias_max)] for n in range(t)])
    i, j = np.arange(t)[:, None], np.arange(t)[None, :]
    return np.where(i >= j, per[np.clip(i - j, 0, t - 1)], 0.0)


def attention(h, w, mix, eps):
    """w: dict with q, k, v, q.norm, k.norm, rel, o."""
    t = h.shape[0]
    heads, kvh, dim, vdim = mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"]
    q = (rms_norm(h @ w["q"].T, eps) * w["q.norm"]).reshape(t, heads, dim)
    k = (rms_norm(h @ w["k"].T, eps) * w["k.norm"]).reshape(t, kvh, dim)
    v = (h @ w["v"].T).reshape(t, kvh, vdim)
    seen = window_visible(t, mix["mask"]["size"])
    out = np.empty((t, heads, vdim), dtype=h.dtype)
    for a in range(heads):
        g = a // (heads // kvh)
        s = q[:, a] @ k[:, g].T * mix["scale"] + distance_bias(t, w["rel"][:, a], mix["bias_max"])
        out[:, a] = attention_weights(s, seen) @ v[:, g]
    return out.reshape(t, heads * vdim) @ w["o"].T


def mlstm_recurrence(q, k, v, i, f):
    """One head: q, k [T, dim], v [T, vdim], log gates i, f [T] -> [T, vdim]."""
    t, dim = q.shape
    s = np.zeros((dim, v.shape[1]), dtype=q.dtype)
    n = np.zeros(dim, dtype=q.dtype)
    m = q.dtype.type(0.0)
    out = np.empty_like(v)
    for a in range(t):
        m_new = max(f[a] + m, i[a])
        keep, add = np.exp(f[a] + m - m_new), np.exp(i[a] - m_new)
        s = keep * s + add * np.outer(k[a], v[a])
        n = keep * n + add * k[a]
        m = m_new
        out[a] = (q[a] @ s) / (max(abs(n @ q[a]), np.exp(-m)) + 1e-6)
    return out


def mlstm(h, w, mix, eps):
    """w: dict with q, k, v, g, o, norm, i, i.b, f, f.b."""
    t = h.shape[0]
    heads, dim, vdim, cap = mix["heads"], mix["dim"], mix["vdim"], mix["gate_cap"]
    q = (h @ w["q"].T * dim ** -0.5).reshape(t, heads, dim)
    k = (h @ w["k"].T).reshape(t, heads, dim)
    v = (h @ w["v"].T).reshape(t, heads, vdim)
    i = cap * np.tanh((h @ w["i"].T + w["i.b"]) / cap)
    f = log_sigmoid(cap * np.tanh((h @ w["f"].T + w["f.b"]) / cap))
    o = np.stack([rms_norm(mlstm_recurrence(q[:, a], k[:, a], v[:, a], i[:, a], f[:, a]), eps)
                  for a in range(heads)], axis=1).reshape(t, heads * vdim)
    return (o * w["norm"] * sigmoid(h @ w["g"].T)) @ w["o"].T


def layer_runs(config):
    """[(layer, pass)] in execution order; pass is None outside the loop."""
    n, loop = len(config["layers"]), config["loop"]
    runs = [(i, None) for i in range(loop["start"])]
    for p in range(loop["times"]):
        runs += [(i, p) for i in range(loop["start"], loop["stop"])]
    return runs + [(i, None) for i in range(loop["stop"], n)]


def embedding(weights, config, tokens):
    return norm_one_plus(weights["embed"][tokens], weights["embed.norm"], config["norm"]["eps"])


def loop_entry(x, x0, weights, p):
    """What happens in front of pass p: merge with the embedding output, then the pass's vector."""
    return np.concatenate([x, x0], axis=-1) @ weights["loop.in"].T + weights["loop.step"][p]


def run_layer(x, weights, config, i):
    spec, eps, pre = config["layers"][i], config["norm"]["eps"], f"l{i}."
    mix = {k[len(pre) + 4:]: v for k, v in weights.items() if k.startswith(pre + "mix.")}
    fn = {"attention": attention, "mlstm": mlstm}[spec["type"]]
    x = x + fn(norm_one_plus(x, weights[pre + "norm1"], eps), mix, spec["mixer"], eps)
    if spec["mlp"] is not None:
        h = norm_one_plus(x, weights[pre + "norm2"], eps)
        x = x + gated_mlp(h, weights[pre + "mlp.gate"], weights[pre + "mlp.up"], weights[pre + "mlp.down"])
    return x


def forward(weights, config, tokens, layers=None):
    """Logits [T, vocab]; `layers`, when a list, receives the residual after every layer run."""
    x0 = embedding(weights, config, np.asarray(tokens))
    x = x0
    for i, p in layer_runs(config):
        if p is not None and i == config["loop"]["start"]:
            x = loop_entry(x, x0, weights, p)
        x = run_layer(x, weights, config, i)
        if layers is not None:
            layers.append(x)
    x = norm_one_plus(x, weights["final.norm"], config["norm"]["eps"])
    return x @ weights["embed"].T * config["logit_scale"]
