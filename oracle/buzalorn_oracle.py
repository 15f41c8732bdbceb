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


def attention_core(q, k, v, scale, window, rel=None, bias_max=None):
    """q [T, heads, dim], k [T, kv_heads, dim], v [T, kv_heads, vdim] -> [T, heads, vdim]."""
    t, heads = q.shape[:2]
    seen = window_visible(t, window)
    out = np.empty((t, heads, v.shape[2]), dtype=q.dtype)
    for a in range(heads):
        g = a // (heads // k.shape[1])
        s = q[:, a] @ k[:, g].T * scale
        if rel is not None:
            s = s + distance_bias(t, rel[:, a], bias_max)
        out[:, a] = attention_weights(s, seen) @ v[:, g]
    return out


def attention(h, w, mix, eps):
    """w: dict with q, k, v, q.norm, k.norm, rel, o."""
    t = h.shape[0]
    heads, kvh, dim, vdim = mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"]
    q = (rms_norm(h @ w["q"].T, eps) * w["q.norm"]).reshape(t, heads, dim)
    k = (rms_norm(h @ w["k"].T, eps) * w["k.norm"]).reshape(t, kvh, dim)
    v = (h @ w["v"].T).reshape(t, kvh, vdim)
    o = attention_core(q, k, v, mix["scale"], mix["mask"]["size"], w["rel"], mix["bias_max"])
    return o.reshape(t, heads * vdim) @ w["o"].T


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


def mlstm_gates(pre_i, pre_f, cap):
    """Log input and log forget gate from their pre-activations."""
    return cap * np.tanh(pre_i / cap), log_sigmoid(cap * np.tanh(pre_f / cap))


def head_norm_gate(o, norm, g, eps):
    """o [T, heads, vdim] normed per head, times norm and sigmoid(g) -> [T, heads * vdim]."""
    return rms_norm(o, eps).reshape(o.shape[0], -1) * norm * sigmoid(g)


def mlstm(h, w, mix, eps):
    """w: dict with q, k, v, g, o, norm, i, i.b, f, f.b."""
    t = h.shape[0]
    heads, dim, vdim = mix["heads"], mix["dim"], mix["vdim"]
    q = (h @ w["q"].T * dim ** -0.5).reshape(t, heads, dim)
    k = (h @ w["k"].T).reshape(t, heads, dim)
    v = (h @ w["v"].T).reshape(t, heads, vdim)
    i, f = mlstm_gates(h @ w["i"].T + w["i.b"], h @ w["f"].T + w["f.b"], mix["gate_cap"])
    o = np.stack([mlstm_recurrence(q[:, a], k[:, a], v[:, a], i[:, a], f[:, a]) for a in range(heads)], axis=1)
    return head_norm_gate(o, w["norm"], h @ w["g"].T, eps) @ w["o"].T


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
