"""Plain, slow Zavevik model in numpy float64: the yardstick for the Zavevik tests.

Whole sequences, no cache, no batching, one function per mechanism, nothing shared with the
package under test.  Notation: a sequence of n tokens is a matrix [n, width]; position p of a
sequence is row p; W x for a stored matrix W [out, in] is written ``x @ W.T``.

Mechanisms
----------
``over_rms``           x / sqrt(mean(x^2) + eps) over the last axis
``distance_bucket``    which row of a table of learned biases belongs to a distance: one row per distance in the first
                       half of the table, then rows whose spans grow geometrically up to a largest distance
``query_factor``       1 + coef ln(floor((p + 1) / every) + 1) at position p
``keys_and_values``    projections, unit-RMS keys and values (what a layer that lends its cache hands out)
``attention``          grouped-query attention over given keys and values: unit-RMS queries times their position's factor,
                       a soft cap on the scores, then the distance's bias of the layer and head
``short_conv``         causal convolution over time per channel (zeros before the start), then silu
``delta_rule``         the gated delta rule as a token-by-token recurrence with one decay per token
``delta_mixer``        projections, convolutions, unit vectors, the recurrence, the heads' norm and silu gate
``table_moe``          experts that a table names for every token id, with equal weights
``token_side``         the layer's own part of a table of token rows, gated by the residual
``forward``            the whole model: logits at every position and the residual after every layer
"""
from __future__ import annotations

import math

import numpy as np

F64 = np.float64
UNIT_EPS = 1e-6             # inside the root of a unit vector's length


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def over_rms(x, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def distance_bucket(n, rows, far):
    half = rows // 2
    if n < half:
        return n
    # (a hair is added so that a distance exactly on a border belongs to the row that starts there)
    return min(rows - 1, int(half + math.floor(math.log(n / half) / math.log(far / half) * (rows - half) + 1e-9)))


def query_factor(p, coef, every):
    return 1.0 + coef * math.log(math.floor((p + 1) / every) + 1.0)


def keys_and_values(h, w, m, eps):
    """(k [n, G, dim], v [n, G, vdim]) as a cache would hold them."""
    n, G = h.shape[0], m["kv_heads"]
    k = over_rms((h @ w["k"].T).reshape(n, G, m["dim"]), eps)
    v = over_rms((h @ w["v"].T).reshape(n, G, m["vdim"]), eps)
    return k, v


def attention(h, w, m, eps, k, v):
    """h [n, width]; w: the tensors q, rel, o; m: heads, kv_heads, dim, vdim, scale, softcap, q_temp, bias_max."""
    n, H, G, dim = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = over_rms((h @ w["q"].T).reshape(n, H, dim), eps)
    temp = m.get("q_temp")
    if temp:
        q = q * np.asarray([query_factor(p, temp["coef"], temp["every"]) for p in range(n)])[:, None, None]
    bias = np.zeros((n, H))                                    # by distance; none without a largest distance
    if m.get("bias_max"):
        bias = w["rel"][[distance_bucket(d, w["rel"].shape[0], m["bias_max"]) for d in range(n)]]
    cap = m.get("softcap")
    out = np.zeros((n, H, v.shape[-1]), dtype=F64)
    for hd in range(H):
        g = hd // (H // G)
        s = (q[:, hd] @ k[:, g].T) * m["scale"]
        if cap:
            s = cap * np.tanh(s / cap)
        for p in range(n):
            z = s[p, :p + 1] + bias[p - np.arange(p + 1), hd]
            e = np.exp(z - z.max())
            out[p, hd] = (e @ v[:p + 1, g]) / e.sum()
    return out.reshape(n, -1) @ w["o"].T


def short_conv(x, taps_w):
    """x [n, channels], taps_w [channels, taps], the last column is the current token's."""
    n, taps = x.shape[0], taps_w.shape[1]
    y = np.zeros_like(x)
    for j in range(taps):
        back = taps - 1 - j
        if back < n:
            y[back:] += x[:n - back] * taps_w[:, j]
    return silu(y)


def delta_rule(q, k, v, beta, g):
    """One head.  q, k [n, dim], v [n, vdim], beta [n], g [n] (decay of the whole state).  Returns o [n, vdim]."""
    S = np.zeros((q.shape[1], v.shape[1]), dtype=F64)
    o = np.zeros_like(v)
    for t in range(q.shape[0]):
        S = g[t] * S
        u = beta[t] * (v[t] - S.T @ k[t])
        S = S + np.outer(k[t], u)
        o[t] = S.T @ q[t]
    return o


def delta_mixer(h, w, m, eps):
    n = h.shape[0]
    H, G, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = short_conv(h @ w["q"].T, w["q.conv"]).reshape(n, G, dim)
    k = short_conv(h @ w["k"].T, w["k.conv"]).reshape(n, G, dim)
    v = short_conv(h @ w["v"].T, w["v.conv"]).reshape(n, H, vdim)
    q = q / np.sqrt((q * q).sum(-1, keepdims=True) + UNIT_EPS) * dim ** -0.5
    k = k / np.sqrt((k * k).sum(-1, keepdims=True) + UNIT_EPS)
    beta = sigmoid(h @ w["b"].T)                                                       # [n, H]
    g = np.exp(-np.exp(w["A_log"]) * softplus(h @ w["a"].T + w["dt_bias"]))            # [n, H]
    gate = silu(h @ w["g"].T).reshape(n, H, vdim)
    out = np.zeros((n, H, vdim), dtype=F64)
    for hd in range(H):
        kv = hd // (H // G)
        out[:, hd] = over_rms(delta_rule(q[:, kv], k[:, kv], v[:, hd], beta[:, hd], g[:, hd]), eps) * w["norm"] * gate[:, hd]
    return out.reshape(n, H * vdim) @ w["o"].T


def expert_ff(h, gate, up, down):
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def table_moe(h, w, m, tokens):
    top = m["router"]["top"]
    out = np.zeros_like(h)
    for t, tok in enumerate(tokens):
        for e in w["table"][tok]:
            e = int(e)
            out[t] += expert_ff(h[t:t + 1], w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"])[0] / top
    return out


def token_side(x, w, rows, eps):
    """x [n, width]; rows [n, dim]: the layer's part of the tokens' rows; w: gate, proj, norm.  What joins the residual."""
    y = (gelu_tanh(x @ w["gate"].T) * rows) @ w["proj"].T
    return over_rms(y, eps) * w["norm"]


def forward(cfg, tensors, tokens):
    """(logits [n, vocab], residual after every layer [layers, n, width]) for one sequence."""
    W = {k: np.asarray(v, dtype=F64) for k, v in tensors.items()}
    tokens = np.asarray(tokens, dtype=np.int64)
    x = W["embed"][tokens]
    eps = cfg["norm"]["eps"]
    after, lent = [], {}
    for i, layer in enumerate(cfg["layers"]):
        pre = f"l{i}."

        def group(name):
            return {k[len(pre) + len(name) + 1:]: v for k, v in W.items() if k.startswith(pre + name + ".")}

        m, wm = layer["mixer"], group("mix")
        if layer["type"] == "attention":
            if m.get("kv_from") is None:
                lent[i] = keys_and_values(x, wm, m, eps)
            y = attention(x, wm, m, eps, *lent[i if m.get("kv_from") is None else m["kv_from"]])
        else:
            y = delta_mixer(x, wm, m, eps)
        x = x + over_rms(y, eps) * W[pre + "norm1"]
        if layer.get("mlp") is not None:
            x = x + over_rms(table_moe(x, group("mlp"), layer["mlp"], tokens), eps) * W[pre + "norm2"]
        if cfg.get("token_side"):
            dim = cfg["token_side"]["dim"]
            x = x + token_side(x, group("side"), W["side.embed"][tokens][:, i * dim:(i + 1) * dim], eps)
        after.append(x.copy())
    h = over_rms(x, eps) * W["final.norm"]
    return h @ W["head"].T, np.stack(after)
