"""Plain, slow Gotulorn model in numpy float64: the yardstick for the Gotulorn tests.

Whole sequences, no cache, no batching, one function per mechanism, nothing shared with the
package under test.  Notation: a sequence of n tokens is a matrix [n, width]; position p of a
sequence is row p; W x for a stored matrix W [out, in] is written ``x @ W.T``.

Mechanisms
----------
``bent``               the elementwise norm: tanh(a x) g + b with one number a
``over_rms``           x / sqrt(mean(x^2) + eps) over the last axis
``turned``             rotation of neighbouring pairs by position times frequency
``sees``               which keys a position sees: the last ``size`` ones and the sequence's first ``first`` ones
``weighted``           softmax attention of one query row over given keys and values
``mix_factor``         the number that a pair of maps is combined with
``keys_and_values``    what a layer of paired maps caches (and what a borrowing layer reads)
``paired_attention``   two softmax maps per head over the same values, their difference normed
``latent_attention``   keys and values of all heads expanded from one normed latent per token
``clamped_ff``         the dense feed-forward with a clamped swish gate
``routed_ff``          the routed feed-forward: the largest logits, a softmax over the chosen ones
``forward``            the whole model: logits at every position and the residual after every layer
"""
from __future__ import annotations

import numpy as np

F64 = np.float64
SWISH = 1.702


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def bent(x, g, b, a):
    return np.tanh(a * x) * g + b


def over_rms(x, eps):
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def turned(x, base):
    """x [n, ..., dims]: row p is turned by the angles p * base^(-2i / dims)."""
    n, dims = x.shape[0], x.shape[-1]
    i = np.arange(dims // 2, dtype=F64)
    angle = np.arange(n, dtype=F64)[:, None] * base ** (-2.0 * i / dims)
    angle = angle.reshape((n,) + (1,) * (x.ndim - 2) + (dims // 2,))
    u, v = x[..., 0::2], x[..., 1::2]
    out = np.empty_like(x)
    out[..., 0::2] = u * np.cos(angle) - v * np.sin(angle)
    out[..., 1::2] = v * np.cos(angle) + u * np.sin(angle)
    return out


def sees(p, mask):
    """The positions that position p sees, in rising order; ``mask`` None: all up to p."""
    j = np.arange(p + 1)
    if not mask:
        return j
    return j[(p - j < mask["size"]) | (j < mask.get("keep_first", 0))]


def weighted(scores, values):
    e = np.exp(scores - scores.max())
    return (e @ values) / e.sum()


def mix_factor(w, diff):
    return float(np.exp((w["lq1"] * w["lk1"]).sum()) - np.exp((w["lq2"] * w["lk2"]).sum()) + diff)


def keys_and_values(h, w, m):
    """(k [n, G, 2, dim], v [n, G, vdim])."""
    n, G = h.shape[0], m["kv_heads"]
    return (h @ w["k"].T).reshape(n, G, 2, m["dim"]), (h @ w["v"].T).reshape(n, G, m["vdim"])


def paired_attention(h, w, m, eps, k, v):
    """h [n, width]; w: q, lq1, lk1, lq2, lk2, o; m: heads, kv_heads, dim, scale, diff, mask."""
    n, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = (h @ w["q"].T).reshape(n, H, 2, m["dim"])
    lam = mix_factor(w, m["diff"])
    out = np.zeros((n, H, v.shape[-1]), dtype=F64)
    for p in range(n):
        j = sees(p, m.get("mask"))
        for hd in range(H):
            g = hd // (H // G)
            one, two = (weighted((k[j, g, t] @ q[p, hd, t]) * m["scale"], v[j, g]) for t in (0, 1))
            out[p, hd] = over_rms(one - lam * two, eps) * (1.0 - m["diff"])
    return out.reshape(n, -1) @ w["o"].T


def latent_attention(h, w, m, eps):
    n, H, d, r, dv, rank = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (h @ w["q"].T).reshape(n, H, d + r)
    down = h @ w["dkv"].T
    c = over_rms(down[:, :rank], eps) * w["dkv.norm"]
    shared = turned(down[:, rank:], m["rot"]["base"]) if r else down[:, rank:]
    q_turned = turned(q[:, :, d:], m["rot"]["base"]) if r else q[:, :, d:]
    k = (c @ w["uk"].T).reshape(n, H, d)
    v = (c @ w["uv"].T).reshape(n, H, dv)
    out = np.zeros((n, H, dv), dtype=F64)
    for hd in range(H):
        s = (q[:, hd, :d] @ k[:, hd].T + q_turned[:, hd] @ shared.T) * m["scale"]
        for p in range(n):
            out[p, hd] = weighted(s[p, :p + 1], v[:p + 1, hd])
    return out.reshape(n, -1) @ w["o"].T


def clamped_ff(h, w, limit):
    g, u = np.minimum(h @ w["gate"].T, limit), np.clip(h @ w["up"].T, -limit, limit)
    return (g * sigmoid(SWISH * g) * (u + 1.0)) @ w["down"].T


def routed_ff(h, w, rec):
    top = rec["router"]["top"]
    z = h @ w["router"].T + w["router.b"]
    y = np.zeros_like(h)
    for t in range(h.shape[0]):
        chosen = np.argsort(-z[t], kind="stable")[:top]
        e = np.exp(z[t, chosen] - z[t, chosen].max())
        for weight, x in zip(e / e.sum(), chosen):
            g = h[t] @ w[f"e{x}.gate"].T
            y[t] += weight * ((g * sigmoid(g) * (h[t] @ w[f"e{x}.up"].T)) @ w[f"e{x}.down"].T)
    return y


def forward(config, weights, tokens):
    """``weights``: name -> float64 array.  Returns (logits [n, vocab], residuals [layers, n, width])."""
    eps = config["norm"]["eps"]

    def norm(name, x):
        return bent(x, weights[name], weights[name + ".b"], weights[name + ".alpha"])

    def part(prefix):
        return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}

    x = norm("embed.norm", weights["embed"][np.asarray(tokens)] * config["embedding"]["scale"])
    lent, after = {}, []
    for i, layer in enumerate(config["layers"]):
        m, w = layer["mixer"], part(f"l{i}.mix.")
        h = norm(f"l{i}.norm1", x)
        if layer["type"] == "latent_attention":
            x = x + latent_attention(h, w, m, eps)
        else:
            if m.get("kv_from") is None:
                lent[i] = keys_and_values(h, w, m)
            x = x + paired_attention(h, w, m, eps, *lent[i if m.get("kv_from") is None else m["kv_from"]])
        mlp = layer.get("mlp")
        if mlp is not None:
            h, w = norm(f"l{i}.norm2", x), part(f"l{i}.mlp.")
            x = x + (clamped_ff(h, w, mlp["limit"]) if mlp["kind"] == "dense" else routed_ff(h, w, mlp))
        after.append(x)
    return norm("final.norm", x) @ weights["head"].T, np.stack(after)
