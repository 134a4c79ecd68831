"""Small Gotulorn configurations and weights for the tests, and the comparison with the plain model.

The configurations differ from each other in every size and option.  A: values larger and smaller than a head's two keys,
windows that the prompts pass many times, a layer that borrows keys and values through a wider mask than its lender's, one
that borrows through no mask at all, a layer without feed-forward, a latent row that is no multiple of 16.  B: a width that is
no multiple of 8, one key/value head for all query heads, a window of one token, nothing kept, a latent part without
rotation, one expert per token, a borrower with a narrower mask.  C: head sizes of 64 and 128 (the tensor-core kernels and
the vectorised preparation), kept tokens that fill more than a page, as many experts as are chosen.  D: sizes that are
multiples of nothing, a window and a number of kept tokens that lie one beside a page's border, an attention layer without a
mask.

Weights are made here, with activations of order one (so that attention is far from uniform and a missing map, kept token,
bias or norm shows), rounded to bfloat16 and stored as bfloat16.
"""
from __future__ import annotations

import json
import os

import numpy as np

import plain_gotulorn
import plain_qwen3


def attn(heads, kv, dim, vdim, size=None, keep=None, diff=0.4, scale=None, kv_from=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "diff": diff, "scale": scale if scale is not None else dim ** -0.5}
    if size is not None:
        m["mask"] = {"size": size}
        if keep is not None:
            m["mask"]["keep_first"] = keep
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def latent(heads, dim, rot_dim, vdim, rank, base=1000.0, scale=None):
    return {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank,
            "scale": scale if scale is not None else (dim + rot_dim) ** -0.5, "rot": {"base": base, "dims": rot_dim}}


def dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(experts, top, ff):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}


def layer(kind, mixer, mlp):
    return {"type": {"a": "attention", "l": "latent_attention"}[kind], "mixer": mixer, "mlp": mlp}


def config_of(vocab, width, scale, eps, layers):
    return {"architecture": "Gotulorn", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "norm": {"eps": eps},
            "layers": layers}


CFG_A = config_of(97, 40, 1.7, 1e-4, [
    layer("a", attn(4, 2, 12, 36, 17, 3, diff=0.3), dense(56, 0.9)),
    layer("l", latent(3, 10, 6, 14, 20), moe(6, 3, 24)),
    layer("a", attn(6, 2, 12, 36, 45, 5, diff=0.6, scale=0.5, kv_from=0), None),
    layer("a", attn(4, 4, 20, 12, 24, 2, diff=0.1), moe(5, 2, 16)),
    layer("a", attn(4, 4, 20, 12, diff=0.7, kv_from=3), dense(24, 2.0)),
    layer("l", latent(4, 8, 10, 24, 38, base=50.0), None),
])
CFG_B = config_of(131, 52, 0.6, 2e-5, [
    layer("l", latent(2, 18, 0, 10, 33), moe(7, 1, 20)),
    layer("a", attn(5, 1, 8, 8, 33, 0, diff=0.2), dense(44, 1.1)),
    layer("a", attn(3, 1, 8, 8, 9, 4, diff=0.5, kv_from=1), moe(4, 4, 12)),
    layer("a", attn(2, 2, 17, 34, 1, 2, diff=0.35), dense(20, 0.7)),
])
CFG_C = config_of(300, 128, 2.5, 1e-6, [
    layer("a", attn(4, 2, 32, 64, 70, 40, diff=0.25), dense(160, 1.3)),
    layer("l", latent(4, 48, 32, 40, 96, base=10000.0), moe(16, 4, 32)),
    layer("a", attn(8, 1, 64, 128, 100, 9, diff=0.55), moe(3, 3, 64)),
    layer("a", attn(8, 1, 64, 96, 64, 32, diff=0.15, scale=0.2), dense(96, 0.6)),
    layer("a", attn(4, 1, 64, 96, 128, 1, diff=0.45, kv_from=3), moe(8, 2, 48)),
])
CFG_D = config_of(83, 50, 1.0, 3e-6, [
    layer("a", attn(7, 7, 5, 13, 31, 33, diff=0.8, scale=0.9), moe(1, 1, 30)),
    layer("l", latent(1, 7, 2, 3, 11, base=7.0), dense(18, 0.5)),
    layer("a", attn(1, 1, 11, 22, diff=0.0), moe(9, 3, 10)),
])
ALL = {"A": CFG_A, "B": CFG_B, "C": CFG_C, "D": CFG_D}


def _bf16(a):
    return plain_qwen3.bf16_round(np.asarray(a, dtype=np.float32)).astype(np.float32)


def make_weights(config, seed):
    """name -> float32 array (every value a bfloat16 number)."""
    rng = np.random.default_rng(seed)
    D, V = config["width"], config["vocab"]
    W = {}

    def mat(name, n_out, n_in, gain=1.0):
        W[name] = _bf16(rng.standard_normal((n_out, n_in)) * gain / np.sqrt(n_in))

    def vec(name, size, lo, hi):
        W[name] = _bf16(rng.uniform(lo, hi, size=size))

    def norm(name):
        vec(name, D, 0.6, 1.6)
        W[name + ".b"] = _bf16(rng.standard_normal(D) * 0.2)
        vec(name + ".alpha", (), 0.5, 1.2)

    W["embed"] = _bf16(rng.standard_normal((V, D)) * 0.7)
    norm("embed.norm")
    mat("head", V, D, 1.5)
    norm("final.norm")
    for i, lay in enumerate(config["layers"]):
        p, m = f"l{i}.", lay["mixer"]
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        norm(p + "norm1")
        mat(p + "mix.o", D, H * dv)
        if lay["type"] == "attention":
            mat(p + "mix.q", H * 2 * d, D, 1.5)
            if m.get("kv_from") is None:
                mat(p + "mix.k", m["kv_heads"] * 2 * d, D, 1.5)
                mat(p + "mix.v", m["kv_heads"] * dv, D)
            for name in ("lq1", "lk1", "lq2", "lk2"):
                W[p + "mix." + name] = _bf16(rng.standard_normal(d) * 0.5 / np.sqrt(d))
        else:
            r, rank = m["rot_dim"], m["kv_rank"]
            mat(p + "mix.q", H * (d + r), D, 1.5)
            mat(p + "mix.dkv", rank + r, D, 1.5)
            vec(p + "mix.dkv.norm", rank, 0.5, 1.5)
            mat(p + "mix.uk", H * d, rank, 1.5)
            mat(p + "mix.uv", H * dv, rank)
        mlp = lay["mlp"]
        if mlp is None:
            continue
        norm(p + "norm2")
        if mlp["kind"] == "dense":
            mat(p + "mlp.gate", mlp["ff"], D, 1.5)
            mat(p + "mlp.up", mlp["ff"], D, 1.5)
            mat(p + "mlp.down", D, mlp["ff"])
            continue
        E, ff = mlp["router"]["experts"], mlp["expert"]["ff"]
        mat(p + "mlp.router", E, D, 2.0)
        W[p + "mlp.router.b"] = _bf16(rng.standard_normal(E))
        for e in range(E):
            mat(f"{p}mlp.e{e}.gate", ff, D, 1.5)
            mat(f"{p}mlp.e{e}.up", ff, D, 1.5)
            mat(f"{p}mlp.e{e}.down", D, ff)
    return W


def write_model(folder, config, weights):
    import torch
    from rust_inference_b200.weights.safetensors_io import save_safetensors
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(config, f)
    save_safetensors(os.path.join(folder, "model.safetensors"),
                     {k: torch.from_numpy(np.ascontiguousarray(v)).reshape(v.shape).to(torch.bfloat16) for k, v in weights.items()})
    return folder


def make_model_dir(base, name, seed=1):
    config = ALL[name]
    weights = make_weights(config, seed)
    return write_model(os.path.join(str(base), f"gotulorn_{name}"), config, weights), config, weights


def as64(weights):
    return {k: v.astype(np.float64) for k, v in weights.items()}


def plain_logits(config, weights, requests):
    W = as64(weights)
    return {rid: plain_gotulorn.forward(config, W, toks)[0] for rid, toks in requests.items()}


def row_error(got, want):
    """The difference of two rows of logits with the mean taken off, relative to the spread of the wanted row."""
    d = got.astype(np.float64) - want
    d = d - d.mean()
    w = want - want.mean()
    return float(np.sqrt((d * d).mean()) / max(np.sqrt((w * w).mean()), 1e-30))


# (nearly every row, mean over all rows, any row).  float32: rounding alone.  bfloat16: activations are rounded to 8 bits
# between the parts, and where two of a router's outputs lie close together that rounding may choose another expert: such a
# row is off by any amount, so one row in fifty may be, and the mean holds them all together.
BOUND = {"float32": (1e-4, 2e-5, 1e-4), "bfloat16": (2.5e-1, 5e-2, 1.5)}


def assert_rows_close(rows, want_by_request, dtype, what=""):
    most, mean_bound, any_row = BOUND[dtype]
    errs = sorted(((row_error(got, want_by_request[rid][p]), rid, p) for (rid, p), got in rows.items()), reverse=True)
    over = [e for e in errs if e[0] > most]
    assert len(over) <= len(errs) // 50 and errs[0][0] <= any_row, f"{what}: {len(over)} of {len(errs)} rows over {most:.1e}: {over[:3]}"
    mean = sum(e[0] for e in errs) / max(len(errs), 1)
    assert mean <= mean_bound, f"{what}: mean error {mean:.3e} exceeds {mean_bound:.1e}"
    return round(errs[0][0], 7), len(over), round(mean, 7)
