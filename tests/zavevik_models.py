"""Small Zavevik configurations and weights for the tests, and the comparison with the plain model.

The configurations differ from each other in every size and option.  A: values larger than keys (head sizes that are
padded), a layer that borrows keys and values from the one before and one that borrows from further back, a query factor
that changes every ten positions, three of six experts per token, a layer without feed-forward, three taps.  B: no soft cap,
no query factor, no distance bias in one layer, no token-fed sublayer, a width that is no multiple of 8, one key/value head
for all query heads, more key channels than the register kernel takes at once, one expert per token.  C: head sizes of 64
and 128 (the tensor-core kernels and the vectorised preparation kernel), a distance bias that reaches beyond the prompts, a
query factor that changes at every position.  D: sizes that are multiples of nothing, one tap, one expert in all, a bias of
two rows.

Weights are made here, with activations of order one (so that attention is far from uniform and a missing bias, factor, gate
or norm shows), rounded to bfloat16 and stored as bfloat16; the tables of experts are int32.
"""
from __future__ import annotations

import json
import os

import numpy as np

import plain_qwen3
import plain_zavevik


def attn(heads, kv, dim, vdim, scale=None, cap=None, temp=None, far=None, rows=0, kv_from=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else dim ** -0.5}
    if cap:
        m["softcap"] = cap
    if temp:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    if far:
        m["bias_max"], m["bias_rows"] = far, rows
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def delta(heads, kv, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv}


def moe(experts, top, ff):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}


def layer(kind, mixer, mlp):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


CFG_A = {
    "architecture": "Zavevik", "vocab": 97, "width": 40, "norm": {"eps": 1e-5}, "token_side": {"dim": 12},
    "layers": [
        layer("attention", attn(4, 2, 24, 40, scale=0.5, cap=6.0, temp=(0.6, 10), far=70, rows=10), moe(6, 3, 24)),
        layer("attention", attn(4, 2, 24, 40, scale=0.3, cap=3.0, temp=(0.2, 7), far=33, rows=8, kv_from=0), None),
        layer("delta", delta(4, 2, 12, 20, 3), moe(5, 2, 16)),
        layer("attention", attn(4, 2, 24, 40, scale=0.4, far=120, rows=6, kv_from=0), moe(4, 1, 40)),
        layer("delta", delta(2, 2, 20, 8, 2), None),
    ],
}
CFG_B = {
    "architecture": "Zavevik", "vocab": 131, "width": 52, "norm": {"eps": 2e-6},
    "layers": [
        layer("delta", delta(2, 1, 136, 24, 4), moe(7, 1, 20)),
        layer("attention", attn(5, 1, 20, 12, far=40, rows=4), moe(3, 2, 28)),
        layer("attention", attn(2, 2, 34, 34, scale=0.6), moe(4, 4, 12)),
    ],
}
CFG_C = {
    "architecture": "Zavevik", "vocab": 300, "width": 128, "norm": {"eps": 1e-6}, "token_side": {"dim": 32},
    "layers": [
        layer("attention", attn(4, 2, 128, 64, cap=9.0, temp=(0.3, 1), far=500, rows=16), moe(16, 4, 32)),
        layer("delta", delta(2, 2, 96, 128, 4), moe(8, 1, 64)),
        layer("attention", attn(8, 1, 64, 64, scale=0.2, cap=20.0, temp=(0.5, 64), far=90, rows=32), moe(8, 2, 48)),
        layer("attention", attn(8, 1, 64, 64, scale=0.15, cap=4.0, far=200, rows=12, kv_from=2), moe(8, 2, 48)),
    ],
}
CFG_D = {
    "architecture": "Zavevik", "vocab": 83, "width": 50, "norm": {"eps": 3e-6}, "token_side": {"dim": 5},
    "layers": [
        layer("attention", attn(7, 7, 10, 6, scale=0.7, cap=5.0, temp=(1.5, 33), far=9, rows=2), moe(1, 1, 30)),
        layer("delta", delta(3, 1, 14, 18, 1), moe(5, 2, 14)),
        layer("attention", attn(1, 1, 22, 22, temp=(0.4, 5), far=61, rows=14), moe(9, 3, 10)),
    ],
}
ALL = {"A": CFG_A, "B": CFG_B, "C": CFG_C, "D": CFG_D}


def _bf16(a):
    return plain_qwen3.bf16_round(np.asarray(a, dtype=np.float32)).astype(np.float32)


def make_weights(config, seed):
    """name -> float32 array (every value a bfloat16 number), or int32 for the tables of experts."""
    rng = np.random.default_rng(seed)
    D, V, n = config["width"], config["vocab"], len(config["layers"])
    W = {}

    def mat(name, n_out, n_in, gain=1.0):
        W[name] = _bf16(rng.standard_normal((n_out, n_in)) * gain / np.sqrt(n_in))

    def vec(name, size, lo, hi):
        W[name] = _bf16(rng.uniform(lo, hi, size=size))

    W["embed"] = _bf16(rng.standard_normal((V, D)) * 0.7)
    mat("head", V, D, 1.5)
    vec("final.norm", (), 0.7, 1.3)
    side = (config.get("token_side") or {}).get("dim", 0)
    if side:
        W["side.embed"] = _bf16(rng.standard_normal((V, n * side)))
    for i, lay in enumerate(config["layers"]):
        p, m = f"l{i}.", lay["mixer"]
        H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        vec(p + "norm1", (), 0.5, 1.5)
        mat(p + "mix.q", (H if lay["type"] == "attention" else G) * d, D, 2.0)
        if m.get("kv_from") is None:
            mat(p + "mix.k", G * d, D, 2.0)
            mat(p + "mix.v", (G if lay["type"] == "attention" else H) * dv, D)
        mat(p + "mix.o", D, H * dv)
        if lay["type"] == "attention":
            if m.get("bias_max"):
                W[p + "mix.rel"] = _bf16(rng.standard_normal((m["bias_rows"], H)) * 1.5)
        else:
            for name, size in (("q", G * d), ("k", G * d), ("v", H * dv)):
                W[p + f"mix.{name}.conv"] = _bf16(rng.standard_normal((size, m["conv"])) * 0.6)
            mat(p + "mix.b", H, D, 2.0)
            mat(p + "mix.a", H, D, 2.0)
            mat(p + "mix.g", H * dv, D, 2.0)
            vec(p + "mix.A_log", H, -2.0, 0.5)
            vec(p + "mix.dt_bias", H, -3.0, 0.5)
            vec(p + "mix.norm", dv, 0.5, 1.5)
        mlp = lay["mlp"]
        if mlp is not None:
            vec(p + "norm2", (), 0.5, 1.5)
            E, top, ff = mlp["router"]["experts"], mlp["router"]["top"], mlp["expert"]["ff"]
            W[p + "mlp.table"] = np.stack([rng.permutation(E)[:top] for _ in range(V)]).astype(np.int32)
            for e in range(E):
                mat(f"{p}mlp.e{e}.gate", ff, D, 2.0)
                mat(f"{p}mlp.e{e}.up", ff, D, 2.0)
                mat(f"{p}mlp.e{e}.down", D, ff)
        if side:
            mat(p + "side.gate", side, D, 2.0)
            mat(p + "side.proj", D, side)
            vec(p + "side.norm", D, 0.3, 1.0)
    return W


def write_model(folder, config, weights):
    """config.json (without the numbers of rows that the biases' tensors give) and model.safetensors in ``folder``."""
    import torch
    from rust_inference_b200.weights.safetensors_io import save_safetensors
    os.makedirs(folder, exist_ok=True)
    config = json.loads(json.dumps(config))
    for lay in config["layers"]:
        lay["mixer"].pop("bias_rows", None)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(config, f)
    save_safetensors(os.path.join(folder, "model.safetensors"),
                     {k: torch.from_numpy(np.ascontiguousarray(v)).reshape(v.shape).to(torch.int32 if v.dtype == np.int32 else torch.bfloat16)
                      for k, v in weights.items()})
    return folder


def make_model_dir(base, name, seed=1):
    config = ALL[name]
    weights = make_weights(config, seed)
    return write_model(os.path.join(str(base), f"zavevik_{name}"), config, weights), config, weights


def as64(weights):
    return {k: v.astype(np.float64) for k, v in weights.items()}


def plain_logits(config, weights, requests):
    W = as64(weights)
    return {rid: plain_zavevik.forward(config, W, toks)[0] for rid, toks in requests.items()}


def row_error(got, want):
    """The difference of two rows of logits with the mean taken off, relative to the spread of the wanted row."""
    d = got.astype(np.float64) - want
    d = d - d.mean()
    w = want - want.mean()
    return float(np.sqrt((d * d).mean()) / max(np.sqrt((w * w).mean()), 1e-30))


# float32: rounding alone.  bfloat16: activations are rounded to 8 bits between the parts of every sublayer, and where a
# head of the delta rule puts out next to nothing its norm makes that rounding large: single rows are a few tenths off (with
# the kernels as with a stand-in that rounds at the same places); the mean over
# all rows is held much tighter (a wrong mechanism moves every row by about one).
BOUND = {"float32": (1e-4, 2e-5), "bfloat16": (8e-1, 6e-2)}


def assert_rows_close(rows, want_by_request, dtype, what=""):
    worst, total = 0.0, 0.0
    for (rid, p), got in sorted(rows.items()):
        err = row_error(got, want_by_request[rid][p])
        worst, total = max(worst, err), total + err
        assert err <= BOUND[dtype][0], f"{what}: request {rid} position {p}: error {err:.3e} exceeds {BOUND[dtype][0]:.1e}"
    mean = total / max(len(rows), 1)
    assert mean <= BOUND[dtype][1], f"{what}: mean error {mean:.3e} exceeds {BOUND[dtype][1]:.1e}"
    return round(worst, 7), round(mean, 7)
