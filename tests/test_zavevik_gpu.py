"""Zavevik on the GPU: each kernel against the plain formulas of tests/plain_zavevik.py, then whole models through trace
replay in several cuttings (whole prompts; prompts then single tokens; prompts in portions down to two tokens; batches of
unequal requests that follow each other on the same slots and pages), in float32 and bfloat16, against the plain model."""
import copy

import numpy as np
import pytest
import torch

import helpers as H
import plain_zavevik as P
import zavevik_models as K

pytestmark = pytest.mark.gpu
DEV = "cuda"


def _t(a, dtype=torch.float32):
    return torch.from_numpy(np.ascontiguousarray(a)).to(DEV, dtype)


def _i(a):
    return torch.tensor(np.asarray(a).tolist(), dtype=torch.int32, device=DEV)


def _np(t):
    return t.double().cpu().numpy()


def _close(got, want, dtype, what, tol32=2e-5, tol16=1.2e-2):
    got, want = _np(got), np.asarray(want, dtype=np.float64)
    tol = tol32 if dtype == torch.float32 else tol16
    err = np.abs(got - want).max() / max(np.abs(want).max(), 1e-30)
    assert err <= tol, f"{what}: error {err:.3e} of the largest value exceeds {tol:.1e}"


# ---- a norm behind the sublayer with one number as gain, and nothing in front of the next one --------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("dim, n", [(52, 5), (50, 70), (3001, 9), (1, 3), (328, 33)])
def test_residual_is_handed_over_after_a_norm_behind_the_sublayer(dim, n, dtype):
    from rust_inference_b200.config.specs import NoNormSpec, PostNormSpec, RMSGainsSpec
    from rust_inference_b200.parts import BuildEnv, build_part
    env = BuildEnv(dtype, torch.device(DEV))
    rng = np.random.default_rng(dim)
    x, eps = (rng.standard_normal((n, dim)) * 3 + 1.0).astype(np.float32), 1e-4
    link = build_part("link", PostNormSpec(size=dim, eps=eps, gain_name="", scalar=True), env)
    link.load({"": _t(np.float32(1.7))})
    reader = build_part("norm", NoNormSpec(size=dim), env)
    resid = _t(x)
    first = reader(resid)                                             # nothing pending yet
    _close(first, x, dtype, "the residual itself", tol32=0.0, tol16=4e-3)
    assert torch.equal(resid, _t(x))
    y = _t(rng.standard_normal((n, dim)) * 4, dtype)
    got = reader(resid, link.pending(y))
    want = x + P.over_rms(_np(y), eps) * 1.7
    _close(resid, want, torch.float32, "new residual", tol32=2e-6)
    _close(got, want, dtype, "handed over", tol32=2e-6, tol16=4e-3)
    alone = _t(x[n - 1:])
    assert torch.equal(reader(alone, link.pending(y[n - 1:].contiguous())), got[n - 1:])      # a row alone: the same bits
    # the model's final norm over wanted rows
    last = build_part("norm", RMSGainsSpec(size=dim, eps=eps, scalar=True), env)
    last.load({"": _t(np.float32(0.6))})
    rows = last(_t(x), link.pending(y), _i([n - 1, 0]))
    _close(rows, (P.over_rms(want, eps) * 0.6)[[n - 1, 0]], dtype, "final norm", tol32=5e-6, tol16=6e-3)


# ---- unit-RMS queries, keys and values, the position's factor on the queries, the append ----------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("Dk, Dv, Dp, own", [(24, 40, 48, True), (20, 12, 32, True), (10, 6, 16, True), (22, 22, 22, True),
                                             (64, 128, 128, True), (96, 32, 96, False), (13, 13, 13, False)])
def test_preparation_of_queries_keys_and_values(Dk, Dv, Dp, own, dtype):
    from rust_inference_b200 import ops
    rng = np.random.default_rng(Dk + Dv)
    T, Hq, KV, eps = 9, 5, 2 if own else 0, 1e-2                    # (an eps that shows)
    def padded(heads, size):
        x = np.zeros((T, heads, Dp))
        x[:, :, :size] = rng.standard_normal((T, heads, size)) * 0.3
        return x.reshape(T, -1)
    proj = _t(np.concatenate([padded(Hq, Dk)] + ([padded(KV, Dk), padded(KV, Dv)] if own else []), axis=1), dtype)
    pos = [40 + t for t in range(T)]
    order = [2, 0, 1, 3]
    kp = torch.zeros((4, max(KV, 1), 32, Dp), dtype=dtype, device=DEV)
    vp = torch.zeros_like(kp)
    factor = np.asarray([P.query_factor(p, 0.8, 43) for p in range(64)])
    q = ops.qkv_prep(proj, 0, Hq * Dp if own else 0, (Hq + KV) * Dp if own else -1, Hq, KV, Dp, Dk, None, None, 0, False, True, eps,
                     kp if own else None, vp if own else None, _i(order).view(1, 4), _i([0] * T), _i(pos), _i([0]), write_kv=own,
                     q_factor=_t(factor), unit_v=True, Dv=Dv)
    x = _np(proj).reshape(T, -1, Dp)
    tol = dict(tol32=1e-5, tol16=6e-3)
    want = P.over_rms(x[:, :Hq, :Dk], eps) * factor[pos][:, None, None]
    _close(q[:, :, :Dk], want, dtype, "queries", **tol)
    assert torch.all(q[:, :, Dk:] == 0)
    for t, p in enumerate(pos if own else []):
        page = order[p // 32]
        _close(kp[page, :, p % 32, :Dk], P.over_rms(x[t, Hq:Hq + KV, :Dk], eps), dtype, "keys", **tol)
        _close(vp[page, :, p % 32, :Dv], P.over_rms(x[t, Hq + KV:, :Dv], eps), dtype, "values", **tol)
    assert torch.all(kp[order[0]] == 0) and torch.all(kp[order[3]] == 0)


# ---- attention with a distance bias -------------------------------------------------------------------------------------------------
def _paged(rng, k, v, page_size=32, spare=3):
    """Keys and values [n, KV, D] of one sequence in pools whose pages are in no order; slot 1 of 2."""
    n, KV, D = k.shape
    pages = -(-n // page_size)
    order = rng.permutation(pages + spare)[:pages]
    kp = torch.zeros((pages + spare, KV, page_size, D), dtype=k.dtype, device=DEV)
    vp = torch.zeros_like(kp)
    for p in range(n):
        kp[order[p // page_size], :, p % page_size] = k[p]
        vp[order[p // page_size], :, p % page_size] = v[p]
    table = torch.full((2, pages + 2), -1, dtype=torch.int32, device=DEV)
    table[1, :pages] = _i(order)
    return kp, vp, table


def _plain_biased(q, k, v, scale, cap, bias, positions):
    """q [m, H, D] at ``positions``; bias [H, distances]."""
    G = q.shape[1] // k.shape[1]
    out = np.zeros_like(q)
    for i, p in enumerate(positions):
        for h in range(q.shape[1]):
            s = (k[:p + 1, h // G] @ q[i, h]) * scale
            if cap:
                s = cap * np.tanh(s / cap)
            z = s + bias[h, np.minimum(p - np.arange(p + 1), bias.shape[1] - 1)]
            e = np.exp(z - z.max())
            out[i, h] = (e @ v[:p + 1, h // G]) / e.sum()
    return out


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("D, Hq, KV, rows, far, cap", [(32, 4, 2, 8, 33, 0.0), (80, 4, 4, 16, 500, 3.0), (64, 4, 2, 16, 90, 2.5),
                                                       (128, 4, 1, 12, 200, 0.0), (64, 20, 1, 6, 120, 6.0), (48, 3, 1, 2, 9, 1.5),
                                                       (128, 2, 2, 32, 64, 9.0), (64, 2, 1, 1, 5, 0.0), (22, 2, 1, 10, 70, 4.0)])
def test_attention_with_a_distance_bias(D, Hq, KV, rows, far, cap, dtype):
    """The bias of one row of the table stands out (its keys get nearly all the weight), a row per head, so that a border
    that is one distance off, or a bias that meets the cap or the scale, shows; as a whole prompt, as portions that start
    inside a block of keys, and token by token, on every attention kernel."""
    from rust_inference_b200 import ops
    from rust_inference_b200.parts.distance import bucket_starts, spread_over_distances
    rng = np.random.default_rng(D + rows)
    n, scale = 330, 0.25
    kt, vt, qt = (_t(rng.standard_normal((n, h, D)), dtype) for h in (KV, KV, Hq))
    rel = rng.standard_normal((rows, Hq))
    for h in range(Hq):
        rel[(rows // 2 + h) % rows, h] += 7.0                       # which row stands out differs from head to head
    starts = bucket_starts(rows, far)
    wide = ops.pad_distance_bias(spread_over_distances(_t(rel), far))
    bias = np.stack([[rel[P.distance_bucket(d, rows, far) if rows > 1 else 0, h] for d in range(n)] for h in range(Hq)])
    kp, vp, table = _paged(rng, kt, vt)
    args = (_np(qt), _np(kt), _np(vt), scale, cap)
    want = _plain_biased(*args, bias, range(n))
    slot = _i([1])
    tol = dict(tol32=3e-5, tol16=2e-2)
    fast = dtype == torch.bfloat16 and D % 16 == 0
    for first in (0, n - 100, n - 2):
        new = n - first
        start, length = _i([0, new]), _i([n])
        got = ops.attention(qt[first:].contiguous(), kp, vp, table, slot, start, length, new, scale, 0, softcap=cap, dist_bias=wide)
        _close(got, want[first:], dtype, f"rows kernel from {first}", **tol)
        if fast:
            got = ops.attention_prefill(qt[first:].contiguous(), kp, vp, table, slot, start, length, new, scale, 0, softcap=cap,
                                        dist_bias=wide)
            _close(got, want[first:], dtype, f"prefill kernel from {first}", **tol)
    edges = sorted({min(max(b + d, 0), n - 1) for b in starts[-3:] for d in (-1, 0, 1)} | {0, 31, 32, 127, 128, 129, n - 1})
    for p in edges:
        length = _i([p + 1])
        got = ops.attention(qt[p:p + 1].contiguous(), kp, vp, table, slot, _i([0, 1]), length, 1, scale, 0, softcap=cap, dist_bias=wide)
        _close(got, want[p:p + 1], dtype, f"rows kernel, token {p}", **tol)
        if fast:
            got = ops.attention_decode(qt[p:p + 1].contiguous(), kp, vp, table, slot, length, scale, 0, 1024, softcap=cap, dist_bias=wide)
            _close(got, want[p:p + 1], dtype, f"decode kernel, token {p}", **tol)
    if rows > 1:
        moved = _plain_biased(*args, np.concatenate([bias[:, 1:], bias[:, -1:]], axis=1), range(n))
        assert np.abs(moved - want).max() > 0.1 * np.abs(want).max(), "a border that is one distance off would not show"
    # without the bias: the kernels' other variant is as it was
    bare = _plain_biased(_np(qt)[n - 70:], *args[1:], np.zeros((Hq, 1)), range(n - 70, n))
    start, length = _i([0, 70]), _i([n])
    got = ops.attention(qt[n - 70:].contiguous(), kp, vp, table, slot, start, length, 70, scale, 0, softcap=cap)
    _close(got, bare, dtype, "rows kernel without a bias", **tol)
    if fast:
        got = ops.attention_prefill(qt[n - 70:].contiguous(), kp, vp, table, slot, start, length, 70, scale, 0, softcap=cap)
        _close(got, bare, dtype, "prefill kernel without a bias", **tol)


@pytest.mark.parametrize("D", [64, 48, 128])
def test_decode_with_a_distance_bias_over_a_batch(D):
    """One-token steps of sequences of very different lengths (the streaming kernel cuts their pages into runs), and the same
    sequences alone."""
    from rust_inference_b200 import ops
    rng = np.random.default_rng(D)
    lengths, Hq, KV, scale = [1, 33, 700, 32, 411], 4, 2, 0.3
    bias = rng.standard_normal((Hq, 130)) * 2.0
    wide = ops.pad_distance_bias(_t(bias))
    pages = sum(-(-n // 32) for n in lengths)
    kp = torch.zeros((pages, KV, 32, D), dtype=torch.bfloat16, device=DEV)
    vp = torch.zeros_like(kp)
    table = torch.full((len(lengths), 32), -1, dtype=torch.int32, device=DEV)
    ids, at, want, qs = rng.permutation(pages), 0, [], []
    for b, n in enumerate(lengths):
        k, v = _t(rng.standard_normal((n, KV, D)), torch.bfloat16), _t(rng.standard_normal((n, KV, D)), torch.bfloat16)
        q = _t(rng.standard_normal((1, Hq, D)), torch.bfloat16)
        mine = ids[at:at + -(-n // 32)]
        at += len(mine)
        table[b, :len(mine)] = _i(mine)
        for p in range(n):
            kp[mine[p // 32], :, p % 32], vp[mine[p // 32], :, p % 32] = k[p], v[p]
        qs.append(q)
        want.append(_plain_biased(_np(q), _np(k), _np(v), scale, 5.0, bias, [n - 1])[0])
    slots = list(range(len(lengths)))
    got = ops.attention_decode(torch.cat(qs), kp, vp, table, _i(slots), _i(lengths), scale, 0, 1024, softcap=5.0, dist_bias=wide)
    _close(got, np.stack(want), torch.bfloat16, "batch", tol16=2e-2)
    for b in slots:
        alone = ops.attention_decode(qs[b], kp, vp, table, _i([b]), _i([lengths[b]]), scale, 0, 1024, softcap=5.0, dist_bias=wide)
        _close(alone, want[b][None], torch.bfloat16, f"sequence {b} alone", tol16=2e-2)


# ---- the delta rule with one decay per head -------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("Hn, G, dim, vdim", [(4, 2, 12, 20), (2, 2, 136, 16), (1, 1, 64, 70), (3, 1, 200, 8), (1, 1, 300, 9), (2, 1, 32, 33),
                                              (2, 2, 128, 128), (1, 1, 1, 3)])
def test_delta_rule_with_one_decay_per_head(Hn, G, dim, vdim, dtype):
    """The recurrence over 75 tokens in one call, in pieces and token by token (the same bits, the same state), its decays as
    columns of a wider matrix."""
    from rust_inference_b200 import ops
    rng = np.random.default_rng(dim)
    T = 75
    C = 2 * G * dim + Hn * vdim
    qkv = rng.standard_normal((T, C)).astype(np.float32)
    wide = _t(np.concatenate([rng.standard_normal((T, 8 + Hn)), rng.standard_normal((T, Hn)) * 2.0 - 1.0], axis=1), dtype)
    dt_bias, a_log = rng.uniform(-2, 1, Hn), rng.uniform(-2, 1, Hn)
    z = wide[:, 8 + Hn:]
    def unit(x):
        return x / np.sqrt((x * x).sum(-1, keepdims=True) + P.UNIT_EPS)
    q = unit(qkv[:, :G * dim].astype(np.float64).reshape(T, G, dim)) * dim ** -0.5
    k = unit(qkv[:, G * dim:2 * G * dim].astype(np.float64).reshape(T, G, dim))
    v = qkv[:, 2 * G * dim:].astype(np.float64).reshape(T, Hn, vdim)
    beta = P.sigmoid(_np(wide)[:, 8:8 + Hn])
    g = np.exp(-np.exp(a_log) * P.softplus(_np(z) + dt_bias))
    want = np.stack([P.delta_rule(q[:, h // (Hn // G)], k[:, h // (Hn // G)], v[:, h], beta[:, h], g[:, h]) for h in range(Hn)], axis=1)

    def run(cuts, slot, S):
        ys, at = [], 0
        for c in cuts:
            part = wide[at:at + c].contiguous()
            ys.append(ops.delta_rule_recurrent(_t(qkv[at:at + c]), 0, G * dim, 2 * G * dim, part, 8, part[:, 8 + Hn:], _t(dt_bias),
                                               _t(a_log), dim ** -0.5, S, _i([slot]), _i([0, c]), Hn, G, dim, vdim, single=(c == 1)))
            at += c
        return torch.cat(ys)

    S = torch.zeros((3, Hn, dim, vdim), dtype=torch.float32, device=DEV)
    whole = run([T], 1, S)
    _close(whole, want, torch.float32, "whole", tol32=3e-5)
    kept = S[1].clone()
    assert torch.all(S[0] == 0) and torch.all(S[2] == 0)
    assert torch.equal(run([2, 1, 7, 33, 30, 2], 2, S), whole) and torch.equal(run([1] * T, 0, S), whole)
    assert torch.equal(S[2], kept) and torch.equal(S[0], kept)
    S[1].zero_()                                                     # a slot that is given out again starts from zeros
    assert torch.equal(run([T], 1, S), whole)
    # two sequences in one step, each alone
    S2 = torch.zeros_like(S)
    both = ops.delta_rule_recurrent(_t(qkv), 0, G * dim, 2 * G * dim, wide, 8, z, _t(dt_bias), _t(a_log), dim ** -0.5, S2, _i([2, 0]),
                                    _i([0, 40, T]), Hn, G, dim, vdim)
    assert torch.equal(both[:40], whole[:40]) and torch.all(S2[1] == 0)


# ---- experts by a table of token ids ----------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T, D, ff, E, top", [(1, 48, 24, 5, 2), (70, 52, 20, 3, 1), (300, 64, 40, 9, 4), (8, 64, 32, 16, 1), (3, 50, 10, 1, 1),
                                              (900, 64, 64, 4, 2), (900, 128, 48, 4, 1)])
def test_experts_by_a_table_against_the_plain_ones(T, D, ff, E, top, dtype):
    from rust_inference_b200.config.specs import GatedFFSpec, MoESpec
    from rust_inference_b200.parts import BuildEnv, StepContext, build_part
    rng = np.random.default_rng(T + E)
    vocab = 40
    spec = MoESpec(hidden_size=D, experts=E, top=top, expert=GatedFFSpec(D, ff, gate="silu"), route="table", table_rows=vocab)
    part = build_part("ffn", spec, BuildEnv(dtype, torch.device(DEV)))
    w = {"table": np.stack([rng.permutation(E)[:top] for _ in range(vocab)])}
    for e in range(E):
        for name, shape in (("gate", (ff, D)), ("up", (ff, D)), ("down", (D, ff))):
            w[f"e{e}.{name}"] = rng.standard_normal(shape) * 1.5 / np.sqrt(shape[1])
    tensors = {n: (_i(a) if n == "table" else _t(a, dtype)) for n, a in w.items()}
    part.load(tensors)
    ids = rng.integers(0, vocab, T)
    x = _t(rng.standard_normal((T, D)), dtype)
    ctx = StepContext(*([None] * 5), num_tokens=T, num_seqs=1, max_new=T, max_len=T, ids=_i(ids))
    got = part(x, ctx)
    plain = {n: (w["table"] if n == "table" else _np(t)) for n, t in tensors.items()}
    want = P.table_moe(_np(x), plain, {"router": {"top": top}}, ids)
    _close(got, want, dtype, "experts", tol32=2e-5, tol16=2e-2)
    alone = part(x[T - 1:].contiguous(), StepContext(*([None] * 5), num_tokens=1, num_seqs=1, max_new=1, max_len=T, ids=_i(ids[-1:])))
    if dtype == torch.float32:
        assert torch.equal(alone, got[T - 1:])
    if top > 1:
        other = dict(plain, table=np.roll(plain["table"], 1, axis=0))
        assert np.abs(P.table_moe(_np(x), other, {"router": {"top": top}}, ids) - want).max() > 0.1 * np.abs(want).max() or E == top


def test_a_table_that_names_no_expert_is_reported():
    """An entry past the experts is left out of the plan and reported through the error word (nothing is followed)."""
    from rust_inference_b200 import ops
    ops.error_flag(DEV).zero_()
    idx, (perm, tiles, meta, _) = ops.moe_plan_table(_i([1, 0, 1]), _i([[0, 1], [2, 5]]), 3)
    assert idx.tolist() == [[2, -1], [0, 1], [2, -1]] and meta.tolist()[1] == 4
    assert int(ops.error_flag(DEV).item()) == 8
    ops.error_flag(DEV).zero_()


# ---- the token-fed sublayer ---------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("D, dim", [(64, 32), (52, 12), (50, 5), (256, 64)])
def test_token_side_for_few_and_many_tokens(D, dim, dtype):
    from rust_inference_b200.config.specs import EmbeddingSpec, PostNormSpec, TokenSideSpec
    from rust_inference_b200.parts import BuildEnv, StepContext, build_part
    env = BuildEnv(dtype, torch.device(DEV))
    rng = np.random.default_rng(D)
    vocab, layers, i = 30, 3, 1
    emb = build_part("embedding", EmbeddingSpec(vocab, D, side_width=layers * dim), env)
    table = _t(rng.standard_normal((vocab, layers * dim)), dtype)
    emb.load({"weight": _t(rng.standard_normal((vocab, D)), dtype), "side": table})
    part = build_part("ffn", TokenSideSpec(hidden_size=D, size=dim, start=i * dim), env)
    w = {"gate": _t(rng.standard_normal((dim, D)) * 2 / np.sqrt(D), dtype), "proj": _t(rng.standard_normal((D, dim)) / np.sqrt(dim), dtype)}
    part.load(w)
    part.bind(emb)
    norm = rng.uniform(0.3, 1.5, D)
    link = build_part("link", PostNormSpec(size=D, eps=1e-5, gain_name="norm"), env)
    link.load({"norm": _t(norm)})
    for T in (1, 3, 12, 16, 20, 70):
        ids = rng.integers(0, vocab, T)
        x = _t(rng.standard_normal((T, D)), dtype)
        ctx = StepContext(*([None] * 5), num_tokens=T, num_seqs=1, max_new=T, max_len=T, ids=_i(ids))
        pend = link.pending(part(x, ctx))
        resid = _t(np.zeros((T, D)))
        from rust_inference_b200 import ops
        ops.rms_gains(resid, (), 0.0, dtype, terms=[(pend.y, pend.out)], post=pend.post)
        rows = _np(table)[ids][:, i * dim:(i + 1) * dim]
        want = P.token_side(_np(x), {"gate": _np(w["gate"]), "proj": _np(w["proj"]), "norm": norm}, rows, 1e-5)
        _close(resid, want, dtype, f"{T} tokens", tol32=2e-5, tol16=2.5e-2)
    with pytest.raises(ValueError, match="columns"):
        build_part("ffn", TokenSideSpec(hidden_size=D, size=dim, start=3 * dim), env).bind(emb)


# ---- whole models ------------------------------------------------------------------------------------------------------------------------
def _portions(reqs, sizes):
    """Each request alone, its prompt brought in portions of ``sizes`` tokens (repeated), every position wanted."""
    steps, n = [], 0
    for rid, toks in reqs.items():
        at, j = 0, 0
        while at < len(toks):
            c = min(sizes[j % len(sizes)], len(toks) - at)
            steps.append({"step": n, "entries": [{"id": rid, "tokens": toks[at:at + c], "want": list(range(c))}],
                          "end": [rid] if at + c == len(toks) else []})
            at, j, n = at + c, j + 1, n + 1
    return steps


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_replay_in_five_cuttings_matches_plain(tmp_path, name, dtype):
    d, config, weights = K.make_model_dir(tmp_path, name, seed=3)
    rng = np.random.default_rng(4)
    reqs = H.random_requests(rng, config["vocab"], [5, 1, 23, 150, 2, 70, 37])
    want = K.plain_logits(config, weights, reqs)
    by_cutting = {}
    for label, steps in (("whole", H.trace_whole(reqs)), ("tail", H.trace_tail(reqs, tail=40)),
                         ("portions", _portions(reqs, [2, 7, 1, 33, 2])), ("pairs", _portions(reqs, [2])),
                         ("batches", H.trace_batches(reqs, 3, [6, 0, 9, 3, 70, 1, 36]))):
        out = str(tmp_path / f"out_{label}")
        H.replay_inprocess(d, dtype, steps, out, device="cuda:0")
        rows = H.collect(steps, out, config["vocab"])
        assert len(rows) == sum(len(t) for t in reqs.values())
        K.assert_rows_close(rows, want, dtype, f"{name} {label} {dtype}")
        by_cutting[label] = rows
    if dtype == "float32":
        H.assert_rows_identical(by_cutting, f"{name} float32")


@pytest.mark.parametrize("kind", ["attention", "borrowed", "delta", "experts"])
def test_one_layer_of_each_kind_alone(tmp_path, kind):
    """Models in which one mechanism decides the logits, without a token-fed sublayer."""
    own = K.attn(6, 3, 20, 36, scale=0.6, cap=8.0, temp=(0.9, 16), far=50, rows=8)
    layers = {"attention": [K.layer("attention", own, None)],
              "borrowed": [K.layer("attention", own, None),
                           K.layer("attention", dict(own, kv_from=0, scale=0.9, softcap=2.0, bias_rows=12, bias_max=80), None)],
              "delta": [K.layer("delta", K.delta(4, 2, 40, 12, 5), None)],
              "experts": [K.layer("delta", K.delta(1, 1, 4, 4, 1), K.moe(11, 2, 36))]}[kind]
    config = {"architecture": "Zavevik", "vocab": 77, "width": 44, "norm": {"eps": 1e-5}, "layers": layers}
    weights = K.make_weights(config, 11)
    d = K.write_model(str(tmp_path / kind), config, weights)
    reqs = H.random_requests(np.random.default_rng(12), config["vocab"], [90, 3, 41])
    want = K.plain_logits(config, weights, reqs)
    for label, steps in (("whole", H.trace_whole(reqs)), ("tail", H.trace_tail(reqs, tail=60)), ("pairs", _portions(reqs, [2]))):
        out = str(tmp_path / f"out_{label}")
        H.replay_inprocess(d, "float32", steps, out, device="cuda:0")
        K.assert_rows_close(H.collect(steps, out, config["vocab"]), want, "float32", f"{kind} {label}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("far", [0, 31, 32, 95, 96, 255])
def test_a_far_key_among_hundreds_is_found(tmp_path, far, dtype):
    """A layer whose queries and keys copy the input, and a second one that borrows its keys and values: the last token
    repeats the token at position ``far`` (a page's first or last place among them), and nothing else in 300 tokens looks like
    it, so both outputs are that token's value (and its own).  As the last token of a prompt and as a token decoded alone."""
    D, d = 32, 16
    m = K.attn(2, 1, d, d, scale=2.0, far=64, rows=8)
    config = {"architecture": "Zavevik", "vocab": 400, "width": D, "norm": {"eps": 1e-6},
              "layers": [K.layer("attention", m, None), K.layer("attention", dict(m, kv_from=0), None)]}
    W = K.make_weights(config, 21)
    eye = np.concatenate([np.eye(d), np.zeros((d, D - d))], axis=1)
    for p in ("l0.", "l1."):
        W[p + "mix.q"] = K._bf16(np.concatenate([eye, eye]))
        rel = np.zeros((8, 2))
        rel[0] = -6.0                                              # a token's own key counts for little
        W[p + "mix.rel"] = K._bf16(rel)
        W[p + "norm1"] = K._bf16(np.float32(0.25))
    W["l0.mix.k"] = K._bf16(eye)
    folder = K.write_model(str(tmp_path / "far"), config, W)
    rng = np.random.default_rng(far)
    toks = [int(t) for t in rng.permutation(399)[:300] + 1]
    toks[far] = 0
    toks.append(0)
    reqs = {"r": toks}
    W64 = K.as64(W)
    want = {"r": P.forward(config, W64, toks)[0]}
    unit = P.over_rms(W64["embed"][toks][:, :d], 1e-6)
    s = (unit @ unit[-1]) * 2.0
    s[-1] -= 6.0
    w = np.exp(s - s.max())
    assert (w / w.sum())[far] > 0.3, "the far key does not stand out: the test would not see it missing"
    for label, steps in (("prompt", H.trace_whole(reqs)), ("decoded", H.trace_tail(reqs, tail=3))):
        out = str(tmp_path / f"out_{label}")
        H.replay_inprocess(folder, dtype, steps, out, device="cuda:0")
        rows = H.collect(steps, out, config["vocab"])
        err = K.row_error(rows[("r", 300)], want["r"][300])
        assert err < (1e-4 if dtype == "float32" else 8e-2), f"{label}: error {err:.3e}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "C"])
def test_long_decoding_through_page_edges(tmp_path, name, dtype):
    """A short prompt, then 260 tokens one by one (graph replays) against the plain model; two sequences of unequal
    length whose states and pages live side by side."""
    d, config, weights = K.make_model_dir(tmp_path, name, seed=6)
    rng = np.random.default_rng(7)
    reqs = H.random_requests(rng, config["vocab"], [270, 200])
    want = K.plain_logits(config, weights, reqs)
    steps = H.trace_batches(reqs, 2, [260, 195])
    out = str(tmp_path / "out")
    H.replay_inprocess(d, dtype, steps, out, device="cuda:0", max_tokens=640)
    K.assert_rows_close(H.collect(steps, out, config["vocab"]), want, dtype, f"long decoding {name} {dtype}")


def test_a_batch_of_twenty_decodes_as_each_alone(tmp_path):
    """More sequences than the mma.sync linears take at once (the tcgen05 products, the gate and the token's row after the
    product), in bfloat16, against the plain model."""
    d, config, weights = K.make_model_dir(tmp_path, "C", seed=16)
    rng = np.random.default_rng(17)
    reqs = H.random_requests(rng, config["vocab"], [3 + 2 * i for i in range(20)])
    want = K.plain_logits(config, weights, reqs)
    steps = H.trace_batches(reqs, 20, [2])
    out = str(tmp_path / "out")
    H.replay_inprocess(d, "bfloat16", steps, out, device="cuda:0")
    K.assert_rows_close(H.collect(steps, out, config["vocab"]), want, "bfloat16", "twenty sequences")


def test_greedy_generation_with_more_requests_than_slots(tmp_path):
    import rust_inference_b200 as ri
    d, config, weights = K.make_model_dir(tmp_path, "A", seed=8)
    W = K.as64(weights)
    rng = np.random.default_rng(9)
    prompts = [[int(t) for t in rng.integers(0, config["vocab"], n)] for n in (3, 1, 9, 40, 2)]
    llm = ri.LLM(d, dtype="float32", max_pages=32, pages_per_seq=4, max_seqs=2)
    got = llm.generate(prompts, max_new_tokens=12)
    assert llm.engine.graph_replays > 0
    for p, g in zip(prompts, got):
        seq = list(p)
        for _ in range(12):
            seq.append(int(np.argmax(P.forward(config, W, seq)[0][-1])))
        assert g == seq[len(p):]


def test_random_model_of_the_design_generates():
    """Weights made on the device, no file: the tables name every expert and the greedy loop runs."""
    from rust_inference_b200.engine import Engine, Entry, Model
    model = Model.from_random(copy.deepcopy(K.CFG_C), seed=1, dtype="bfloat16", device="cuda:0")
    table = model.blocks[0].ffn.table
    assert int(table.min()) == 0 and int(table.max()) == 15
    engine = Engine(model, max_tokens=256, max_seqs=2)
    s = engine.new_sequence()
    logits = engine.step([Entry(s, [5, 9, 200])])
    assert torch.isfinite(logits).all() and float(logits.std()) > 0
    engine.check_device_errors()
