"""Gotulorn on the GPU: each kernel against the plain formulas of tests/plain_gotulorn.py, then whole models through trace
replay in several cuttings (whole prompts; prompts then single tokens; prompts in portions down to two tokens; batches of
unequal requests that follow each other on the same slots and pages), in float32 and bfloat16, against the plain model."""
import copy

import numpy as np
import pytest
import torch

import gotulorn_models as K
import helpers as H
import plain_gotulorn as P

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


def _no_error():
    from rust_inference_b200 import ops
    assert int(ops.error_flag(DEV).item()) == 0


# ---- Dynamic Tanh ---------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("dim, n", [(52, 5), (50, 70), (3001, 9), (1, 3), (1024, 33), (1028, 2)])
def test_dynamic_tanh_takes_in_what_is_pending(dim, n, dtype):
    from rust_inference_b200.config.specs import DynTanhSpec, PostNormSpec
    from rust_inference_b200.parts import BuildEnv, build_part
    env = BuildEnv(dtype, torch.device(DEV))
    rng = np.random.default_rng(dim)
    x, g, b, a = rng.standard_normal((n, dim)) * 3, rng.uniform(0.5, 1.5, dim), rng.standard_normal(dim), 0.7
    part = build_part("norm", DynTanhSpec(size=dim), env)
    part.load({"": _t(g), ".b": _t(b), ".alpha": _t(np.float32(a))})
    resid = _t(x)
    x64 = _np(resid)
    _close(part(resid), P.bent(x64, g, b, a), dtype, "alone", tol32=2e-6, tol16=5e-3)
    assert torch.equal(resid, _t(x))
    y = _t(rng.standard_normal((n, dim)) * 2, dtype)
    want = x64 + _np(y)
    rows = part(_t(x), y, _i([n - 1, 0]))
    _close(rows, P.bent(want, g, b, a)[[n - 1, 0]], dtype, "chosen rows", tol32=3e-6, tol16=5e-3)
    got = part(resid, y)
    _close(resid, want, torch.float32, "new residual", tol32=1e-6)
    _close(got, P.bent(want, g, b, a), dtype, "with an output pending", tol32=3e-6, tol16=5e-3)
    assert torch.equal(got[n - 1], rows[0]) and torch.equal(part(_t(x[n - 1:]), y[n - 1:].contiguous()), got[n - 1:])
    # behind a link that norms the output first, or weighs it: joined in front, by the kernel that other norms use
    link = build_part("link", PostNormSpec(size=dim, eps=1e-3, gain_name="", scalar=True), env)
    link.load({"": _t(np.float32(1.3))})
    resid = _t(x)
    got = part(resid, link.pending(y))
    want = x64 + P.over_rms(_np(y), 1e-3) * 1.3
    _close(resid, want, torch.float32, "residual behind a link", tol32=3e-6)
    _close(got, P.bent(want, g, b, a), dtype, "behind a link", tol32=5e-6, tol16=5e-3)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("dim, n", [(52, 5), (50, 70), (3001, 4), (1024, 33)])
def test_normed_embedding(dim, n, dtype):
    from rust_inference_b200 import ops
    from rust_inference_b200.config.specs import DynTanhSpec, EmbeddingSpec, RMSGainsSpec
    from rust_inference_b200.parts import BuildEnv, build_part
    env = BuildEnv(dtype, torch.device(DEV))
    rng = np.random.default_rng(dim)
    g, b, a, s = rng.uniform(0.5, 1.5, dim), rng.standard_normal(dim), 0.4, 3.5
    table = _t(rng.standard_normal((40, dim)), dtype)
    ids = rng.integers(0, 40, n)
    part = build_part("embedding", EmbeddingSpec(40, dim, scale=s, norm=DynTanhSpec(size=dim)), env)
    part.load({"weight": table, "norm": _t(g), "norm.b": _t(b), "norm.alpha": _t(np.float32(a))})
    got = part(_i(ids))
    assert got.dtype == torch.float32
    _close(got, P.bent(_np(table)[ids] * s, g, b, a), torch.float32, "rows", tol32=2e-6)
    # another kind of norm in the same place
    part = build_part("embedding", EmbeddingSpec(40, dim, scale=s, norm=RMSGainsSpec(size=dim, eps=1e-3)), env)
    part.load({"weight": table, "norm": _t(g)})
    got = part(_i(ids))
    assert got.dtype == torch.float32
    _close(got, P.over_rms(_np(table)[ids] * s, 1e-3) * g, torch.float32, "rows behind an RMS norm", tol32=3e-6)
    _no_error()
    ops.embed_dyn_tanh(_i([1, 40]), table, s, _t([a]), _t(g), _t(b))                 # an id outside the table is reported
    assert int(ops.error_flag(DEV).item()) == 1
    ops.error_flag(DEV).zero_()


# ---- a window beside kept first tokens ---------------------------------------------------------------------------------------------
def _paged(rng, k, v, sees_any, page_size=32, spare=3):
    """Keys and values [n, KV, D] of one sequence in pools whose pages are in no order (slot 1 of 2); pages of which no key is
    seen are unmapped, and whatever no key was written to holds NaN."""
    n, KV, D = k.shape
    pages = -(-n // page_size)
    order = rng.permutation(pages + spare)[:pages]
    kp = torch.full((pages + spare, KV, page_size, D), float("nan"), dtype=k.dtype, device=DEV)
    vp = torch.full_like(kp, float("nan"))
    table = torch.full((2, pages + 2), -1, dtype=torch.int32, device=DEV)
    for page in range(pages):
        keys = range(page * page_size, min(n, (page + 1) * page_size))
        if not any(sees_any[j] for j in keys):
            continue
        table[1, page] = int(order[page])
        m = len(keys)
        kp[order[page], :, :m] = k[keys[0]:keys[0] + m].transpose(0, 1)
        vp[order[page], :, :m] = v[keys[0]:keys[0] + m].transpose(0, 1)
    return kp, vp, table


def _plain_masked(q, k, v, scale, mask, positions):
    G = q.shape[1] // k.shape[1]
    out = np.zeros((len(positions),) + q.shape[1:])
    for i, p in enumerate(positions):
        j = P.sees(p, mask)
        for h in range(q.shape[1]):
            out[i, h] = P.weighted((k[j, h // G] @ q[p, h]) * scale, v[j, h // G])
    return out


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("D, Hq, KV, size, keep", [(32, 4, 2, 43, 7), (80, 4, 4, 1, 1), (64, 4, 2, 70, 33), (128, 4, 1, 64, 64),
                                                   (64, 20, 1, 31, 3), (48, 3, 1, 200, 129), (128, 2, 2, 129, 0), (64, 2, 1, 33, 300),
                                                   (22, 2, 1, 50, 32), (176, 6, 2, 45, 5), (128, 8, 2, 300, 1)])
def test_attention_with_kept_first_tokens(D, Hq, KV, size, keep, dtype):
    """A query that sees one of the loud keys hears nothing else: they stand further apart than the window is long, the first one
    right behind the kept tokens, and the last kept token is loud where none of them is in sight, so that one key too many or
    too few at either edge shows.  As a whole prompt, as portions that start inside a block of keys, and token by token
    around pages, blocks and the mask's edges, on every attention kernel; pages that nobody sees are not mapped."""
    from rust_inference_b200 import ops
    rng = np.random.default_rng(D + size)
    n, scale, mask = 420, 0.25, {"size": size, "keep_first": keep}
    k, v, q = (rng.standard_normal((n, h, D)) for h in (KV, KV, Hq))
    q, k = q * 1.5 * D ** -0.25, k * 1.5 * D ** -0.25
    q[..., 0], k[..., 0] = 3.0, 0.0
    if keep:
        k[keep - 1, :, 0] = 7.0
    k[keep::size + 3, :, 0] = 13.0
    kt, vt, qt = _t(k, dtype), _t(v, dtype), _t(q, dtype)
    args = (_np(qt), _np(kt), _np(vt), scale)
    want = _plain_masked(*args, mask, range(n))
    slot, tol, fast = _i([1]), dict(tol32=3e-5, tol16=2e-2), dtype == torch.bfloat16 and D % 16 == 0
    for first in (0, n - 290, n - 100, n - 2):
        seen = np.zeros(n, bool)
        for p in range(first, n):
            seen[P.sees(p, mask)] = True
        kp, vp, table = _paged(rng, kt, vt, seen)
        new = n - first
        start, length, part = _i([0, new]), _i([n]), qt[first:].contiguous()
        got = ops.attention(part, kp, vp, table, slot, start, length, new, scale, size, keep=keep)
        _close(got, want[first:], dtype, f"rows kernel from {first}", **tol)
        if fast:
            got = ops.attention_prefill(part, kp, vp, table, slot, start, length, new, scale, size, keep=keep)
            _close(got, want[first:], dtype, f"prefill kernel from {first}", **tol)
    edges = {e + d for e in (keep, size, keep + size, 2 * size, 32, 64, 128, 256, keep + size + 31) for d in (-2, -1, 0, 1)}
    for p in sorted(e for e in edges | {0, n - 1} if 0 <= e < n):
        seen = np.zeros(n, bool)
        seen[P.sees(p, mask)] = True
        kp, vp, table = _paged(rng, kt[:p + 1], vt[:p + 1], seen)
        length, one = _i([p + 1]), qt[p:p + 1].contiguous()
        got = ops.attention(one, kp, vp, table, slot, _i([0, 1]), length, 1, scale, size, keep=keep)
        _close(got, want[p:p + 1], dtype, f"rows kernel, token {p}", **tol)
        if fast:
            got = ops.attention_decode(one, kp, vp, table, slot, length, scale, size, 1024, keep=keep)
            _close(got, want[p:p + 1], dtype, f"decode kernel, token {p}", **tol)
            got = ops.attention_prefill(one, kp, vp, table, slot, _i([0, 1]), length, 1, scale, size, keep=keep)
            _close(got, want[p:p + 1], dtype, f"prefill kernel, token {p}", **tol)
    _no_error()
    masks = [{"size": size + 1, "keep_first": keep}, {"size": size, "keep_first": keep + 1}]
    masks += [{"size": size - 1, "keep_first": keep}] if size > 1 else []
    masks += [{"size": size, "keep_first": keep - 1}] if keep else []
    for off in masks:
        if keep + size + 8 < n:
            moved = _plain_masked(*args, off, range(n))
            assert np.abs(moved - want).max() > 0.1 * np.abs(want).max(), "an edge that is one token off would not show"


@pytest.mark.parametrize("D, Hq, KV, size, keep", [(64, 4, 2, 40, 35), (48, 4, 2, 70, 3), (128, 8, 1, 100, 64), (128, 40, 2, 33, 5)])
@pytest.mark.parametrize("lengths", [[1, 33, 700, 32, 411], [5 + 17 * i for i in range(40)]])
def test_decode_with_kept_tokens_over_a_batch(D, Hq, KV, size, keep, lengths):
    """One-token steps of sequences of very different lengths (the streaming kernel cuts their visible pages into runs), more
    of them than a warp has lanes; and prompts of very different lengths in one step."""
    from rust_inference_b200 import ops
    rng = np.random.default_rng(D + len(lengths))
    scale, mask = 0.3, {"size": size, "keep_first": keep}
    pages = sum(-(-n // 32) for n in lengths)
    kp = torch.zeros((pages, KV, 32, D), dtype=torch.bfloat16, device=DEV)
    vp = torch.zeros_like(kp)
    table = torch.full((len(lengths), 32), -1, dtype=torch.int32, device=DEV)
    ids, at, want, qs, wants = rng.permutation(pages), 0, [], [], []
    for b, n in enumerate(lengths):
        k, v, q = (_t(rng.standard_normal((n, h, D)), torch.bfloat16) for h in (KV, KV, Hq))
        mine = ids[at:at + -(-n // 32)]
        at += len(mine)
        table[b, :len(mine)] = _i(mine)
        for j, page in enumerate(mine):
            m = min(32, n - 32 * j)
            kp[page, :, :m], vp[page, :, :m] = k[32 * j:32 * j + m].transpose(0, 1), v[32 * j:32 * j + m].transpose(0, 1)
        qs.append(q)
        want.append(_plain_masked(_np(q), _np(k), _np(v), scale, mask, [n - 1])[0])
        if len(lengths) < 8:
            wants.append(_plain_masked(_np(q), _np(k), _np(v), scale, mask, range(n)))
    slots = list(range(len(lengths)))
    last = torch.stack([q[-1] for q in qs])
    got = ops.attention_decode(last, kp, vp, table, _i(slots), _i(lengths), scale, size, 1024, keep=keep)
    _close(got, np.stack(want), torch.bfloat16, "batch", tol16=2e-2)
    for b in slots[:6]:
        alone = ops.attention_decode(last[b:b + 1].contiguous(), kp, vp, table, _i([b]), _i([lengths[b]]), scale, size, 1024, keep=keep)
        _close(alone, want[b][None], torch.bfloat16, f"sequence {b} alone", tol16=2e-2)
    if wants:
        start = np.concatenate([[0], np.cumsum(lengths)])
        got = ops.attention_prefill(torch.cat(qs), kp, vp, table, _i(slots), _i(start), _i(lengths), max(lengths), scale, size, keep=keep)
        _close(got, np.concatenate(wants), torch.bfloat16, "prompts together", tol16=2e-2)
    _no_error()


# ---- differential attention -----------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("Hq, dim, Dp, KV", [(3, 12, 48, 2), (5, 5, 16, 5), (4, 32, 64, 2), (2, 64, 128, 0), (1, 17, 48, 1), (2, 11, 22, 1)])
def test_queries_of_two_maps_get_rows_of_their_own(Hq, dim, Dp, KV, dtype):
    from rust_inference_b200 import ops
    rng = np.random.default_rng(dim)
    T, dv = 9, min(Dp, dim + 3)

    def padded(heads, size):
        x = np.zeros((T, heads, Dp))
        x[:, :, :size] = rng.standard_normal((T, heads, size))
        return x.reshape(T, -1)
    proj = _t(np.concatenate([padded(Hq, 2 * dim)] + ([padded(KV, 2 * dim), padded(KV, dv)] if KV else []), axis=1), dtype)
    pos, order = [28 + t for t in range(T)], [2, 0, 1, 3]
    kp = torch.zeros((4, max(KV, 1), 32, Dp), dtype=dtype, device=DEV)
    vp = torch.zeros_like(kp)
    q = ops.qkv_prep(proj, 0, Hq * Dp if KV else 0, (Hq + KV) * Dp if KV else -1, Hq, KV, Dp, 2 * dim, None, None, 0, False, False, 0.0,
                     kp if KV else None, vp if KV else None, _i(order).view(1, 4), _i([0] * T), _i(pos), _i([0]), write_kv=KV > 0,
                     Dv=dv, maps=2)
    x = proj.view(T, -1, Dp)
    want = torch.zeros((T, Hq, 2, Dp), dtype=dtype, device=DEV)
    want[:, :, 0, :dim], want[:, :, 1, dim:2 * dim] = x[:, :Hq, :dim], x[:, :Hq, dim:2 * dim]
    assert torch.equal(q, want.view(T, 2 * Hq, Dp))
    for t, p in enumerate(pos if KV else []):
        assert torch.equal(kp[order[p // 32], :, p % 32], x[t, Hq:Hq + KV]) and torch.equal(vp[order[p // 32], :, p % 32], x[t, Hq + KV:])


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T, Hq, Dp, vdim, width", [(1, 2, 48, 36, 48), (70, 3, 128, 128, 128), (9, 1, 64, 33, 48), (5, 4, 22, 13, 16),
                                                    (300, 2, 16, 3, 16), (3, 2, 272, 270, 272), (6, 5, 256, 200, 208), (2, 1, 512, 512, 512)])
def test_pairs_of_maps_are_put_together(T, Hq, Dp, vdim, width, dtype):
    from rust_inference_b200 import ops
    rng = np.random.default_rng(Dp)
    x = _t(rng.standard_normal((T, 2 * Hq, Dp)), dtype)             # (padding columns too: they must not count)
    lam, eps, gain = 0.83, 1e-2, 0.37
    got = ops.pair_heads(x, lam, eps, gain, width, vdim)
    a = _np(x)[:, :, :vdim]
    _close(got[:, :, :vdim], P.over_rms(a[:, 0::2] - lam * a[:, 1::2], eps) * gain, dtype, "pairs", tol32=3e-6, tol16=5e-3)
    assert torch.all(got[:, :, vdim:] == 0) and got.shape == (T, Hq, width)
    assert torch.equal(ops.pair_heads(x[T - 1:].contiguous(), lam, eps, gain, width, vdim), got[T - 1:])
    if dtype == torch.float32:                                      # float32 results of an attention kernel, rounded once
        got = ops.pair_heads(x, lam, eps, gain, width, vdim, out_dtype=torch.bfloat16)
        _close(got[:, :, :vdim], P.over_rms(a[:, 0::2] - lam * a[:, 1::2], eps) * gain, torch.bfloat16, "rounded", tol16=5e-3)
        assert torch.all(got[:, :, vdim:] == 0) and got.dtype == torch.bfloat16


@pytest.mark.parametrize("D, dim, vdim, Hq, KV, size, keep", [(128, 64, 128, 8, 2, 200, 4), (64, 32, 64, 2, 1, 0, 0), (128, 20, 120, 4, 4, 70, 40), (64, 30, 33, 6, 1, 33, 1),
                                                              (96, 40, 88, 6, 2, 45, 7), (128, 60, 17, 2, 2, 129, 128), (48, 17, 34, 20, 1, 64, 3)])
def test_attention_kernels_put_pairs_together(D, dim, vdim, Hq, KV, size, keep):
    """Prompts and portions of very different lengths in one step, then one token each: every bfloat16 kernel with the two maps
    put together in float32, against the plain formulas; the pieces a sequence falls into do not depend on the others."""
    from rust_inference_b200 import ops
    rng = np.random.default_rng(D + dim)
    lengths, news = [300, 1, 45, 129, 460, 77], [300, 1, 2, 129, 130, 33]
    scale, lam, eps, gain, width = 0.4, 0.7, 1e-3, 0.6, -(-vdim // 16) * 16
    mask = {"size": size, "keep_first": keep} if size else None
    pages = sum(-(-n // 32) for n in lengths)
    kp = torch.zeros((pages, KV, 32, D), dtype=torch.bfloat16, device=DEV)
    vp = torch.zeros_like(kp)
    table = torch.full((len(lengths), 16), -1, dtype=torch.int32, device=DEV)
    ids, at, qs, want = rng.permutation(pages), 0, [], []
    for b, n in enumerate(lengths):
        k, v, q = (_t(rng.standard_normal((n, h, d)), torch.bfloat16) for h, d in ((KV, 2 * dim), (KV, vdim), (2 * Hq, dim)))
        mine = ids[at:at + -(-n // 32)]
        at += len(mine)
        table[b, :len(mine)] = _i(mine)
        for j, page in enumerate(mine):
            m = min(32, n - 32 * j)
            kp[page, :, :m, :2 * dim] = k[32 * j:32 * j + m].transpose(0, 1)
            vp[page, :, :m, :vdim] = v[32 * j:32 * j + m].transpose(0, 1)
        rows = torch.zeros((n, Hq, 2, D), dtype=torch.bfloat16, device=DEV)
        rows[:, :, 0, :dim], rows[:, :, 1, dim:2 * dim] = q[:, 0::2], q[:, 1::2]
        qs.append(rows.view(n, 2 * Hq, D)[n - news[b]:])
        k64, v64, q64, out = _np(k).reshape(n, KV, 2, dim), _np(v), _np(q).reshape(n, Hq, 2, dim), []
        for p in range(n - news[b], n):
            j = P.sees(p, mask)
            for h in range(Hq):
                g = h // (Hq // KV)
                one, two = (P.weighted((k64[j, g, t] @ q64[p, h, t]) * scale, v64[j, g]) for t in (0, 1))
                out.append(P.over_rms(one - lam * two, eps) * gain)
        want.append(np.asarray(out).reshape(news[b], Hq, vdim))
    pair = (lam, eps, gain, width, vdim)
    start = np.concatenate([[0], np.cumsum(news)])
    slots = list(range(len(lengths)))
    got = ops.attention_prefill(torch.cat(qs), kp, vp, table, _i(slots), _i(start), _i(lengths), max(news), scale, size, keep=keep,
                                pair=pair, pair_dim=dim)
    assert got.shape == (sum(news), Hq, width) and torch.all(got[:, :, vdim:] == 0)
    _close(got[:, :, :vdim], np.concatenate(want), torch.bfloat16, "prompts together", tol16=3e-2)
    for b in slots:
        alone = ops.attention_prefill(qs[b].contiguous(), kp, vp, table, _i([b]), _i([0, news[b]]), _i([lengths[b]]), news[b], scale, size,
                                      keep=keep, pair=pair, pair_dim=dim)
        assert torch.equal(alone, got[start[b]:start[b + 1]]), f"sequence {b} alone"
    last = torch.cat([q[-1:] for q in qs])
    got = ops.attention_decode(last, kp, vp, table, _i(slots), _i(lengths), scale, size, 1024, keep=keep, pair=pair)
    assert torch.all(got[:, :, vdim:] == 0)
    _close(got[:, :, :vdim], np.stack([w[-1] for w in want]), torch.bfloat16, "one token each", tol16=3e-2)
    _no_error()


def _mixer(spec, dtype, w):
    from rust_inference_b200.parts import BuildEnv, build_part, part_class
    env = BuildEnv(dtype, torch.device(DEV))
    part = build_part("mixer", spec, env)
    infos = part_class("mixer", spec).param_infos(spec)
    tensors = {n: _t(w[n], dtype if i.role == "matrix" else torch.float32) for n, i in infos.items()}
    part.load(tensors)
    part.prepare(512)
    return part, {n: _np(t) for n, t in tensors.items()}


def _contexts(cuts):
    """One sequence in slot 1 brought in ``cuts``; (first token, context) each."""
    from rust_inference_b200.parts import StepContext
    at = 0
    for c in cuts:
        yield at, StepContext(tok_seq=_i([0] * c), tok_pos=_i(range(at, at + c)), seq_slot=_i([1]), seq_start=_i([0, c]),
                              seq_len=_i([at + c]), num_tokens=c, num_seqs=1, max_new=c, max_len=at + c)
        at += c


def _run_mixer(part, x, cuts, lender=None):
    """The mixer over x in pieces on a fresh cache whose pages are in no order (``lender``: a part that writes the entry)."""
    from rust_inference_b200.cache.kv_cache import LayerCache
    req = (lender or part).cache_request()
    pages = -(-x.shape[0] // 32)
    order = np.random.default_rng(0).permutation(pages + 2)[:pages]
    kp = torch.full((pages + 2, req.kv_heads, 32, req.head_dim), float("nan"), dtype=x.dtype, device=DEV)
    vp = kp if req.shared_kv else torch.full_like(kp, float("nan"))
    table = torch.full((2, pages), -1, dtype=torch.int32, device=DEV)
    table[1] = _i(order)
    out = []
    for at, ctx in _contexts(cuts):
        piece = x[at:at + ctx.num_tokens].contiguous()
        if lender is not None:
            lender(piece, ctx, LayerCache(kp, vp, table, 32, None, True))
        out.append(part(piece, ctx, LayerCache(kp, vp, table, 32, None, lender is None)))
    return torch.cat(out)


CUTS = ([150], [2] * 75, [90] + [1] * 60, [1] * 150, [33, 31, 1, 64, 21])


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("mixer", [K.attn(4, 2, 12, 36, 17, 3, diff=0.3), K.attn(3, 1, 32, 64, 40, 33, diff=0.6), K.attn(8, 1, 64, 128, 64, 6),
                                   K.attn(2, 2, 20, 12), K.attn(20, 1, 32, 40, 50, 2), K.attn(2, 1, 9, 7, 1, 1, diff=0.0),
                                   K.attn(2, 1, 100, 272, 33, 2)])
def test_differential_attention_alone(mixer, dtype):
    """The mixer, and a second one with other heads, another mask and other constants that borrows its keys and values."""
    from rust_inference_b200.models.gotulorn import GotulornConfig
    other = dict(mixer, heads=2 * mixer["kv_heads"], diff=0.9, scale=0.7 * mixer["scale"], mask={"size": 61, "keep_first": 1}, kv_from=0)
    config = K.config_of(11, 64, 1.0, 1e-3, [K.layer("a", mixer, None), K.layer("a", other, None)])
    W = K.make_weights(config, 7)
    spec = GotulornConfig.from_dict(config).to_spec()
    part, w = _mixer(spec.layers[0].mixer, dtype, {n[len("l0.mix."):]: t for n, t in W.items() if n.startswith("l0.mix.")})
    borrower, w2 = _mixer(spec.layers[1].mixer, dtype, {n[len("l1.mix."):]: t for n, t in W.items() if n.startswith("l1.mix.")})
    x = _t(np.random.default_rng(8).standard_normal((150, 64)), dtype)
    k, v = P.keys_and_values(_np(x), w, mixer)
    want, want2 = P.paired_attention(_np(x), w, mixer, 1e-3, k, v), P.paired_attention(_np(x), w2, other, 1e-3, k, v)
    first = None
    for cuts in CUTS:
        got = _run_mixer(part, x, cuts)
        _close(got, want, dtype, f"cut {cuts[:3]}", tol32=2e-5, tol16=4e-2)
        first = got if first is None else first
        if dtype == torch.float32:
            assert torch.equal(got, first)
        _close(_run_mixer(borrower, x, cuts, lender=part), want2, dtype, f"borrowed, cut {cuts[:3]}", tol32=2e-5, tol16=4e-2)
    _no_error()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("mixer", [K.latent(3, 10, 6, 14, 20), K.latent(4, 48, 32, 40, 96), K.latent(2, 18, 0, 10, 33), K.latent(1, 7, 2, 3, 11, base=7.0),
                                   K.latent(20, 16, 16, 16, 112), K.latent(2, 24, 64, 32, 450, base=10000.0)])
def test_latent_attention_alone(mixer, dtype):
    """Rows of rank + rotated part that are, and are not, a multiple of 16 elements."""
    from rust_inference_b200.models.gotulorn import GotulornConfig
    config = K.config_of(11, 64, 1.0, 1e-3, [K.layer("l", mixer, None)])
    W = K.make_weights(config, 9)
    part, w = _mixer(GotulornConfig.from_dict(config).to_spec().layers[0].mixer, dtype, {n[len("l0.mix."):]: t for n, t in W.items() if n.startswith("l0.mix.")})
    assert part.cache_request().head_dim % 16 == 0
    x = _t(np.random.default_rng(10).standard_normal((150, 64)), dtype)
    want, first = P.latent_attention(_np(x), w, mixer, 1e-3), None
    for cuts in CUTS:
        got = _run_mixer(part, x, cuts)
        _close(got, want, dtype, f"cut {cuts[:3]}", tol32=2e-5, tol16=4e-2)
        first = got if first is None else first
        if dtype == torch.float32:
            assert torch.equal(got, first)
    _no_error()


# ---- feed-forwards -------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T, D, E, top", [(1, 48, 5, 2), (70, 52, 3, 3), (300, 64, 40, 4), (9, 50, 1, 1), (33, 256, 130, 8), (4, 2048, 600, 5)])
def test_router_by_logits(T, D, E, top, dtype):
    from rust_inference_b200 import ops
    rng = np.random.default_rng(E)
    x, router, b = _t(rng.standard_normal((T, D)), dtype), _t(rng.standard_normal((E, D)) * 2 / np.sqrt(D)), _t(rng.standard_normal(E) * 2)
    idx, w = ops.moe_route(x, router, None, top, "logits", bias=b)
    z = _np(x) @ _np(router).T + _np(b)
    order = np.argsort(-z, axis=1, kind="stable")[:, :top]
    assert np.array_equal(np.sort(idx.cpu().numpy(), axis=1), np.sort(order, axis=1))
    zc = np.take_along_axis(z, idx.cpu().numpy().astype(np.int64), axis=1)
    e = np.exp(zc - zc.max(1, keepdims=True))
    _close(w, e / e.sum(1, keepdims=True), torch.float32, "weights", tol32=2e-5)
    again, _ = ops.moe_route(x, router, None, top, "logits")
    order = np.argsort(-(z - _np(b)), axis=1, kind="stable")[:, :top]
    assert np.array_equal(np.sort(again.cpu().numpy(), axis=1), np.sort(order, axis=1))       # without the bias
    # logits far apart: softmax over all outputs would underflow for the chosen ones behind the first
    far = _t(np.linspace(0.0, -400.0, E) if E > 1 else [0.0])
    idx, w = ops.moe_route(torch.zeros_like(x), router, None, top, "logits", bias=far)
    assert np.array_equal(idx.cpu().numpy(), np.tile(np.arange(top), (T, 1))) and torch.isfinite(w).all()
    assert torch.allclose(w.sum(1), torch.ones(T, device=DEV))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rec", [K.dense(48, 0.8), K.dense(30, 1.4), K.moe(6, 3, 24), K.moe(1, 1, 20), K.moe(4, 4, 12), K.moe(16, 1, 40)])
def test_feed_forwards_for_few_and_many_tokens(rec, dtype):
    from rust_inference_b200.models.gotulorn import GotulornConfig
    from rust_inference_b200.parts import BuildEnv, StepContext, build_part, part_class
    D = 56
    config = K.config_of(11, D, 1.0, 1e-3, [K.layer("a", K.attn(1, 1, 8, 8), rec)])
    W = {n[len("l0.mlp."):]: t for n, t in K.make_weights(config, 3).items() if n.startswith("l0.mlp.")}
    spec = GotulornConfig.from_dict(config).to_spec().layers[0].ffn
    part = build_part("ffn", spec, BuildEnv(dtype, torch.device(DEV)))
    tensors = {n: _t(W[n], dtype if i.role == "matrix" else torch.float32) for n, i in part_class("ffn", spec).param_infos(spec).items()}
    part.load(tensors)
    w = {n: _np(t) for n, t in tensors.items()}
    for T in (1, 3, 16, 40, 700):
        x = _t(np.random.default_rng(T).standard_normal((T, D)) * 1.5, dtype)
        got = part(x, StepContext(*([None] * 5), num_tokens=T, num_seqs=1, max_new=T, max_len=T))
        want = P.clamped_ff(_np(x), w, rec["limit"]) if rec["kind"] == "dense" else P.routed_ff(_np(x), w, rec)
        _close(got, want, dtype, f"{T} tokens", tol32=2e-5, tol16=2.5e-2)


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
    reqs = H.random_requests(rng, config["vocab"], [5, 1, 23, 230, 2, 70, 37])
    want = K.plain_logits(config, weights, reqs)
    by_cutting = {}
    for label, steps in (("whole", H.trace_whole(reqs)), ("tail", H.trace_tail(reqs, tail=40)),
                         ("portions", _portions(reqs, [2, 7, 1, 33, 2])), ("pairs", _portions(reqs, [2])),
                         ("batches", H.trace_batches(reqs, 3, [6, 0, 9, 3, 70, 1, 36]))):
        out = str(tmp_path / f"out_{label}")
        H.replay_inprocess(d, dtype, steps, out, device="cuda:0")
        rows = H.collect(steps, out, config["vocab"])
        assert len(rows) == sum(len(t) for t in reqs.values())
        print(name, label, dtype, K.assert_rows_close(rows, want, dtype, f"{name} {label} {dtype}"))
        by_cutting[label] = rows
    if dtype == "float32":
        H.assert_rows_identical(by_cutting, f"{name} float32")


# A query finds one key: a token t + HAY looks for token t (what its query reads is what that token's key reads), every token
# of a prompt stands there once, and nothing else looks like it to the query.
HAY = 400


def _finder(kind, borrowed=False, size=None, keep=None):
    D, d = 64, 32
    if kind == "l":
        layers = [K.layer("l", K.latent(2, d, 0, d, d, scale=3.0), None)]
    else:
        m = K.attn(2, 1, d, d, size, keep, diff=0.2, scale=3.0)
        layers = [K.layer("a", dict(m, mask={"size": 9, "keep_first": 1}) if borrowed and size else m, None)]
        if borrowed:
            layers.append(K.layer("a", dict(m, kv_from=0), None))
    config = K.config_of(2 * HAY, D, 1.0, 1e-6, layers)
    W = K.make_weights(config, 21)
    E = np.sign(np.random.default_rng(22).standard_normal((2 * HAY, D)))
    E[HAY:, :d] = E[:HAY, d:]
    W["embed"] = K._bf16(E)
    reads_query, reads_key = np.concatenate([np.eye(d), np.zeros((d, d))], axis=1), np.concatenate([np.zeros((d, d)), np.eye(d)], axis=1)
    for name in ["embed.norm"] + [f"l{i}.norm1" for i in range(len(layers))]:
        W[name], W[name + ".b"], W[name + ".alpha"] = np.ones(D, np.float32), np.zeros(D, np.float32), np.float32(1.0)
    for i in range(len(layers)):
        p = f"l{i}."
        if i + 1 < len(layers):
            W[p + "mix.o"] = K._bf16(W[p + "mix.o"] * 0.2)             # so that the second layer still reads the token
        if kind == "l":
            W[p + "mix.q"] = K._bf16(np.concatenate([reads_query] * 2))
            W[p + "mix.dkv"] = K._bf16(reads_key)
            W[p + "mix.dkv.norm"] = np.ones(d, np.float32)
            W[p + "mix.uk"] = K._bf16(np.concatenate([np.eye(d)] * 2))
        else:
            W[p + "mix.q"] = K._bf16(np.concatenate([reads_query, 0 * reads_query] * 2))      # the second map looks for nothing
            if p + "mix.k" in W:
                W[p + "mix.k"] = K._bf16(np.concatenate([reads_key, reads_key]))
    return config, W


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind, far", [("l", 0), ("l", 31), ("l", 96), ("l", 255), ("own", 0), ("own", 95), ("own", 32), ("borrowed", 31), ("borrowed", 192)])
def test_a_far_key_among_hundreds_is_found(tmp_path, kind, far, dtype):
    """The last token looks for the token at position ``far`` (a page's first or last place among them) of 300.  As the last
    token of a prompt, as a token decoded alone, and in a portion of two."""
    config, W = _finder("l" if kind == "l" else "a", kind == "borrowed")
    toks = [int(t) for t in np.random.default_rng(far).permutation(HAY)[:300]]
    toks.append(toks[far] + HAY)
    W64 = K.as64(W)
    want = P.forward(config, W64, toks)[0]
    blind = list(toks)
    blind[far] = next(t for t in range(HAY) if t not in toks)
    assert K.row_error(P.forward(config, W64, blind)[0][300], want[300]) > 0.3, "the far key would not be missed"
    folder, reqs = K.write_model(str(tmp_path / "m"), config, W), {"r": toks}
    for label, steps in (("prompt", H.trace_whole(reqs)), ("decoded", H.trace_tail(reqs, tail=3)), ("pairs", _portions(reqs, [2, 297, 2]))):
        out = str(tmp_path / f"out_{label}")
        H.replay_inprocess(folder, dtype, steps, out, device="cuda:0")
        err = K.row_error(H.collect(steps, out, config["vocab"])[("r", 300)], want[300])
        assert err < (1e-4 if dtype == "float32" else 8e-2), f"{label}: error {err:.3e}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("borrowed", [False, True])
@pytest.mark.parametrize("size, keep", [(44, 7), (33, 32), (64, 33), (31, 1), (97, 0)])
def test_keys_at_the_edges_of_window_and_kept_tokens(tmp_path, size, keep, borrowed, dtype):
    """Some positions look for the key just inside the window, some for the one just outside, some for the first and the last
    kept token and the one behind it.  A mask that is one token off in any way would show."""
    config, W = _finder("a", borrowed, size, keep)
    n = 230
    toks = [int(t) for t in np.random.default_rng(size + keep).permutation(HAY)[:n]]
    for i, p in enumerate(range(140, 220, 7)):
        key = p - size + 1 if i % 2 == 0 else p - size
        if toks[key] < HAY:                                            # (not a position that looks for something itself)
            toks[p] = toks[key] + HAY
    for p, key in ((221, 0), (224, keep - 1), (227, keep)):
        if key >= 0:
            toks[p] = toks[key] + HAY
    reqs = {"r": toks}
    W64 = K.as64(W)
    want = P.forward(config, W64, toks)[0]
    masks = [{"size": size + 1, "keep_first": keep}, {"size": size - 1, "keep_first": keep}, {"size": size, "keep_first": keep + 1}]
    for mask in masks + ([{"size": size, "keep_first": keep - 1}] if keep else []):
        c = copy.deepcopy(config)
        c["layers"][-1]["mixer"]["mask"] = mask
        off = P.forward(c, W64, toks)[0]
        assert max(K.row_error(off[p], want[p]) for p in range(140, n)) > 0.2, f"{mask} would not show"
    folder = K.write_model(str(tmp_path / "m"), config, W)
    for label, steps in (("prompt", H.trace_whole(reqs)), ("decoded", H.trace_tail(reqs, tail=n - 130)), ("pairs", _portions(reqs, [2])),
                         ("thirties", _portions(reqs, [30]))):
        out = str(tmp_path / f"out_{label}")
        H.replay_inprocess(folder, dtype, steps, out, device="cuda:0")
        rows = H.collect(steps, out, config["vocab"])
        for p in range(n):
            err = K.row_error(rows[("r", p)], want[p])
            assert err < (1e-4 if dtype == "float32" else 1.2e-1), f"{label}: position {p}: error {err:.3e}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "C"])
def test_long_decoding_through_page_edges(tmp_path, name, dtype):
    """A short prompt, then 260 tokens one by one (graph replays) against the plain model; two sequences of unequal
    length whose pages live side by side."""
    d, config, weights = K.make_model_dir(tmp_path, name, seed=6)
    rng = np.random.default_rng(7)
    reqs = H.random_requests(rng, config["vocab"], [270, 200])
    want = K.plain_logits(config, weights, reqs)
    steps = H.trace_batches(reqs, 2, [260, 195])
    out = str(tmp_path / "out")
    H.replay_inprocess(d, dtype, steps, out, device="cuda:0", max_tokens=640)
    print(name, dtype, K.assert_rows_close(H.collect(steps, out, config["vocab"]), want, dtype, f"long decoding {name} {dtype}"))


def test_a_batch_of_forty_decodes_as_each_alone(tmp_path):
    """More sequences than the mma.sync linears take at once and than a warp has lanes, in bfloat16, against the plain model."""
    d, config, weights = K.make_model_dir(tmp_path, "C", seed=16)
    rng = np.random.default_rng(17)
    reqs = H.random_requests(rng, config["vocab"], [3 + 3 * i for i in range(40)])
    want = K.plain_logits(config, weights, reqs)
    steps = H.trace_batches(reqs, 40, [2])
    out = str(tmp_path / "out")
    H.replay_inprocess(d, "bfloat16", steps, out, device="cuda:0")
    K.assert_rows_close(H.collect(steps, out, config["vocab"]), want, "bfloat16", "forty sequences")


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
    from rust_inference_b200.engine import Engine, Entry, Model
    model = Model.from_random(copy.deepcopy(K.CFG_C), seed=1, dtype="bfloat16", device="cuda:0")
    engine = Engine(model, max_tokens=256, max_seqs=2)
    s = engine.new_sequence()
    logits = engine.step([Entry(s, [5, 9, 200])])
    assert torch.isfinite(logits).all() and float(logits.std()) > 0
    engine.check_device_errors()
