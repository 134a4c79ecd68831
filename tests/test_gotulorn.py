"""Gotulorn without a GPU: the configuration class, the tensor list, the schedule with its borrowed cache entries, what the
cache keeps (first tokens beside a window, the keys of the widest reader), the plain model's mechanisms, and the engine's host
logic with the kernels replaced by the stand-ins of tests/emu_ops.py, against the plain model of tests/plain_gotulorn.py."""
import copy

import numpy as np
import pytest
import torch

import gotulorn_models as K
import helpers as H
import plain_gotulorn as P
from rust_inference_b200.cache.allocator import PageTable
from rust_inference_b200.parts.base import CacheRequest


def test_spec_lists_parts_and_schedule():
    from rust_inference_b200.config import config_from_dict
    from rust_inference_b200.engine.model import expected_tensors
    cfg = config_from_dict(copy.deepcopy(K.CFG_A))
    assert type(cfg).__name__ == "GotulornConfig" and cfg.to_dict() == K.CFG_A
    spec = cfg.to_spec()
    assert [(e.layer, e.cache, e.writes) for e in spec.schedule] == \
        [(0, 0, True), (1, 1, True), (2, 0, False), (3, 2, True), (4, 2, False), (5, 3, True)]
    assert spec.cache_entries() == [0, 1, 3, 5] and not spec.tie_embeddings
    assert spec.embedding.scale == 1.7 and spec.embedding.norm.kind == spec.final_norm.kind == "dyn_tanh"
    first, third = spec.layers[0], spec.layers[2]
    m = first.mixer
    assert (m.maps, m.head_dim, m.v_head_dim, m.window, m.keep_first, m.pair_diff, m.own_kv) == (2, 12, 36, 17, 3, 0.3, True)
    assert not third.mixer.own_kv and third.ffn is None and third.ffn_norm is None
    assert (first.ffn.gate, first.ffn.limit) == ("clamped_swish", 0.9)
    f = spec.layers[1].ffn
    assert (f.score, f.router_bias, f.top, f.expert.gate) == ("logits", "router.b", 3, "silu")
    assert spec.layers[4].mixer.window == 0 and spec.layers[4].mixer.keep_first == 0
    for config in K.ALL.values():
        expected = expected_tensors(config_from_dict(copy.deepcopy(config)).to_spec())
        weights = K.make_weights(config, 0)
        assert {n: tuple(i.shape) for n, i in expected.items()} == {n: w.shape for n, w in weights.items()}


@pytest.mark.parametrize("change, text", [
    (lambda c: c["layers"][0].update(type="conv"), "not built"),
    (lambda c: c["layers"][0]["mlp"].update(kind="gelu"), "not built"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=2), "earlier layer"),
    (lambda c: c["layers"][4]["mixer"].update(kv_from=2), "of its own"),
    (lambda c: c["layers"][4]["mixer"].update(kv_from=1), "of its own"),
    (lambda c: c["layers"][2]["mixer"].update(vdim=20), "vdim"),
    (lambda c: c["layers"][0]["mixer"].update(heads=5), "kv_heads"),
    (lambda c: c["layers"][0]["mixer"].update(scale=0.0), "scale"),
    (lambda c: c["layers"][0]["mixer"].pop("diff"), "diff"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(keep_first=-1), "keep_first"),
    (lambda c: c["layers"][1]["mixer"].update(rot_dim=5), "rot_dim"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=4), "dims"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=7), "top"),
    (lambda c: c["layers"][0]["mlp"].pop("limit"), "limit"),
    (lambda c: c.pop("embedding"), "scale"),
])
def test_bad_configurations_are_refused(change, text):
    from rust_inference_b200.config import ConfigError, config_from_dict
    c = copy.deepcopy(K.CFG_A)
    change(c)
    with pytest.raises(ConfigError, match=text):
        config_from_dict(c)


# ---- what the cache keeps -----------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("window, keep", [(40, 5), (1, 32), (33, 33), (31, 64), (100, 1), (64, 200), (7, 0)])
def test_pages_of_the_first_tokens_stay_beside_a_window(window, keep):
    t = PageTable(num_slots=2, num_pages=24, max_pages_per_seq=40, page_size=32, window=window, keep=keep)
    for slot in (0, 1):
        total = 0
        for n in [1, 31, 2, 17, 64, 5] * 3:
            if total + n > 400:
                break
            t.extend(slot, n)
            total += n
            t.release_behind_window(slot)
            for p in range(-(-total // 32)):
                needed = (p + 1) * 32 > total - window + 1 or p * 32 < keep
                assert (t.table[slot][p] >= 0) == needed, (total, p)
            t.check()
        t.release(0)                                        # a slot's pages, kept ones too, come back when it is given up
        t.check()
    t.release(1)
    assert t.free_pages == 24


def test_a_lender_keeps_what_its_readers_see():
    from rust_inference_b200.config import config_from_dict
    from rust_inference_b200.engine import Model
    own = CacheRequest(kv_heads=2, head_dim=16, window=17, keep_first=3)
    other = CacheRequest(kv_heads=2, head_dim=16, window=45, keep_first=2)
    both = own.for_readers([other])
    assert (both.window, both.keep_first) == (45, 3) and own.for_readers([own]) is own
    assert own.for_readers([CacheRequest(kv_heads=2, head_dim=16)]).mask == 0
    assert own.for_readers([CacheRequest(kv_heads=2, head_dim=16, chunk=8)]).mask == 0
    reqs = Model(config_from_dict(copy.deepcopy(K.CFG_A)).to_spec(), "float32", "cpu").cache_requests()
    assert [(r.window, r.kept) for r in reqs] == [(45, 5), (0, 0), (0, 0), (0, 0)]
    assert [r.head_dim for r in reqs] == [48, 32, 48, 48]
    reqs = Model(config_from_dict(copy.deepcopy(K.CFG_C)).to_spec(), "float32", "cpu").cache_requests()
    assert [(r.window, r.kept) for r in reqs] == [(70, 40), (0, 0), (100, 9), (128, 32)]


# ---- the plain model's mechanisms -------------------------------------------------------------------------------------------------
def test_plain_mask_and_pair():
    assert P.sees(9, {"size": 3, "keep_first": 2}).tolist() == [0, 1, 7, 8, 9]
    assert P.sees(3, {"size": 3, "keep_first": 2}).tolist() == [0, 1, 2, 3]
    assert P.sees(1, {"size": 1, "keep_first": 5}).tolist() == [0, 1]
    assert P.sees(4, {"size": 2}).tolist() == [3, 4] and P.sees(4, None).tolist() == list(range(5))
    w = {"lq1": np.array([0.5, 1.0]), "lk1": np.array([1.0, 0.1]), "lq2": np.array([0.0, 1.0]), "lk2": np.array([3.0, 0.2])}
    assert np.isclose(P.mix_factor(w, 0.7), np.exp(0.6) - np.exp(0.2) + 0.7)
    # one key in sight: both maps give its value v, and (1 - lam) v is normed, so the sign of 1 - lam is all that is left of lam
    m = {"heads": 1, "kv_heads": 1, "dim": 2, "scale": 1.0, "diff": 0.7, "mask": {"size": 1}}
    v = np.array([[[3.0, -4.0]]])
    w.update(q=np.ones((4, 5)), o=np.eye(2))
    out = P.paired_attention(np.ones((1, 5)), w, m, 0.0, np.ones((1, 1, 2, 2)), v)
    assert np.allclose(out, -v[0] / np.sqrt(12.5) * 0.3)


def test_plain_router_weighs_the_chosen_alone():
    w = {"router": np.zeros((3, 1)), "router.b": np.array([2.0, 5.0, 4.0])}
    for e in range(3):
        w.update({f"e{e}.gate": np.array([[1.0]]), f"e{e}.up": np.array([[1.0]]), f"e{e}.down": np.array([[float(e)]])})
    y = P.routed_ff(np.array([[1.0]]), w, {"router": {"top": 2}})
    a = np.exp(1.0) / (np.exp(1.0) + 1.0)
    assert np.allclose(y, P.sigmoid(1.0) * (a * 1.0 + (1 - a) * 2.0))


def test_every_mechanism_shows_in_the_logits():
    """Planted mistakes in the plain model (a window one token off, a kept token left out, keys of another layer, a map's
    factor, a router without its bias, weights over all experts) move the logits by far more than the tolerances."""
    config = copy.deepcopy(K.CFG_A)
    W = K.as64(K.make_weights(config, 3))
    toks = [int(t) for t in np.random.default_rng(4).integers(0, 97, 60)]
    want = P.forward(config, W, toks)[0]

    def moved(change_config=lambda c: None, change_weights=lambda w: None, patch=None):
        c, w, kept = copy.deepcopy(config), dict(W), {}
        change_config(c)
        change_weights(w)
        for name, f in (patch or {}).items():
            kept[name] = getattr(P, name)
            setattr(P, name, f)
        try:
            got = P.forward(c, w, toks)[0]
        finally:
            for name, f in kept.items():
                setattr(P, name, f)
        return float(np.mean([K.row_error(g, x) for g, x in zip(got, want)]))

    sees = P.sees
    assert moved() == 0.0
    assert moved(lambda c: c["layers"][0]["mixer"]["mask"].update(size=18)) > 5e-3
    assert moved(lambda c: c["layers"][0]["mixer"]["mask"].update(keep_first=2)) > 5e-3
    assert moved(lambda c: c["layers"][2]["mixer"]["mask"].update(size=17)) > 5e-3
    assert moved(patch={"sees": lambda p, m: sees(p, m and dict(m, keep_first=0))}) > 0.02
    assert moved(patch={"mix_factor": lambda w, diff: diff}) > 0.02
    assert moved(patch={"over_rms": lambda x, eps: x}) > 0.05
    assert moved(lambda c: c["embedding"].update(scale=1.0)) > 0.05
    assert moved(change_weights=lambda w: w.update({"l1.mlp.router.b": 0 * w["l1.mlp.router.b"]})) > 0.02
    assert moved(lambda c: c["layers"][0]["mlp"].update(limit=1.2)) > 5e-3
    assert moved(lambda c: c["layers"][1]["mixer"]["rot"].update(base=900.0)) > 1e-3
    assert moved(change_weights=lambda w: w.update({"l3.norm1.b": 0 * w["l3.norm1.b"]})) > 5e-3


# ---- the engine's host logic on the stand-ins -----------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_replay_three_ways_matches_plain(tmp_path, emulated_ops, name):
    d, config, weights = K.make_model_dir(tmp_path, name, seed=3)
    rng = np.random.default_rng(4)
    reqs = H.random_requests(rng, config["vocab"], [5, 1, 23, 85, 2, 35])
    want = K.plain_logits(config, weights, reqs)
    for label, steps in (("whole", H.trace_whole(reqs)), ("tail", H.trace_tail(reqs, tail=12)),
                         ("batches", H.trace_batches(reqs, 3, [6, 0, 9, 3]))):
        out = str(tmp_path / f"out_{label}")
        H.replay_inprocess(d, "float32", steps, out)
        rows = H.collect(steps, out, config["vocab"])
        assert len(rows) == sum(len(t) for t in reqs.values())
        K.assert_rows_close(rows, want, "float32", f"{name} {label}")


def test_windowed_pages_are_given_back_while_kept_ones_stay(tmp_path, emulated_ops):
    """One sequence decoded far past its window with hardly more pages than the window needs."""
    from rust_inference_b200.engine import Engine, Entry, Model
    config = K.config_of(97, 40, 1.0, 1e-5, [K.layer("a", K.attn(4, 2, 12, 24, 20, 3), K.dense(24, 1.0)),
                                             K.layer("a", K.attn(2, 2, 12, 24, 33, 1, kv_from=0), None)])
    W = K.make_weights(config, 5)
    d = K.write_model(str(tmp_path / "m"), config, W)
    engine = Engine(Model.from_dir(d, dtype="float32", device="cpu"), max_tokens=32 * 7, max_seqs=1, max_seq_len=32 * 7, use_graphs=False)
    toks = [int(t) for t in np.random.default_rng(6).integers(0, 97, 150)]
    want = P.forward(config, K.as64(W), toks)[0]
    s = engine.new_sequence()
    got = [engine.step([Entry(s, toks[:40], "all")])]
    for t in toks[40:]:
        got.append(engine.step([Entry(s, [t])]).clone())
        pages = engine.cache.groups[0].pages
        assert pages.table[s][0] >= 0                                  # the kept tokens' page
    assert pages.free_pages >= 7 - 4                                   # kept, two or three of the window
    K.assert_rows_close({("r", p): r for p, r in enumerate(torch.cat(got).numpy())}, {"r": want}, "float32")
    engine.release(s)
    engine.cache.check()
    assert engine.cache.free_pages() == 7


def test_greedy_generation_matches_plain(tmp_path, emulated_ops):
    """Greedy tokens through the generation loop (two batches on the same slots) against the plain model."""
    import rust_inference_b200 as ri
    d, config, weights = K.make_model_dir(tmp_path, "A", seed=8)
    W = K.as64(weights)
    prompts = [[5, 9, 2], [7], [90, 3, 3, 8, 1, 60]]
    llm = ri.LLM(d, dtype="float32", device="cpu", max_pages=16, pages_per_seq=2, max_seqs=2, use_graphs=False)
    got = llm.generate(prompts, max_new_tokens=5)
    for p, g in zip(prompts, got):
        seq = list(p)
        for _ in range(5):
            seq.append(int(np.argmax(P.forward(config, W, seq)[0][-1])))
        assert g == seq[len(p):]
