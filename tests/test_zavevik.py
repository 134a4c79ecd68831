"""Zavevik without a GPU: the configuration class, the tensor list, the schedule with its borrowed cache entries, the
distance buckets, the plain model's mechanisms, and the engine's host logic (pages that a second layer reads, states beside
them, slots used again) with the kernels replaced by the stand-ins of tests/emu_ops.py, against the plain model of
tests/plain_zavevik.py."""
import copy
import math

import numpy as np
import pytest

import helpers as H
import plain_zavevik as P
import zavevik_models as K


def test_spec_lists_parts_and_schedule():
    from rust_inference_b200.config import config_from_dict
    from rust_inference_b200.engine.model import expected_tensors
    cfg = config_from_dict(copy.deepcopy(K.CFG_A))
    assert type(cfg).__name__ == "ZavevikConfig" and cfg.to_dict() == K.CFG_A
    spec = cfg.to_spec()
    assert [(e.layer, e.cache, e.writes) for e in spec.schedule] == \
        [(0, 0, True), (1, 0, False), (2, 1, True), (3, 0, False), (4, 2, True)]
    assert spec.cache_entries() == [0, 2, 4] and not spec.tie_embeddings and spec.final_norm.scalar
    assert spec.embedding.side_width == 5 * 12
    first, second = spec.layers[0], spec.layers[1]
    assert first.arrangement == "postnorm" and first.mixer_link.scalar and first.side.start == 0 and second.side.start == 12
    m = first.mixer
    assert (m.unit_rms, m.unit_values, m.softcap, m.temperature, m.bias_rows, m.bias_far, m.v_head_dim, m.own_kv) == \
        (True, True, 6.0, (0.6, 10.0), 10, 70.0, 40, True)
    assert not second.mixer.own_kv and second.ffn is None and second.ffn_link is None
    d = spec.layers[2].mixer
    assert (d.kind, d.decay, d.gate, d.gate_fn, d.conv) == ("gated_delta", "head", "full", "silu", 3)
    f = first.ffn
    assert (f.route, f.table_rows, f.top, f.expert.gate) == ("table", 97, 3, "silu")
    for config in K.ALL.values():
        expected = expected_tensors(config_from_dict(copy.deepcopy(config)).to_spec())
        weights = K.make_weights(config, 0)
        assert {n: tuple(i.shape) for n, i in expected.items()} == {n: w.shape for n, w in weights.items()}


@pytest.mark.parametrize("change, text", [
    (lambda c: c["layers"][0].update(type="conv"), "not built"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "not built"),
    (lambda c: c["layers"][1]["mixer"].update(kv_from=1), "earlier layer"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=1), "of its own"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=2), "of its own"),
    (lambda c: c["layers"][1]["mixer"].update(dim=20), "dim"),
    (lambda c: c["layers"][0]["mixer"].update(heads=5), "kv_heads"),
    (lambda c: c["layers"][0]["mixer"].update(scale=0.0), "scale"),
    (lambda c: c["layers"][0]["mixer"]["q_temp"].update(every=0), "every"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=7), "top"),
    (lambda c: c["layers"][2]["mixer"].pop("conv"), "conv"),
    (lambda c: c.pop("width"), "width"),
])
def test_bad_configurations_are_refused(change, text):
    from rust_inference_b200.config import ConfigError, config_from_dict
    c = copy.deepcopy(K.CFG_A)
    change(c)
    with pytest.raises(ConfigError, match=text):
        config_from_dict(c)


def test_rows_of_a_bias_come_from_its_tensor(tmp_path):
    from rust_inference_b200.config import ConfigError, load_config
    d, config, _ = K.make_model_dir(tmp_path, "C", seed=2)
    cfg = load_config(d)
    with pytest.raises(ConfigError, match="rows"):
        cfg.to_spec()
    spec = cfg.with_checkpoint(d).to_spec()
    assert [l.mixer.bias_rows for l in spec.layers if l.mixer.kind == "attention"] == [16, 32, 12]


@pytest.mark.parametrize("rows, far", [(2, 9), (4, 40), (6, 120), (8, 33), (10, 70), (14, 61), (16, 500), (32, 90), (16, 16), (20, 320)])
def test_distance_buckets(rows, far):
    """The borders of the rows against the formula, distance by distance, and the table spread over the distances."""
    import torch
    from rust_inference_b200.parts.distance import bucket_starts, spread_over_distances
    starts = bucket_starts(rows, far)
    assert starts[0] == 0 and len(starts) == rows and starts[:rows // 2] == list(range(rows // 2))
    for n in range(2 * far + 3):
        row = max(i for i in range(rows) if starts[i] <= n)
        assert row == P.distance_bucket(n, rows, far), n
    table = torch.randn(rows, 3)
    wide = spread_over_distances(table, far)
    assert wide.shape[0] == 3 and wide.shape[1] <= far + 1
    for n in range(2 * far + 3):
        assert torch.equal(wide[:, min(n, wide.shape[1] - 1)], table[P.distance_bucket(n, rows, far)])


def test_query_factor_table():
    import torch
    from rust_inference_b200.config import config_from_dict
    from rust_inference_b200.parts import BuildEnv, build_part
    mixer = config_from_dict(copy.deepcopy(K.CFG_A)).to_spec().layers[0].mixer
    part = build_part("mixer", mixer, BuildEnv(torch.float32, torch.device("cpu")))
    part.prepare(64)
    want = [P.query_factor(p, 0.6, 10) for p in range(64)]
    assert np.abs(part.q_factor.numpy() - want).max() < 1e-6
    assert want[8] == 1.0 and math.isclose(want[9], 1.0 + 0.6 * math.log(2.0))      # the tenth position is the first with a factor


def test_random_tables_name_different_experts():
    import torch
    from rust_inference_b200.weights.random_init import random_tensor
    a = random_tensor(5, "l0.mlp.table", (200, 3), "table", torch.float32, below=7)
    assert a.dtype == torch.int32 and int(a.min()) >= 0 and int(a.max()) == 6
    assert all(len(set(r)) == 3 for r in a.tolist()) and len(set(a[:, 0].tolist())) == 7
    assert torch.equal(random_tensor(5, "l0.mlp.table", (50, 3), "table", torch.float32, below=7, first_row=100), a[100:150])


def test_plain_delta_rule_decays_the_whole_state_by_one_number():
    rng = np.random.default_rng(0)
    q, k, v = rng.standard_normal((3, 4)), rng.standard_normal((3, 4)), rng.standard_normal((3, 2))
    k /= np.linalg.norm(k, axis=1, keepdims=True)
    o = P.delta_rule(q, k, v, np.array([1.0, 0.5, 0.0]), np.array([0.3, 0.9, 0.5]))
    S = np.outer(k[0], v[0])
    assert np.allclose(o[0], S.T @ q[0])
    S = 0.9 * S
    S = S + np.outer(k[1], 0.5 * (v[1] - S.T @ k[1]))
    assert np.allclose(o[1], S.T @ q[1])
    assert np.allclose(o[2], (0.5 * S).T @ q[2])


@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_replay_three_ways_matches_plain(tmp_path, emulated_ops, name):
    d, config, weights = K.make_model_dir(tmp_path, name, seed=3)
    rng = np.random.default_rng(4)
    reqs = H.random_requests(rng, config["vocab"], [5, 1, 23, 40, 2, 35])
    want = K.plain_logits(config, weights, reqs)
    for label, steps in (("whole", H.trace_whole(reqs)), ("tail", H.trace_tail(reqs, tail=12)),
                         ("batches", H.trace_batches(reqs, 3, [6, 0, 9, 3]))):
        out = str(tmp_path / f"out_{label}")
        H.replay_inprocess(d, "float32", steps, out)
        rows = H.collect(steps, out, config["vocab"])
        assert len(rows) == sum(len(t) for t in reqs.values())
        K.assert_rows_close(rows, want, "float32", f"{name} {label}")


def test_every_mechanism_shows_in_the_logits():
    """Planted mistakes in the plain model (a bias one distance off, a factor one position early, the borrowed keys of the
    wrong layer, an expert left out, the token's row of the next layer) move the logits by far more than the tolerances."""
    config = copy.deepcopy(K.CFG_A)
    config["layers"][4] = K.layer("attention", K.attn(4, 2, 24, 40, scale=0.5, cap=6.0, far=70, rows=10), None)
    config["layers"].append(K.layer("attention", K.attn(4, 2, 24, 40, scale=0.4, far=120, rows=6, kv_from=4), None))
    W = K.as64(K.make_weights(config, 3))
    toks = [int(t) for t in np.random.default_rng(4).integers(0, 97, 60)]
    want = P.forward(config, W, toks)[0]

    def moved(change_config=lambda c: None, change_weights=lambda w: None, patch=None):
        c, w = copy.deepcopy(config), dict(W)
        change_config(c)
        change_weights(w)
        kept = {}
        for name, f in (patch or {}).items():
            kept[name] = getattr(P, name)
            setattr(P, name, f)
        try:
            got = P.forward(c, w, toks)[0]
        finally:
            for name, f in kept.items():
                setattr(P, name, f)
        return float(np.mean([K.row_error(g, x) for g, x in zip(got, want)]))

    bucket, factor = P.distance_bucket, P.query_factor
    assert moved() == 0.0
    assert moved(patch={"distance_bucket": lambda n, rows, far: bucket(n + 1, rows, far)}) > 0.05
    assert moved(patch={"query_factor": lambda p, coef, every: factor(p + 1, coef, every)}) > 1e-3
    assert moved(lambda c: c["layers"][5]["mixer"].update(kv_from=0)) > 0.05
    assert moved(lambda c: c["layers"][0]["mixer"].pop("softcap")) > 1e-3
    assert moved(change_weights=lambda w: w.update({"l2.mlp.table": w["l2.mlp.table"][:, :1].repeat(2, axis=1)})) > 0.05
    assert moved(change_weights=lambda w: w.update({"side.embed": np.roll(w["side.embed"], 12, axis=1)})) > 0.05
    assert moved(change_weights=lambda w: w.update({"l2.mix.dt_bias": w["l2.mix.dt_bias"][::-1]})) > 5e-3


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
