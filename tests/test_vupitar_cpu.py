"""CPU suite of the Vupitar family: the config reader, the registry, and the NumPy statement of the design against
hand-made cases (element-wise norm, rotation, chunk visibility, exponential gates, clamped unit, routing, loop) and
against itself (one-token steps with carried state against a whole run)."""
import json

import numpy as np
import pytest

from llama3_np_b200.stack import ATTN_SOFTMAX, FF_CLAMP, MLSTM, ROUTE_SOFTMAX_GLU, WINDOW
from llama3_np_b200.vupitar import stack_config
from oracle import ref_vupitar as R

LEFT = {"heads": 4, "kv_heads": 2, "dim": 8, "vdim": 12, "scale": 0.3, "mask": {"size": 7}, "rot": {"base": 777.0, "dims": 4}}
RIGHT = {"heads": 3, "dim": 6, "vdim": 10, "gate_cap": 9.0}
CFG = {
    "architecture": "Vupitar", "vocab": 53, "width": 40, "norm": {"eps": 1e-4}, "embedding": {"scale": 2.5},
    "loop": {"start": 1, "stop": 3, "times": 2},
    "layers": [
        {"type": "parallel", "mixer": {"left": LEFT, "right": RIGHT, "left_scale": 0.75, "right_scale": 1.5}, "mlp": None},
        {"type": "parallel", "mixer": {"left": dict(LEFT, mask={"size": 5}), "right": RIGHT, "left_scale": 1.0, "right_scale": 0.5},
         "mlp": {"kind": "dense", "ff": 28, "limit": 1.25}},
        {"type": "parallel", "mixer": {"left": dict(LEFT, heads=2, kv_heads=1), "right": dict(RIGHT, dim=4), "left_scale": 0.4, "right_scale": 0.6},
         "mlp": {"kind": "moe", "router": {"experts": 5, "top": 2}, "expert": {"ff": 12}, "shared": {"ff": 20}}},
    ],
}


def test_config_reader_takes_every_size_from_the_config():
    sc = stack_config(CFG, max_seq_len=77, max_batch_size=3, dtype="bfloat16")
    assert (sc.width, sc.vocab, sc.max_seq_len, sc.max_batch_size, sc.dtype) == (40, 53, 77, 3, "bfloat16")
    assert sc.norm_input and sc.norm_tanh and sc.dual_norm and sc.loop_x0 and sc.loop == (1, 3, 2) and not sc.token_shift and not sc.loop_in
    assert sc.norm_eps == pytest.approx(1e-4) and sc.embed_scale == pytest.approx(2.5)
    a, b, c = sc.layers
    assert (a.mixer, a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.chunked, a.rot_dims, a.rot_base, a.rot_layout, a.scale) == (WINDOW, 4, 2, 8, 12, 7, True, 4, 777.0, 1, 0.3)
    assert a.attn_kind == ATTN_SOFTMAX and a.qk_norm and a.proj_bias and a.head_gate and not a.qk_unit and a.keep_first == 0
    assert (a.mix_scale, a.pair_scale, a.ff) == (0.75, 1.5, 0)
    assert (a.pair.mixer, a.pair.heads, a.pair.dim, a.pair.vdim, a.pair.gate_cap) == (MLSTM, 3, 6, 10, 9.0)
    assert (b.window, b.ff, b.ff_kind, b.ff_limit, b.experts) == (5, 28, FF_CLAMP, 1.25, 0) and b.ff_slope == pytest.approx(1.702)
    assert (c.ff, c.experts, c.top, c.router_kind, c.shared_ff, c.shared_gate) == (12, 5, 2, ROUTE_SOFTMAX_GLU, 20, True)
    plain = json.loads(json.dumps(CFG))
    del plain["loop"], plain["embedding"], plain["layers"][2]["mlp"]["shared"], plain["layers"][0]["mixer"]["left"]["kv_heads"]
    sc = stack_config(plain)
    assert sc.loop is None and not sc.loop_x0 and sc.embed_scale == 1.0 and sc.layers[0].kv_heads == 4
    assert (sc.layers[2].shared_ff, sc.layers[2].shared_gate) == (0, False)
    for edit in (lambda c: c["layers"][1].update(type="hyena"), lambda c: c["layers"][1]["mlp"].update(kind="conv")):
        bad = json.loads(json.dumps(CFG))
        edit(bad)
        with pytest.raises(ValueError):
            stack_config(bad)


def test_registry_knows_the_architecture():
    from llama3_np_b200.models import ARCHITECTURES
    assert "Vupitar" in ARCHITECTURES


def test_element_wise_norm():
    y = R.dynamic_tanh(np.array([0.0, 2.0, -100.0]), 0.5, np.array([3.0, 1.0, 2.0]), np.array([0.1, 0.0, -1.0]))
    assert np.allclose(y, [0.1, np.tanh(1.0), -3.0])


def test_rotation_pairs_the_halves():
    v = np.arange(1.0, 9.0)
    r = R.rotate_halves(v, 5, 4, 100.0)
    assert np.allclose(r[4:], v[4:])  # entries past `dims` pass unchanged
    assert np.allclose(r[[0, 2]], [np.cos(5.0) - 3 * np.sin(5.0), 3 * np.cos(5.0) + np.sin(5.0)])
    assert np.allclose(r[[1, 3]], [2 * np.cos(0.5) - 4 * np.sin(0.5), 4 * np.cos(0.5) + 2 * np.sin(0.5)])
    assert np.allclose(R.rotate_halves(v, 9, 0, 100.0), v)


def test_chunks_are_counted_from_position_zero():
    assert [j for j in range(20) if R.visible_in_chunk(13, j, 5)] == [10, 11, 12, 13]
    assert [j for j in range(20) if R.visible_in_chunk(10, j, 5)] == [10]
    assert [j for j in range(20) if R.visible_in_chunk(4, j, 5)] == [0, 1, 2, 3, 4]
    assert [j for j in range(20) if R.visible_in_chunk(3, j, 0)] == [0, 1, 2, 3]


def test_gates_are_capped_and_the_running_maximum_cancels():
    i, f = R.mlstm_gates(np.array([1000.0, 0.5]), np.array([-1000.0, 0.0]), 7.0)
    assert np.allclose(i, [7.0, 7.0 * np.tanh(0.5 / 7)]) and np.allclose(f, [np.log(1 / (1 + np.exp(7.0))), np.log(0.5)])
    # the stabilised recurrence equals the plain one with numerator and max(|n . q|, 1) (but for the small constant)
    rng = np.random.default_rng(0)
    S, n, m = np.zeros((3, 4)), np.zeros(3), 0.0
    S2, n2 = np.zeros((3, 4)), np.zeros(3)
    for _ in range(12):
        q, k, v = rng.standard_normal(3), rng.standard_normal(3), rng.standard_normal(4)
        i, f = 2 * rng.standard_normal(), -abs(rng.standard_normal())
        S, n, m, o = R.mlstm_update(S, n, m, q, k, v, i, f)
        S2 = np.exp(f) * S2 + np.exp(i) * np.outer(k, v)
        n2 = np.exp(f) * n2 + np.exp(i) * k
        assert np.allclose(o, S2.T @ q / max(abs(n2 @ q), 1.0), rtol=1e-4)
        assert np.allclose(S * np.exp(m), S2) and m >= i


def test_clamped_unit():
    P = {"gate": np.eye(2), "up": np.eye(2), "down": np.eye(2)}
    y = R.clamped_unit(np.array([3.0, -4.0]), P, 1.5)
    assert np.allclose(y, [1.5 / (1 + np.exp(-1.702 * 1.5)) * 2.5, -4.0 / (1 + np.exp(1.702 * 4.0)) * -0.5])


def test_routing_weighs_the_best_by_their_own_sum():
    best, w = R.route(np.log(np.array([1.0, 5.0, 2.0, 8.0])), 2)
    assert list(best) == [3, 1] and np.allclose(w, [8 / 13, 5 / 13])
    best, w = R.route(np.array([0.0, 0.0, 0.0]), 2)
    assert list(best) == [0, 1] and np.allclose(w, 0.5)


def test_layer_runs_and_what_joins_the_stream_ahead_of_a_pass():
    t = R.random_model(CFG, 3)
    o = R.OracleVupitar(CFG, t)
    assert o.runs == [(0, -1), (1, 0), (2, -1), (1, 1), (2, -1)]
    seen = []
    o.layer = lambda i, x, st, pos: seen.append(x) or x   # layers that change nothing
    o.step(7)
    x0 = t["embed"][7].astype(np.float64) * 2.5
    s = t["loop.step"].astype(np.float64)
    assert np.allclose(seen[0], x0) and np.allclose(seen[1], x0 + s[0]) and np.allclose(seen[2], x0 + s[0])
    assert np.allclose(seen[3], 2 * x0 + s[0] + s[1]) and np.allclose(seen[4], 2 * x0 + s[0] + s[1])


def test_both_sublayers_read_the_same_stream():
    cfg = json.loads(json.dumps(CFG))
    t = R.random_model(cfg, 5)
    o = R.OracleVupitar(cfg, t)
    x = np.random.default_rng(1).standard_normal(40)
    both = o.layer(1, x, {"left": {}, "right": {}}, 0) - x
    cfg2 = json.loads(json.dumps(CFG))
    cfg2["layers"][1]["mlp"] = None
    mixer = R.OracleVupitar(cfg2, t).layer(1, x, {"left": {}, "right": {}}, 0) - x
    cfg2 = json.loads(json.dumps(CFG))
    cfg2["layers"][1]["mixer"].update(left_scale=0.0, right_scale=0.0)
    ff = R.OracleVupitar(cfg2, t).layer(1, x, {"left": {}, "right": {}}, 0) - x
    assert np.allclose(both, mixer + ff)


def test_steps_with_carried_state_equal_a_whole_run():
    t = R.random_model(CFG, 4)
    ids = np.random.default_rng(5).integers(0, 53, 17)
    o = R.OracleVupitar(CFG, t)
    whole, res = o.run(ids, want_residual=True)
    assert res.shape == (5, 17, 40)
    o.reset()
    parts = np.concatenate([o.run(ids[:5]), o.run(ids[5:6]), o.run(ids[6:])])
    assert np.allclose(parts, whole)
    o.reset()
    assert not np.allclose(o.run(ids[1:])[0], whole[1])  # the first token is part of every later answer
