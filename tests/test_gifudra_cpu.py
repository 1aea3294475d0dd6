"""CPU suite of the Gifudra family: the config reader, and the NumPy statement of the design against hand-made cases
(rotation, sink, streams, shared caches, gates) and against itself (one-token steps with carried state against a whole
run)."""
import json

import numpy as np
import pytest

from llama3_np_b200.gifudra import stack_config
from llama3_np_b200.stack import FF_RELU2, LATENT
from oracle import ref_gifudra as R


def _mixer(**kw):
    m = {"heads": 3, "dim": 8, "rot_dim": 4, "vdim": 6, "q_rank": 12, "kv_rank": 20, "scale": 0.25, "rot": {"base": 777.0, "dims": 4}}
    m.update(kw)
    return m


CFG = {
    "architecture": "Gifudra", "vocab": 53, "width": 40, "norm": {"eps": 1e-4}, "embedding": {"scale": 2.5}, "streams": 3,
    "logit_scale": 0.75,
    "layers": [
        {"type": "latent_attention", "mixer": _mixer(), "mlp": {"kind": "dense", "ff": 28}},
        {"type": "latent_attention", "mixer": _mixer(heads=2, dim=5, vdim=7, q_rank=9, scale=0.5, kv_from=0), "mlp": None},
    ],
}


def test_config_reader_takes_every_size_from_the_config():
    sc = stack_config(CFG, max_seq_len=77, max_batch_size=3, dtype="bfloat16")
    assert (sc.width, sc.vocab, sc.max_seq_len, sc.max_batch_size, sc.dtype) == (40, 53, 77, 3, "bfloat16")
    assert sc.norm_input and sc.layer_scale and sc.tied_head and not sc.norm_one_plus and not sc.token_shift and not sc.norm_scalar
    assert sc.norm_eps == pytest.approx(1e-4) and sc.embed_scale == pytest.approx(2.5) and sc.logit_scale == pytest.approx(0.75)
    assert sc.streams == 3 and sc.loop is None
    a, b = sc.layers
    assert (a.mixer, a.heads, a.dim, a.rot_dim, a.rot_dims, a.vdim, a.q_rank, a.kv_rank) == (LATENT, 3, 8, 4, 4, 6, 12, 20)
    assert (a.scale, a.rot_base, a.rot_layout, a.sink, a.gate_wide, a.kv_from) == (0.25, 777.0, 1, True, True, None)
    assert (a.ff, a.ff_kind, a.experts) == (28, FF_RELU2, 0)
    assert (b.heads, b.dim, b.vdim, b.q_rank, b.scale, b.kv_from, b.ff) == (2, 5, 7, 9, 0.5, 0, 0)
    brief = json.loads(json.dumps(CFG))
    for k in ("kv_rank", "rot_dim", "rot"):
        del brief["layers"][1]["mixer"][k]
    b = stack_config(brief).layers[1]
    assert (b.kv_rank, b.rot_dim, b.rot_dims, b.rot_base, b.dim) == (20, 4, 4, 777.0, 5)
    plain = json.loads(json.dumps(CFG))
    del plain["streams"], plain["embedding"], plain["logit_scale"]
    sc = stack_config(plain)
    assert (sc.streams, sc.embed_scale, sc.logit_scale) == (0, 1.0, 1.0)
    for edit in (lambda c: c["layers"][1].update(type="hyena"), lambda c: c["layers"][0]["mlp"].update(kind="moe")):
        bad = json.loads(json.dumps(CFG))
        edit(bad)
        with pytest.raises(ValueError):
            stack_config(bad)


def test_registry_knows_the_architecture():
    from llama3_np_b200.models import ARCHITECTURES
    assert "Gifudra" in ARCHITECTURES


def test_rotation_pairs_the_halves():
    v = np.arange(1.0, 9.0)
    r = R.rotate_halves(v, 5, 4, 100.0)
    assert np.allclose(r[4:], v[4:])  # entries past `dims` pass unchanged
    a0, a1 = 5.0, 5.0 * 100.0 ** (-0.5)
    assert np.allclose(r[[0, 2]], [np.cos(a0) - 3 * np.sin(a0), 3 * np.cos(a0) + np.sin(a0)])
    assert np.allclose(r[[1, 3]], [2 * np.cos(a1) - 4 * np.sin(a1), 4 * np.cos(a1) + 2 * np.sin(a1)])
    q, k = np.random.default_rng(0).standard_normal((2, 6))  # a product depends on the distance of the positions only
    assert R.rotate_halves(q, 40, 6, 50.0) @ R.rotate_halves(k, 33, 6, 50.0) == pytest.approx(
        R.rotate_halves(q, 107, 6, 50.0) @ R.rotate_halves(k, 100, 6, 50.0))


def test_sink_takes_weight_without_a_value():
    z = np.array([0.0, np.log(2.0)])
    assert np.allclose(R.sink_softmax(z, 0.0), [0.25, 0.5])
    assert np.allclose(R.sink_softmax(z, -np.inf), [1 / 3, 2 / 3])
    assert np.allclose(R.sink_softmax(z + 900.0, 900.0), [0.25, 0.5])
    assert R.sink_softmax(z, 800.0).sum() < 1e-100


def test_streams_move_all_at_once():
    X = np.array([[1.0, 10.0], [2.0, 20.0]])
    P = {"hc1.in": np.array([0.5, -1.0]), "hc1.out": np.array([1.0, 3.0]), "hc1.mix": np.array([[0.0, 1.0], [2.0, 0.0]])}
    assert np.allclose(R.streams_in(X, P, 1), [-1.5, -15.0])
    # stream 0 receives 2 x stream 1, stream 1 receives stream 0, both from the OLD rows
    assert np.allclose(R.streams_out(X, np.array([0.1, 0.2]), P, 1), [[4.1, 40.2], [1.3, 10.6]])
    assert np.allclose(R.streams_out(X[:1], np.array([0.1, 0.2]), {}, 1), [[1.1, 10.2]])


def test_shared_cache_layers_read_the_owner_s_rows():
    t = R.random_model(CFG, 3)
    assert not any(k.startswith("l1.mix.dkv") for k in t) and "l1.norm2" not in t and "l1.ls2" not in t and "head" not in t
    o = R.OracleGifudra(CFG, t)
    ids = np.random.default_rng(1).integers(0, 53, 6)
    a = o.run(ids)
    assert len(o.state[0]["c"]) == 6 and "c" not in o.state[1]
    t2 = dict(t)
    t2["l0.mix.dkv"] = t["l0.mix.dkv"] * np.array([[1.0]] * 20 + [[1.5]] * 4)  # the rotated key part reaches layer 1, too
    o2 = R.OracleGifudra(CFG, t2)
    assert not np.allclose(o2.run(ids), a)


def test_steps_with_carried_state_equal_a_whole_run():
    t = R.random_model(CFG, 4)
    ids = np.random.default_rng(5).integers(0, 53, 17)
    o = R.OracleGifudra(CFG, t)
    whole, res = o.run(ids, want_residual=True)
    assert res.shape == (2, 17, 40)
    o.reset()
    parts = np.concatenate([o.run(ids[:5]), o.run(ids[5:6]), o.run(ids[6:])])
    assert np.allclose(parts, whole)
    o.reset()
    assert not np.allclose(o.run(ids[1:])[0], whole[1])  # the first token is part of every later answer
