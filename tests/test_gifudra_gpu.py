"""Gifudra on the GPU against the plain NumPy statement of the design (oracle/ref_gifudra.py): every mechanism alone,
whole prompts against token-by-token decoding and against portions down to two tokens, batches against single
sequences, reused slots, far and planted keys, sinks, shared caches, residual streams, odd sizes, the tensor-core
prompt attention at many shapes, and greedy generation through the library's own loop and scheduler.  Small random
models; fp32 mode is held to 1e-4 of the logit scale, bf16 to 5e-2."""
import json

import numpy as np
import pytest

from oracle.ref_gifudra import OracleGifudra, random_model, to_bf16_grid

pytestmark = pytest.mark.gpu

BAR = {"float32": 1e-4, "bfloat16": 5e-2}


def latent(heads=3, dim=16, rot_dim=8, vdim=24, q_rank=40, kv_rank=48, scale=0.25, base=10000.0, kv_from=None, ff=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale,
         "rot": {"base": base, "dims": rot_dim}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(layers, width=56, vocab=97, streams=3, eps=1e-5, embed=3.0, logit=0.5):
    c = {"architecture": "Gifudra", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width,
         "embedding": {"scale": embed}, "logit_scale": logit}
    if streams is not None:
        c["streams"] = streams
    return c


def build(cfg, seed=0, dtype="float32", max_seq_len=128, max_batch_size=1, tensors=None):
    from llama3_np_b200.gifudra import Gifudra
    t = random_model(cfg, seed) if tensors is None else tensors
    return Gifudra(cfg, t, dtype=dtype, max_seq_len=max_seq_len, max_batch_size=max_batch_size), OracleGifudra(cfg, t)


def err(got, want):
    """largest row error: rms of the mean-free difference over the rms of the mean-free logits"""
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    d = got - want
    d = d - d.mean(-1, keepdims=True)
    w = want - want.mean(-1, keepdims=True)
    return float(np.max(np.sqrt((d * d).mean(-1)) / np.sqrt((w * w).mean())))


def toks(n, vocab, seed=1):
    return np.random.default_rng(seed).integers(0, vocab, n)


def fresh(o):
    o.reset()
    return o


def in_portions(m, ids, sizes):
    """logits of every token, fed in portions of the given sizes (repeated)"""
    pos, i, rows = 0, 0, []
    while pos < len(ids):
        c = min(sizes[i % len(sizes)], len(ids) - pos)
        i += 1
        rows.append(m.forward_rows(ids[None, pos:pos + c], pos, list(range(c))))
        pos += c
    return np.concatenate(rows)


ALONE = {
    "latent": config([latent()]),
    "one_stream": config([latent()], streams=1),
    "no_streams": config([latent(ff=40), latent()], streams=None),
    "two_streams": config([latent(heads=2, ff=24)], streams=2, width=40),
    "five_streams": config([latent(heads=2, ff=32)], streams=5, width=48),
    "eleven_streams": config([latent(heads=1)], streams=11, width=32),
    "feed_forward": config([latent(heads=1, dim=8, vdim=8, ff=88)]),
    "shared_cache": config([latent(), latent(heads=5, dim=8, vdim=16, q_rank=24, scale=0.4, kv_from=0), latent(heads=1, vdim=40, kv_from=0)]),
}


@pytest.mark.parametrize("name", sorted(ALONE))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_each_mechanism_alone(name, dtype):
    cfg = ALONE[name]
    m, o = build(cfg, seed=3, dtype=dtype)
    ids = toks(40, cfg["vocab"])
    got, resid = m.forward_rows(ids[None], 0, list(range(40)), want_residual=True)
    want, wres = o.run(ids, want_residual=True)
    assert resid.shape == (len(cfg["layers"]), 40, cfg["width"])
    assert err(got, want) < BAR[dtype]
    assert np.allclose(resid, wres, rtol=1e-4, atol=1e-4) if dtype == "float32" else np.abs(resid - wres).max() < 0.05 * np.abs(wres).max()
    # a decoded token after the prompt, and the residual trace of a single token
    nxt = toks(1, cfg["vocab"], seed=2)
    got, resid = m.forward_rows(nxt[None], 40, [0], want_residual=True)
    want, wres = o.run(nxt, want_residual=True)
    assert err(got, want) < BAR[dtype]
    if dtype == "float32":
        assert np.allclose(resid, wres, rtol=1e-4, atol=1e-4)
    m.close()


def test_stream_weights_are_indexed_from_to():
    """A mix matrix that is far from symmetric, one stream that nothing reads and one that no sublayer writes to."""
    cfg = config([latent(heads=2, ff=24), latent(heads=2)], streams=3, width=40)
    t = random_model(cfg, 4, bf16_round=False)
    for i in range(2):
        for q in ("1", "2") if i == 0 else ("1",):
            t[f"l{i}.hc{q}.mix"] = np.array([[0.0, 1.5, 0.25], [0.5, 0.0, 2.0], [1.0, -0.5, 0.0]])
            t[f"l{i}.hc{q}.in"] = np.array([0.0, 1.0, -0.75])
            t[f"l{i}.hc{q}.out"] = np.array([1.25, -0.5, 0.0])
    t = to_bf16_grid(t)
    m, o = build(cfg, tensors=t)
    ids = toks(20, cfg["vocab"], seed=5)
    want = o.run(ids)
    assert err(in_portions(m, ids, [12, 1, 3]), want) < BAR["float32"]
    for k in t:  # and the transposed matrix is another model
        if k.endswith(".mix"):
            t[k] = t[k].T.copy()
    assert err(OracleGifudra(cfg, t).run(ids), want) > 1e-2
    m.close()


MIXED = config([latent(ff=40), latent(heads=2, dim=8, rot_dim=16, vdim=16, q_rank=16, kv_rank=32, scale=0.3),
                latent(heads=5, dim=8, vdim=8, q_rank=24, scale=0.4, kv_from=0, ff=24),
                latent(heads=4, dim=24, rot_dim=16, vdim=8, q_rank=32, kv_rank=32, scale=0.2, kv_from=1, ff=32)], streams=4)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_prompt_then_token_by_token_and_portions(dtype):
    m, o = build(MIXED, seed=5, dtype=dtype, max_seq_len=160)
    n = 150
    ids = toks(n, MIXED["vocab"], seed=6)
    want = o.run(ids)
    whole = m.forward_rows(ids[None], 0, list(range(n)))
    assert err(whole, want) < BAR[dtype]
    one = np.stack([m.forward(ids[None, t:t + 1], t)[0] for t in range(n)])
    assert err(one, want) < BAR[dtype]
    # 4 / 5 and 8 / 9 tokens sit on the borders between the projections' paths and between the two forms of attention
    for sizes in ([37, 3, 2, 2], [2], [64, 1, 5, 2, 31], [9, 8, 4, 5]):
        got = in_portions(m, ids, sizes)
        assert err(got, want) < BAR[dtype], sizes
        if dtype == "float32":
            assert err(got, whole) < 2e-5
    m.close()


def test_shared_cache_rows_are_the_owner_s():
    cfg = config([latent(), latent(kv_from=0), latent(), latent(kv_from=2), latent(kv_from=0)], streams=2)
    m, o = build(cfg, seed=7)
    ids = toks(21, cfg["vocab"], seed=8)
    want = o.run(ids)
    assert err(in_portions(m, ids, [13, 8]), want) < BAR["float32"]
    for run, owner in enumerate((0, 0, 2, 2, 0)):
        cache, _ = m.read_state(run)
        st = o.state[owner]
        assert np.allclose(cache[:21], np.concatenate([np.stack(st["c"]), np.stack(st["kr"])], axis=1), rtol=1e-4, atol=1e-4)
    assert not np.allclose(m.read_state(0)[0][:21], m.read_state(2)[0][:21], atol=1e-3)
    m.close()


@pytest.mark.parametrize("change", [{"kv_rank": 40}, {"rot_dim": 16}, {"base": 500.0}])
def test_a_shared_cache_of_another_shape_is_refused(change):
    with pytest.raises(ValueError):
        build(config([latent(), latent(kv_from=0, **change)]))
    with pytest.raises(ValueError):
        build(config([latent(), latent(kv_from=0), latent(kv_from=1)]))  # layer 1 has no rows of its own
    with pytest.raises(ValueError):
        build(config([latent(kv_from=0)]))


@pytest.mark.parametrize("sink", [-30.0, 0.0, 6.0, 40.0])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_sink_counts_once_however_the_keys_are_split(sink, dtype):
    """Sinks from negligible to far above every score: prompts, portions and single tokens whose keys are split over many
    CTAs; the very first token sees itself and the sink only."""
    cfg = config([latent(heads=3, dim=16, rot_dim=16, vdim=16, kv_rank=48, scale=0.3)], streams=2)
    t = random_model(cfg, 9)
    t["l0.mix.sink"] = np.array([sink, sink - 1.0, sink + 0.5])
    m, o = build(cfg, tensors=t, dtype=dtype, max_seq_len=320)
    ids = toks(300, cfg["vocab"], seed=10)
    want, wres = o.run(ids, want_residual=True)
    total = np.sum(o.state[0]["p"][0])  # of the last token's weights, head 0
    assert abs(total - 1.0) < 1e-6 if sink < -20 else total < 1.0 - 1e-4
    got, res = m.forward_rows(ids[None, :290], 0, list(range(290)), want_residual=True)
    assert err(got, want[:290]) < BAR[dtype]
    if dtype == "float32":
        assert np.allclose(res, wres[:, :290], rtol=1e-4, atol=1e-4)
    tail = np.concatenate([m.forward_rows(ids[None, 290:292], 290, [0, 1])] + [m.forward(ids[None, i:i + 1], i) for i in range(292, 300)])
    assert err(tail, want[290:]) < BAR[dtype]
    first = m.forward(ids[None, :1], 0)
    assert err(first, want[:1]) < BAR[dtype]
    m.close()


def test_gate_is_one_number_per_value():
    """Gates driven to 0 or 1 by large weights: a gate applied per head, or read from another place, would show."""
    cfg = config([latent(heads=3, vdim=16)], streams=2)
    t = random_model(cfg, 11, bf16_round=False)
    t["l0.mix.g"] = t["l0.mix.g"] * 20.0
    t = to_bf16_grid(t)
    for dtype in ("float32", "bfloat16"):
        m, o = build(cfg, tensors=t, dtype=dtype)
        ids = toks(30, cfg["vocab"], seed=12)
        want = o.run(ids)
        assert err(in_portions(m, ids, [20, 2, 1]), want) < BAR[dtype]
        m.close()


def test_long_decoding_matches_the_oracle():
    cfg = config([latent(heads=2, dim=8, rot_dim=8, vdim=8, q_rank=16, kv_rank=24, ff=16), latent(heads=1, kv_rank=24, kv_from=0)], width=40, vocab=50)
    m, o = build(cfg, seed=13, max_seq_len=400)
    ids = toks(380, 50, seed=14)
    want = o.run(ids)
    m.forward_rows(ids[None, :20], 0, [])
    got = np.stack([m.forward(ids[None, t:t + 1], t)[0] for t in range(20, 380)])
    assert err(got, want[20:]) < BAR["float32"]
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_batch_rows_equal_single_sequences_and_slots_are_reused(dtype):
    t = random_model(MIXED, 15)
    m, o = build(MIXED, tensors=t, dtype=dtype, max_seq_len=64, max_batch_size=6)
    for B in (3, 6):  # three rows go through the GEMV, six through the batched path
        ids = np.stack([toks(30, MIXED["vocab"], seed=16 + s) for s in range(B)])
        batch = m.forward_rows(ids[:, :25], 0, list(range(25 * B)))
        step = m.forward(ids[:, 25:26], 25)
        for b in range(B):
            want = fresh(o).run(ids[b, :26])
            assert err(batch[b * 25:(b + 1) * 25], want[:25]) < BAR[dtype]
            assert err(step[b], want[25]) < BAR[dtype]
    # slot 0 held a longer sequence: a new one that starts there must not see its rows
    again = m.forward_rows(ids[2:3, :12], 0, list(range(12)))
    assert err(again, fresh(o).run(ids[2, :12])) < BAR[dtype]
    tail = m.forward(ids[2:3, 12:13], 12)
    assert err(tail, o.run(ids[2, 12:13])) < BAR[dtype]
    with pytest.raises(RuntimeError):
        m.forward(ids[:1, :1], 7)
    m.close()


def _sharp(t, layer, gain):
    t[f"l{layer}.mix.uq"] = t[f"l{layer}.mix.uq"] * gain
    t[f"l{layer}.mix.uk"] = t[f"l{layer}.mix.uk"] * gain


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_far_keys_dominate_attention(dtype):
    """Queries and keys are scaled up until the softmax is nearly one-hot, so single keys anywhere in the past carry the
    output; hundreds of tokens, in a prompt and in decoding, where the keys of a sequence are split over CTAs."""
    cfg = config([latent(heads=3, dim=16, rot_dim=8, vdim=16, q_rank=24, kv_rank=56, scale=1.0)], width=32, vocab=50, streams=2)
    t = random_model(cfg, 17)
    _sharp(t, 0, 5.0 if dtype == "float32" else 3.3)
    t = to_bf16_grid(t)
    m, o = build(cfg, tensors=t, dtype=dtype, max_seq_len=700)
    ids = toks(650, 50, seed=18)
    want = o.run(ids)
    p = np.stack(o.state[0]["p"])  # the last token's weights: peaked, and not on its neighbours
    assert p.max(axis=1).min() > 0.3 and (649 - p.argmax(axis=1)).max() > 100
    # rounded keys move a nearly tied maximum of such a sharp softmax: nine rows in ten are held to the bar in bf16
    q = 1.0 if dtype == "float32" else 0.9
    rows = lambda g, w: np.quantile([err(a[None], b[None]) for a, b in zip(g, w)], q)
    assert rows(m.forward_rows(ids[None, :600], 0, list(range(600))), want[:600]) < 2 * BAR[dtype]
    assert rows(np.stack([m.forward(ids[None, i:i + 1], i)[0] for i in range(600, 650)]), want[600:]) < 2 * BAR[dtype]
    m.close()


def planted_model(seed, token=7, gain=24.0):
    """One layer whose attention every query spends on the rows of ONE token id, wherever they are: all embeddings share a
    direction u, the one-dimensional query latent reads it and so has one sign, and the key expansion answers with the
    embedding's component along the planted token's own direction - large for that token only.  The queries' rotated part is
    zero."""
    cfg = config([latent(heads=2, dim=8, rot_dim=8, vdim=8, q_rank=1, kv_rank=56, scale=1.0)], width=24, vocab=30, embed=1.0, streams=2)
    rng = np.random.default_rng(seed)
    t = random_model(cfg, seed, bf16_round=False)
    u = np.zeros(24)
    u[0] = 1.0
    noise = rng.standard_normal((30, 24)) * 0.5
    noise[:, 0] = 0.0
    t["embed"] = u[None, :] + noise
    t["l0.norm1"] = np.ones(24)
    t["l0.hc1.in"] = np.array([0.5, 0.5])
    d = noise[token] / np.linalg.norm(noise[token])
    t["l0.mix.dq"] = 5.0 * u[None, :]
    t["l0.mix.dq.norm"] = np.ones(1)
    uq = np.zeros((2, 16, 1))
    uq[:, 0, 0] = 1.0
    t["l0.mix.uq"] = uq.reshape(32, 1)
    t["l0.mix.dkv"][0] = 3.0 * d
    t["l0.mix.dkv.norm"] = np.ones(56)
    uk = np.zeros((2, 8, 56))
    uk[:, 0, 0] = gain
    t["l0.mix.uk"] = uk.reshape(16, 56)
    t["l0.mix.sink"] = np.zeros(2)
    return cfg, to_bf16_grid(t)


@pytest.mark.parametrize("planted", [0, 31, 32, 63, 64, 127, 128, 257])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_one_planted_key_is_found_from_everywhere(planted, dtype):
    """The planted token sits once in the sequence: at the first position, at a tile's last row, at the next tile's first
    row, far inside.  Every later token must put its weight there, in a prompt, in portions and token by token."""
    cfg, t = planted_model(19)
    m, o = build(cfg, tensors=t, dtype=dtype, max_seq_len=420)
    ids = toks(400, 30, seed=20 + planted)
    ids[ids == 7] = 8
    ids[planted] = 7
    want = o.run(ids)
    p = np.stack(o.state[0]["p"])
    assert p[:, planted].min() > 0.8, p[:, planted]
    got = np.concatenate([m.forward_rows(ids[None, :250], 0, list(range(250))), m.forward_rows(ids[None, 250:300], 250, list(range(50))),
                          np.stack([m.forward(ids[None, i:i + 1], i)[0] for i in range(300, 400)])])
    assert err(got, want) < BAR[dtype]
    ids2 = ids.copy()
    ids2[planted] = 9  # without the planted row the answer is another one: the row matters
    assert err(fresh(o).run(ids2)[-1:], want[-1:]) > 2 * BAR[dtype]
    m.close()


ODD = {
    # sizes the vector and tensor-core paths do not take, and values that a usual configuration makes equal or 1
    "width_not_8": config([latent(heads=3, dim=12, rot_dim=6, vdim=10, q_rank=20, kv_rank=28, ff=10), latent(heads=1, dim=7, rot_dim=6, kv_rank=28, kv_from=0)], width=44, vocab=33),
    "width_not_4": config([latent(heads=1, dim=5, rot_dim=2, vdim=3, q_rank=7, kv_rank=9, scale=1.0, ff=7)], width=30, vocab=40, eps=1e-3, embed=1.0, logit=1.0),
    "row_not_4": config([latent(heads=5, dim=6, rot_dim=6, vdim=6, q_rank=10, kv_rank=13, scale=0.5)], width=40, vocab=25, streams=7),
    "many_heads": config([latent(heads=35, dim=4, rot_dim=4, vdim=2, q_rank=12, kv_rank=8, scale=0.5)], width=24, vocab=25),
    "wide_values": config([latent(heads=2, dim=8, rot_dim=8, vdim=72, q_rank=12, kv_rank=136, scale=0.3, ff=80)], width=48, vocab=31),
    "values_wider_than_the_latent": config([latent(heads=2, dim=8, rot_dim=8, vdim=120, q_rank=12, kv_rank=64, scale=0.3)], width=48, vocab=31),
    "long_latent": config([latent(heads=2, dim=8, rot_dim=16, vdim=8, q_rank=8, kv_rank=600, scale=0.3)], width=32, vocab=31),
    "one_of_everything": config([latent(heads=1, dim=1, rot_dim=2, vdim=1, q_rank=1, kv_rank=1, scale=1.0, ff=1)], width=8, vocab=9, streams=1, embed=1.0, logit=1.0),
}


@pytest.mark.parametrize("name", sorted(ODD))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_odd_sizes(name, dtype):
    cfg = ODD[name]
    m, o = build(cfg, seed=23, dtype=dtype)
    ids = toks(33, cfg["vocab"], seed=24)
    want = o.run(ids)
    got = np.concatenate([m.forward_rows(ids[None, :20], 0, list(range(20))), m.forward_rows(ids[None, 20:22], 20, [0, 1]),
                          np.stack([m.forward(ids[None, i:i + 1], i)[0] for i in range(22, 33)])])
    assert err(got, want) < BAR[dtype]
    m.close()


# (heads, dim, rot_dim, vdim, kv_rank): partial and several 64-entry slices on every side of the tensor-core attention
TC_SHAPES = [(2, 8, 8, 8, 56), (3, 40, 24, 48, 64), (2, 72, 64, 40, 88), (1, 128, 64, 128, 136), (2, 136, 8, 136, 72), (5, 64, 72, 192, 104),
             (4, 56, 0, 64, 128)]


@pytest.mark.parametrize("shape", TC_SHAPES)
def test_tensor_core_prompt_attention_shapes(shape):
    """bf16 prompts whose attention runs on expanded keys and values: a prompt of several query tiles, a portion behind it that
    starts inside a key block and ends inside a query tile, two sequences at once, then single tokens on the folded form."""
    H, dim, rot, dv, rank = shape
    cfg = config([latent(heads=H, dim=dim, rot_dim=rot, vdim=dv, q_rank=64, kv_rank=rank, scale=1.5 / np.sqrt(dim + rot))], width=64, vocab=60, streams=2)
    m, o = build(cfg, seed=25, dtype="bfloat16", max_seq_len=330, max_batch_size=2)
    ids = np.stack([toks(310, 60, seed=s) for s in (26, 27)])
    want = [fresh(o).run(ids[b]) for b in range(2)]
    a = m.forward_rows(ids[:, :203], 0, list(range(406)))
    c = m.forward_rows(ids[:, 203:300], 203, list(range(194)))
    tail = [m.forward(ids[:, i:i + 1], i) for i in range(300, 310)]
    for b in range(2):
        got = np.concatenate([a[b * 203:(b + 1) * 203], c[b * 97:(b + 1) * 97], np.stack([x[b] for x in tail])])
        assert err(got, want[b]) < BAR["bfloat16"]
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_library_loop(dtype):
    m, o = build(MIXED, seed=28, dtype=dtype, max_seq_len=96, max_batch_size=2)
    prompts = np.stack([toks(12, MIXED["vocab"], seed=s) for s in (29, 30)])
    lazy = np.concatenate(list(m.generate(prompts, 40)), axis=1)
    bulk = m.generate_all(prompts, 40)
    assert np.array_equal(lazy, bulk)
    # every emitted token is the oracle's argmax for the same prefix, unless its top two are closer than the error bar
    margin = 1e-3 if dtype == "float32" else 0.2
    for b in range(2):
        seq = np.concatenate([prompts[b], bulk[b]])
        lg = fresh(o).run(seq[:-1])
        for i in range(40):
            row = lg[11 + i]
            top = np.sort(row)[-2:]
            if top[1] - top[0] > margin * np.std(row):
                assert int(np.argmax(row)) == int(bulk[b, i]), f"sequence {b}, new token {i}"
    m.close()


def test_scheduler_runs_unequal_prompts_as_each_alone():
    m, _ = build(MIXED, seed=31, max_seq_len=64, max_batch_size=2)
    prompts = [toks(n, MIXED["vocab"], seed=32 + n) for n in (5, 9, 5, 2, 9)]
    outs = m.generate_ragged(prompts, 10)
    for p, got in zip(prompts, outs):
        assert np.array_equal(got, m.generate_all(p[None], 10)[0])
    m.close()


def _write_folder(tmp_path, cfg, t):
    from test_risalix_cpu import write_safetensors
    write_safetensors(tmp_path / "model.safetensors", t)
    (tmp_path / "config.json").write_text(json.dumps(cfg))


def test_registry_and_checkpoint_folder(tmp_path):
    from llama3_np_b200.models import load_model
    cfg = config([latent(heads=2, ff=24), latent(kv_from=0)], width=32, vocab=41)
    t = random_model(cfg, 33)
    _write_folder(tmp_path, cfg, t)
    m = load_model(str(tmp_path), dtype="float32", max_seq_len=32)
    assert type(m).__name__ == "Gifudra"
    ids = toks(16, 41, seed=34)
    assert err(m.forward_rows(ids[None], 0, list(range(16))), OracleGifudra(cfg, t).run(ids)) < BAR["float32"]
    m.close()


def test_missing_and_unknown_tensors_are_errors():
    from llama3_np_b200.gifudra import Gifudra
    cfg = config([latent(heads=2, ff=24), latent(kv_from=0)], width=32, vocab=41)
    t = random_model(cfg, 35)
    for drop in ("l0.hc2.mix", "l1.mix.sink", "l0.ls2", "l0.mix.dkv"):
        with pytest.raises(RuntimeError):
            Gifudra(cfg, {k: v for k, v in t.items() if k != drop})
    for name, like in (("head", "embed"), ("l1.mix.dkv", "l0.mix.dkv"), ("l1.mlp.up", "l0.mlp.up"), ("l0.mlp.gate", "l0.mlp.up")):
        with pytest.raises(ValueError):
            Gifudra(cfg, {**t, name: t[like]})
    # the feed-forward's norm, scale and stream weights of a layer that has none are ignored
    Gifudra(cfg, {**t, **{"l1." + n: t["l0." + n] for n in ("norm2", "ls2", "hc2.in", "hc2.out", "hc2.mix")}}).close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_runner_replays_a_trace(tmp_path, dtype):
    """bin/trace_run as a user runs it: two requests after one another through the same slot, portions cut in odd places
    and longer than one forward call."""
    import os
    import subprocess
    import sys
    from conftest import ROOT
    cfg = config([latent(heads=2, kv_rank=56, ff=24), latent(heads=3, kv_rank=56, kv_from=0)], width=32, vocab=41)
    t = random_model(cfg, 36)
    _write_folder(tmp_path, cfg, t)
    o = OracleGifudra(cfg, t)
    reqs = {"a": toks(43, 41, seed=37), "b": toks(9, 41, seed=38)}
    want = {k: fresh(o).run(v) for k, v in reqs.items()}
    steps, expect, n = [], {}, 0
    for rid, cuts in (("a", [31, 1, 2, 9]), ("b", [9])):
        pos = 0
        for c in cuts:
            w = [c - 1, 0] if c > 1 else [0]
            steps.append({"step": n, "entries": [{"id": rid, "tokens": [int(x) for x in reqs[rid][pos:pos + c]], "want": w}],
                          "end": [rid] if pos + c == len(reqs[rid]) else []})
            expect[n] = want[rid][[pos + i for i in w]]
            pos += c
            n += 1
    steps.append({"step": n, "entries": [], "end": []})
    out = tmp_path / "out"
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", dtype,
                        "--out", str(out), "--max-tokens", "64", "--piece", "13"],
                       input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done ")] == [f"done {i}" for i in range(n + 1)]
    for i, e in expect.items():
        assert err(np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(-1, 41), e) < BAR[dtype], i


def test_generate_command_prints_the_loop_s_tokens(tmp_path):
    import os
    import subprocess
    import sys
    from conftest import ROOT
    from llama3_np_b200.models import load_model
    cfg = config([latent(heads=2, ff=24)], width=32, vocab=47)
    _write_folder(tmp_path, cfg, random_model(cfg, 39))
    prompts = np.stack([toks(7, 47, seed=s) for s in (40, 41)])
    (tmp_path / "prompts.txt").write_text("\n".join(" ".join(str(int(x)) for x in p) for p in prompts) + "\n")
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "generate"), "--model", str(tmp_path), "--dtype", "float32",
                        "--batch-file", str(tmp_path / "prompts.txt"), "--new", "12"], capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    printed = np.array([[int(x) for x in line.split()] for line in r.stdout.strip().splitlines()[-2:]])
    m = load_model(str(tmp_path), dtype="float32", max_seq_len=19, max_batch_size=2)
    assert np.array_equal(printed, m.generate_all(prompts, 12))
    m.close()


def _random_config(rng):
    layers, owners = [], []
    W = int(rng.integers(2, 12)) * 8
    for i in range(int(rng.integers(1, 5))):
        ff = int(rng.integers(1, 9)) * 8 if rng.random() < 0.6 else None
        kw = dict(heads=int(rng.integers(1, 6)), dim=int(rng.integers(1, 8)) * 8, vdim=int(rng.integers(1, 8)) * 8, q_rank=int(rng.integers(1, 8)) * 8,
                  scale=float(rng.uniform(0.1, 0.5)), ff=ff)
        if owners and rng.random() < 0.5:
            j = int(rng.choice(owners))
            o = layers[j]["mixer"]
            layers.append(latent(rot_dim=o["rot_dim"], kv_rank=o["kv_rank"], base=o["rot"]["base"], kv_from=j, **kw))
        else:
            owners.append(i)
            layers.append(latent(rot_dim=int(rng.integers(1, 5)) * 8, kv_rank=int(rng.integers(4, 16)) * 8, base=float(rng.choice([100.0, 1e4, 1e6])), **kw))
    return config(layers, width=W, vocab=int(rng.integers(20, 120)), streams=int(rng.integers(1, 7)), eps=float(rng.choice([1e-6, 1e-3])),
                  embed=float(rng.uniform(0.5, 9.0)), logit=float(rng.uniform(0.1, 2.0)))


@pytest.mark.parametrize("seed", range(8))
def test_configurations_drawn_at_random(seed):
    rng = np.random.default_rng(100 + seed)
    cfg = _random_config(rng)
    t = random_model(cfg, seed)
    ids = toks(90, cfg["vocab"], seed=seed)
    want = OracleGifudra(cfg, t).run(ids)
    for dtype in ("float32", "bfloat16"):
        m, _ = build(cfg, tensors=t, dtype=dtype)
        got = np.concatenate([m.forward_rows(ids[None, :80], 0, list(range(80))), np.stack([m.forward(ids[None, i:i + 1], i)[0] for i in range(80, 90)])])
        assert err(got, want) < BAR[dtype], (dtype, cfg)
        cuts = [int(c) for c in rng.choice([1, 2, 3, 7, 12, 33], 6)]
        assert err(in_portions(m, ids, cuts), want) < BAR[dtype], (dtype, cuts)
        m.close()


def test_larger_shapes_take_the_tensor_core_projections():
    cfg = config([latent(heads=4, dim=32, rot_dim=32, vdim=64, q_rank=128, kv_rank=128, scale=0.1, ff=512),
                  latent(heads=2, dim=64, rot_dim=32, vdim=128, q_rank=64, kv_rank=128, scale=0.1, kv_from=0, ff=256)], width=256, vocab=300, streams=4)
    for dtype in ("bfloat16", "float32"):
        m, o = build(cfg, seed=42, dtype=dtype, max_seq_len=300)
        ids = toks(280, 300, seed=43)
        want = o.run(ids)
        got = np.concatenate([m.forward_rows(ids[None, :270], 0, list(range(270))), np.stack([m.forward(ids[None, i:i + 1], i)[0] for i in range(270, 280)])])
        assert err(got, want) < BAR[dtype]
        m.close()
