"""Vupitar on the GPU against the plain NumPy statement of the design (oracle/ref_vupitar.py): every mechanism alone,
whole prompts against token-by-token decoding and against portions down to two tokens, batches against single sequences,
reused slots, keys just inside and just outside a chunk (planted so that one key decides the output), states of the
matrix memory, strong gates, looped blocks, routing, long decoding, odd sizes, and greedy generation through the
library's own loop and scheduler.  Small random models; fp32 mode is held to 1e-4 of the logit scale, bf16 to 6e-2."""
import json

import numpy as np
import pytest

from oracle.ref_vupitar import OracleVupitar as Oracle
from oracle.ref_vupitar import random_model

pytestmark = pytest.mark.gpu

FP32_BAR, BF16_BAR = 1e-4, 6e-2
DENSE = {"kind": "dense", "ff": 88, "limit": 1.1}
MOE = {"kind": "moe", "router": {"experts": 6, "top": 2}, "expert": {"ff": 40}, "shared": {"ff": 56}}


def left(heads=6, kv_heads=2, dim=24, vdim=40, size=11, dims=16, base=5000.0, scale=0.23):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": size}, "rot": {"base": base, "dims": dims}, "scale": scale}


def right(heads=3, dim=16, vdim=32, gate_cap=11.0):
    return {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": gate_cap}


def layer(l=None, r=None, ls=0.8, rs=1.2, mlp=DENSE):
    return {"type": "parallel", "mixer": {"left": l or left(), "right": r or right(), "left_scale": ls, "right_scale": rs}, "mlp": mlp}


def config(layers, width=96, vocab=101, loop=None, eps=1e-5, scale=3.0):
    c = {"architecture": "Vupitar", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width, "embedding": {"scale": scale}}
    if loop:
        c["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return c


def build(cfg, seed=0, dtype="float32", max_seq_len=128, max_batch_size=1, tensors=None):
    from llama3_np_b200.vupitar import Vupitar
    t = random_model(cfg, seed) if tensors is None else tensors
    return Vupitar(cfg, t, dtype=dtype, max_seq_len=max_seq_len, max_batch_size=max_batch_size), Oracle(cfg, t)


def row_errs(got, want):
    """per row: rms of the mean-free difference over the rms of the mean-free logits"""
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    d = got - want
    d = d - d.mean(-1, keepdims=True)
    w = want - want.mean(-1, keepdims=True)
    return np.sqrt((d * d).mean(-1)) / np.sqrt((w * w).mean())


def err(got, want):
    return float(row_errs(got, want).max())


def close(got, want, dtype):
    return err(got, want) < (FP32_BAR if dtype == "float32" else BF16_BAR)


def toks(n, vocab, seed=1):
    return np.random.default_rng(seed).integers(0, vocab, n)


def fresh(o):
    o.reset()
    return o


def portions(m, ids, cuts, start=0):
    """the logits of every token, the sequence fed in portions of the given sizes (the last size repeats)"""
    out, pos, k = [], 0, 0
    while pos < len(ids):
        c = min(cuts[min(k, len(cuts) - 1)], len(ids) - pos)
        out.append(m.forward_rows(ids[None, pos:pos + c], start + pos, list(range(c))))
        pos += c
        k += 1
    return np.concatenate(out)


ALONE = {
    "attention_only": dict(layers=[layer(rs=0.0, mlp=None)]),
    "matrix_memory_only": dict(layers=[layer(ls=0.0, mlp=None)]),
    "pair": dict(layers=[layer(mlp=None)]),
    "clamped_unit": dict(layers=[layer(ls=0.05, rs=0.05, mlp={"kind": "dense", "ff": 72, "limit": 0.6})]),
    "experts": dict(layers=[layer(ls=0.05, rs=0.05, mlp=MOE)]),
    "experts_without_a_shared_one": dict(layers=[layer(mlp={k: v for k, v in MOE.items() if k != "shared"})]),
    "all_experts_chosen": dict(layers=[layer(mlp=dict(MOE, router={"experts": 3, "top": 3}))]),
    "one_expert": dict(layers=[layer(mlp=dict(MOE, router={"experts": 5, "top": 1}))]),
    "loop": dict(layers=[layer(mlp=None), layer(mlp=MOE)], loop=(0, 2, 3)),
    "no_embedding_scale": dict(layers=[layer()], scale=1.0),
}


@pytest.mark.parametrize("name", sorted(ALONE))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_each_mechanism_alone(name, dtype):
    cfg = config(**ALONE[name])
    m, o = build(cfg, seed=3, dtype=dtype)
    ids = toks(40, cfg["vocab"])
    got, resid = m.forward_rows(ids[None], 0, list(range(40)), want_residual=True)
    want, wres = o.run(ids, want_residual=True)
    assert resid.shape == (len(o.runs), 40, cfg["width"])
    assert close(got, want, dtype)
    assert close(portions(m, ids, [9, 2, 1]), want, dtype)
    if dtype == "float32":
        assert np.allclose(resid, wres, rtol=1e-4, atol=1e-4)
    m.close()


MIXED = [layer(), layer(l=left(heads=4, kv_heads=1, dim=32, vdim=16, size=7, dims=32), r=right(heads=2, dim=24, vdim=56), mlp=MOE),
         layer(l=left(heads=2, kv_heads=2, dim=40, vdim=8, size=16, dims=10), r=right(heads=5, dim=8, vdim=12, gate_cap=6.0), mlp=None),
         layer(r=right(heads=4, dim=32, vdim=16), mlp=dict(MOE, router={"experts": 7, "top": 3}))]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_prompt_then_token_by_token_and_portions(dtype):
    cfg = config(MIXED, loop=(1, 3, 2))
    m, o = build(cfg, seed=5, dtype=dtype)
    ids = toks(70, cfg["vocab"], seed=6)
    want = o.run(ids)
    whole = m.forward_rows(ids[None], 0, list(range(70)))
    assert close(whole, want, dtype)
    assert close(portions(m, ids, [1]), want, dtype)
    for cuts in ([2], [3, 2, 7, 2, 17, 5, 2], [33, 2, 4], [64, 1], [8, 9]):
        got = portions(m, ids, cuts)
        assert close(got, want, dtype), cuts
        if dtype == "float32":  # the paths differ by the order of a few sums only
            assert err(got, whole) < 2e-5, cuts
    m.close()


@pytest.mark.parametrize("loop", [None, (0, 3, 1), (0, 3, 2), (2, 3, 4), (1, 2, 2), (0, 1, 5)])
def test_loop_bounds_steps_and_the_embedding_output(loop):
    cfg = config([layer(mlp=None), layer(mlp=MOE), layer()], width=48, loop=loop)
    m, o = build(cfg, seed=9)
    assert m.n_runs == len(o.runs)
    ids = toks(24, cfg["vocab"], seed=10)
    want, wres = o.run(ids, want_residual=True)
    got, resid = m.forward_rows(ids[None], 0, list(range(24)), want_residual=True)
    assert err(got, want) < FP32_BAR
    assert np.allclose(resid, wres, rtol=1e-4, atol=1e-4)
    assert err(portions(m, ids, [7, 2, 9, 1]), want) < FP32_BAR
    m.close()


def test_long_decoding_matches_the_oracle():
    """160 tokens one by one behind a short prompt: chunks of 7, 11 and 16 positions end and start among decoded tokens."""
    cfg = config(MIXED)
    m, o = build(cfg, seed=11, max_seq_len=192)
    ids = toks(165, cfg["vocab"], seed=12)
    assert err(portions(m, ids, [5, 1]), o.run(ids)) < FP32_BAR
    m.close()


def test_batch_rows_equal_single_sequences_and_slots_are_reused():
    cfg = config(MIXED[:3], loop=(0, 2, 2))
    m, o = build(cfg, seed=13, max_batch_size=3)
    seqs = np.stack([toks(26, cfg["vocab"], seed=s) for s in (14, 15, 16)])
    want = np.stack([fresh(o).run(s) for s in seqs])
    pos = 0
    for n in (17, 2, 1, 1, 5):  # the batch as a whole, continued in portions of unequal sizes and single tokens
        got = m.forward_rows(seqs[:, pos:pos + n], pos, list(range(3 * n))).reshape(3, n, -1)
        assert err(got, want[:, pos:pos + n]) < FP32_BAR, pos
        pos += n
    # slot 0 starts another sequence at position 0: nothing of the old one is left
    other = toks(20, cfg["vocab"], seed=17)
    assert err(m.forward_rows(other[None], 0, list(range(20))), fresh(o).run(other)) < FP32_BAR
    # and a shorter one after a longer one, fed token by token (cache rows past its position hold the old sequence)
    short = toks(6, cfg["vocab"], seed=18)
    assert err(portions(m, short, [1]), fresh(o).run(short)) < FP32_BAR
    m.close()


@pytest.mark.parametrize("batch", [2, 4, 7])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_decoded_batches_equal_each_alone(batch, dtype):
    """Single-token calls of 2 .. 7 rows take other projection kernels than a row alone."""
    cfg = config([layer(mlp=MOE), layer()], width=128, vocab=160)
    m, o = build(cfg, seed=70, dtype=dtype, max_batch_size=batch)
    seqs = np.stack([toks(14, 160, seed=71 + s) for s in range(batch)])
    want = np.stack([fresh(o).run(s) for s in seqs])
    m.forward_rows(seqs[:, :9], 0, [0])
    for p in range(9, 14):
        assert close(m.forward_rows(seqs[:, p:p + 1], p, list(range(batch))), want[:, p], dtype), p
    m.close()


def bf16(a):
    """Rounded to bfloat16, so that both modes load the same numbers."""
    a = np.ascontiguousarray(a, dtype=np.float32)
    return ((a.view(np.uint32) + 0x8000) & 0xFFFF0000).view(np.float32)


def planted(cfg, t, key_tok, query_tok):
    """Rewrites layer 0's attention so that the key of `key_tok` stands out for the query of `query_tok`: both point along the
    entries that do not rotate, every other query and key lies in the rotating ones, whose norm weights are small; the key's
    value is large."""
    o = Oracle(cfg, t)
    W, mc = cfg["width"], cfg["layers"][0]["mixer"]["left"]
    H, G, dk, dv, rd = mc["heads"], mc["kv_heads"], mc["dim"], mc["vdim"], mc["rot"]["dims"]
    t = dict(t)

    def h_of(tok):
        x = o.t["embed"][tok] * cfg["embedding"]["scale"]
        return o.norm(x, o.layers[0], "norm1")

    # directions that answer to one token only: dual vectors of the tokens' inputs
    D = np.linalg.pinv(np.stack([h_of(k) for k in range(cfg["vocab"])]).T)
    u = np.zeros(dk)
    u[rd:] = 1.0
    rng = np.random.default_rng(0)
    base = np.concatenate([np.ones(rd), np.zeros(dk - rd)])
    for nm, n, tok in (("q", H, query_tok), ("k", G, key_tok)):
        noise = 0.1 * rng.standard_normal((n * dk, W)) * np.tile(base, n)[:, None]
        t[f"l0.mix.left.{nm}"] = bf16(noise + 20.0 * np.outer(np.tile(u, n), D[tok]))
        t[f"l0.mix.left.{nm}.b"] = bf16(0.05 * rng.standard_normal(n * dk))
        t[f"l0.mix.left.{nm}.norm"] = bf16(np.where(u > 0, 1.0, 0.25))
    t["l0.mix.left.v"] = bf16(t["l0.mix.left.v"] + 15.0 * np.outer(np.ones(G * dv), D[key_tok]))
    t["l0.mix.left.g"] = np.zeros((H, W), np.float32)
    return t


@pytest.mark.parametrize("kv_heads, vdim", [(1, 40), (2, 64), (4, 32)])   # decoded by the tiled kernel / by the decode kernel
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_planted_key_just_inside_and_just_outside_a_chunk(kv_heads, vdim, dtype):
    """One key decides the attention's output.  It sits at the chunk's first position, right ahead of it, at the chunk's
    middle, right ahead of the query, in the chunk before; the query is the last token of a prompt, of a portion of two
    tokens, or decoded alone, and sits inside a chunk, at a chunk's last and at a chunk's first position."""
    size = 37
    l = left(heads=4, kv_heads=kv_heads, dim=24, vdim=vdim, size=size, dims=8, scale=0.9)
    cfg = config([layer(l=l, ls=2.0, rs=0.1, mlp=None)], vocab=60, width=96)
    KEY, QUERY = 58, 59
    t = planted(cfg, random_model(cfg, 19), KEY, QUERY)
    m, o = build(cfg, dtype=dtype, tensors=t, max_seq_len=160)
    for n in (4 * size - 9, 3 * size, 3 * size + 1):   # the query is token n - 1
        start = (n - 1) // size * size
        outs = {}
        for at in sorted({start, start - 1, (start + n - 1) // 2, n - 2, start - size + 1} - {n - 1}):
            ids = toks(n, 58, seed=20)  # ids below the two special tokens
            ids[at], ids[n - 1] = KEY, QUERY
            want = fresh(o).run(ids)
            outs[at] = want[-1]
            assert close(m.forward_rows(ids[None], 0, [n - 1]), want[-1:], dtype), ("prompt", n, at)
            got = portions(m, ids, [n - 30, 13, 15, 2])
            assert close(got[-2:], want[-2:], dtype), ("portion of two", n, at)
            got = portions(m, ids, [n - 1, 1])
            assert close(got[-1:], want[-1:], dtype), ("decoded", n, at)
        if start in outs:  # the planted key is worth seeing: inside and outside differ by far more than the error bar
            assert err(outs[start], outs[start - 1]) > 0.3
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_norm_weights_biases_and_gates_matter(dtype):
    """Large biases, uneven norm weights and open / shut gates: dropping any of them shows."""
    cfg = config([layer(mlp=None), layer(mlp=None)], vocab=50)
    t = random_model(cfg, 21)
    rng = np.random.default_rng(22)
    for i in range(2):
        p = f"l{i}.mix.left."
        for nm in ("q", "k", "v", "o"):
            t[p + nm + ".b"] = bf16(rng.standard_normal(t[p + nm + ".b"].shape))
        t[p + "q.norm"] = bf16(rng.uniform(0.2, 1.5, t[p + "q.norm"].shape))
        t[p + "k.norm"] = bf16(rng.uniform(-1.5, 1.5, t[p + "k.norm"].shape))
        t[p + "g"] = bf16(2.0 * t[p + "g"])
    m, o = build(cfg, dtype=dtype, tensors=t)
    ids = toks(30, 50, seed=22)
    want = o.run(ids)
    assert close(m.forward_rows(ids[None], 0, list(range(30))), want, dtype)
    assert close(portions(m, ids, [9, 2, 1]), want, dtype)
    m.close()
    for nm in ("q.b", "k.b", "v.b", "o.b", "g"):
        t2 = dict(t)
        for i in range(2):
            t2[f"l{i}.mix.left.{nm}"] = np.zeros_like(t[f"l{i}.mix.left.{nm}"])
        assert err(Oracle(cfg, t2).run(ids), want) > 100 * FP32_BAR, nm


def test_states_after_a_prompt_and_after_a_slot_is_used_again():
    """The matrix memories, normalisers and running maxima a prompt leaves, read back from the slot; then the same slot runs
    another sequence in portions and must hold that sequence's state only."""
    cfg = config([layer(mlp=None), layer(r=right(heads=2, dim=20, vdim=12), mlp=None)], width=48, vocab=50, loop=(0, 2, 2))
    m, o = build(cfg, seed=38)

    def check(ids):
        for run in range(len(o.runs)):
            S, rest = m.read_state(run)
            st = o.state[run]["right"]
            H, dk = st["n"].shape
            assert np.allclose(S, st["S"], rtol=1e-4, atol=1e-5), run
            assert np.allclose(rest[:H * dk].reshape(H, dk), st["n"], rtol=1e-4, atol=1e-5), run
            assert np.allclose(rest[H * dk:], st["m"], rtol=1e-4, atol=1e-5), run

    ids = toks(21, 50, seed=39)
    m.forward(ids[None], 0)
    fresh(o).run(ids)
    check(ids)
    other = toks(9, 50, seed=40)
    portions(m, other, [4, 1, 2, 1, 1])
    fresh(o).run(other)
    check(other)
    m.close()


@pytest.mark.parametrize("shape", [(16, 32), (64, 64), (128, 192), (192, 64), (20, 12)])
@pytest.mark.parametrize("strong", [False, True])
def test_matrix_memory_over_long_prompts(shape, strong):
    """Prompts of 128 tokens and more run chunk-parallel for states of 64, 128, 192 x multiples of 64 and token by token for the
    others; decode steps run in one launch.  All must agree, also with gates at both ends of their range (a forgotten
    past, a dominating token, a normaliser below its floor)."""
    dk, dv = shape
    cfg = config([layer(ls=0.0, r=right(heads=2, dim=dk, vdim=dv, gate_cap=15.0), mlp=None)], width=64, vocab=80)
    t = random_model(cfg, 46)
    if strong:
        t["l0.mix.right.i"] = (12.0 * t["l0.mix.right.i"]).astype(np.float32)
        t["l0.mix.right.f"] = (12.0 * t["l0.mix.right.f"]).astype(np.float32)
        t["l0.mix.right.i.b"] = np.array([6.0, -8.0], np.float32)
        t["l0.mix.right.f.b"] = np.array([-4.0, 5.0], np.float32)
    m, o = build(cfg, tensors=t, max_seq_len=400)
    ids = toks(330, 80, seed=47)
    want = o.run(ids)
    whole = m.forward_rows(ids[None], 0, list(range(330)))
    assert err(whole, want) < FP32_BAR
    mixed = portions(m, ids, [130, 3, 150, 1, 1, 40, 1])
    assert err(mixed, want) < FP32_BAR
    assert err(mixed, whole) < 3e-5
    S, rest = m.read_state(0)
    st = o.state[0]["right"]
    scale = np.abs(st["S"]).max()
    assert np.abs(S - st["S"]).max() < 1e-4 * scale
    assert np.abs(rest[-2:] - st["m"]).max() < 1e-4
    m.close()
    if strong:   # logits of gates at the ends of their range turn a bf16 input's rounding into factors: fp32 mode only
        return
    # bf16 mode: the same prompts with queries, keys and values as bf16 operands of warp-level tensor products
    m, _ = build(cfg, tensors=t, dtype="bfloat16", max_seq_len=400)
    assert err(m.forward_rows(ids[None], 0, list(range(330))), want) < BF16_BAR
    S2, rest2 = m.read_state(0)
    assert np.abs(S2 - st["S"]).max() < 2e-2 * scale and np.abs(rest2[:2 * dk].reshape(2, dk) - st["n"]).max() < 2e-2 * np.abs(st["n"]).max()
    assert err(portions(m, ids, [130, 3, 150, 1, 1, 40, 1]), want) < BF16_BAR
    m.close()


def test_keys_far_away_through_the_matrix_memory():
    """Chunks of 4 positions: what a token 200 places back said can only arrive through the matrix memories."""
    cfg = config([layer(l=left(heads=2, kv_heads=1, dim=8, vdim=8, size=4, dims=8)), layer(l=left(heads=2, kv_heads=1, dim=8, vdim=8, size=4, dims=8))],
                 width=48, vocab=50)
    t = random_model(cfg, 23)
    for i in range(2):
        t[f"l{i}.mix.right.f.b"] = np.full(3, 9.0, np.float32)   # slow decays: the memory lasts
    m, o = build(cfg, tensors=t, max_seq_len=256)
    ids = toks(230, 50, seed=24)
    ids2 = ids.copy()
    ids2[10] = (ids[10] + 7) % 50
    want, want2 = o.run(ids), fresh(o).run(ids2)
    assert err(want[-1:], want2[-1:]) > 1e-3   # the far token is felt at the end
    for seq, w in ((ids, want), (ids2, want2)):
        assert err(m.forward_rows(seq[None], 0, [229]), w[-1:]) < FP32_BAR
        assert err(portions(m, seq, [100, 2, 97, 1])[-1:], w[-1:]) < FP32_BAR
    m.close()


def test_routing_is_sharp_and_every_expert_is_used():
    """A router that chooses clearly and differently from token to token; the chosen experts' weights are far from equal."""
    mlp = {"kind": "moe", "router": {"experts": 9, "top": 3}, "expert": {"ff": 24}, "shared": {"ff": 16}}
    cfg = config([layer(ls=0.1, rs=0.1, mlp=mlp)], vocab=70)
    t = random_model(cfg, 60)
    t["l0.mlp.router"] = (3.0 * t["l0.mlp.router"]).astype(np.float32)
    t["l0.mlp.shared.sg"] = (4.0 * t["l0.mlp.shared.sg"]).astype(np.float32)
    m, o = build(cfg, tensors=t)
    ids = toks(64, 70, seed=61)
    want = o.run(ids)
    assert err(m.forward_rows(ids[None], 0, list(range(64))), want) < FP32_BAR
    assert err(portions(m, ids, [1, 2, 8, 5]), want) < FP32_BAR
    m.close()


ODD = {
    "ones": dict(layers=[layer(l=left(heads=1, kv_heads=1, dim=8, vdim=8, size=1, dims=0), r=right(heads=1, dim=1, vdim=1),
                               mlp={"kind": "moe", "router": {"experts": 1, "top": 1}, "expert": {"ff": 8}, "shared": {"ff": 8}})], width=40, loop=(0, 1, 1)),
    "off_the_grid": dict(layers=[layer(l=left(heads=6, kv_heads=2, dim=10, vdim=36, size=5, dims=6), r=right(heads=3, dim=12, vdim=20), mlp={"kind": "dense", "ff": 52, "limit": 2.0}),
                                 layer(l=left(heads=3, kv_heads=3, dim=12, vdim=68, size=200, dims=4), r=right(heads=5, dim=13, vdim=7),
                                       mlp={"kind": "moe", "router": {"experts": 5, "top": 4}, "expert": {"ff": 20}, "shared": {"ff": 36}})], width=120, loop=(0, 2, 2)),
    "odd_width": dict(layers=[layer(l=left(heads=3, kv_heads=1, dim=6, vdim=5, size=9, dims=2), r=right(heads=2, dim=5, vdim=9), mlp={"kind": "dense", "ff": 33, "limit": 0.9}),
                              layer(mlp={"kind": "moe", "router": {"experts": 3, "top": 2}, "expert": {"ff": 15}, "shared": {"ff": 11}})], width=62),
    "wide_groups": dict(layers=[layer(l=left(heads=8, kv_heads=1, dim=32, vdim=64, size=13, dims=32), r=right(heads=2, dim=16, vdim=16), mlp=None),
                                layer(l=left(heads=16, kv_heads=1, dim=16, vdim=16, size=150, dims=4), r=right(heads=1, dim=8, vdim=128), mlp=None),
                                layer(l=left(heads=8, kv_heads=2, dim=256, vdim=32, size=21, dims=0, scale=0.08), mlp=None)], width=96),
    "wide_heads": dict(layers=[layer(l=left(heads=2, kv_heads=1, dim=128, vdim=128, size=17, dims=64, scale=0.09), r=right(heads=1, dim=256, vdim=256)),
                               layer(l=left(heads=2, kv_heads=2, dim=64, vdim=256, size=8, dims=32, scale=0.12), r=right(heads=2, dim=64, vdim=384))], width=128),
}


@pytest.mark.parametrize("name", sorted(ODD))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_odd_sizes(name, dtype):
    cfg = config(vocab=77, **ODD[name])
    m, o = build(cfg, seed=25, dtype=dtype)
    ids = toks(45, 77, seed=26)
    want = o.run(ids)
    assert close(m.forward_rows(ids[None], 0, list(range(45))), want, dtype)
    assert close(portions(m, ids, [11, 2, 1, 1, 20, 3]), want, dtype)
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_library_loop(dtype):
    cfg = config(MIXED, loop=(0, 2, 2))
    m, o = build(cfg, seed=27, dtype=dtype, max_seq_len=96, max_batch_size=2)
    prompts = np.stack([toks(12, cfg["vocab"], seed=s) for s in (28, 29)])
    lazy = np.concatenate(list(m.generate(prompts, 40)), axis=1)
    bulk = m.generate_all(prompts, 40)
    assert np.array_equal(lazy, bulk)
    # teacher-forced: every emitted token is the oracle's argmax for the same prefix, unless the oracle's top two
    # are closer than the mode's error bar
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
    cfg = config(MIXED[:3], loop=(1, 2, 2))
    m, _ = build(cfg, seed=30, max_seq_len=64, max_batch_size=2)
    prompts = [toks(n, cfg["vocab"], seed=31 + n) for n in (5, 9, 5, 2, 9)]
    outs = m.generate_ragged(prompts, 10)
    for p, got in zip(prompts, outs):
        assert np.array_equal(got, m.generate_all(p[None], 10)[0])
    m.close()


def _write_folder(tmp_path, cfg, t):
    from test_risalix_cpu import write_safetensors
    write_safetensors(tmp_path / "model.safetensors", t)
    (tmp_path / "config.json").write_text(json.dumps(cfg))


def test_registry_checkpoint_folder_and_tensors_no_layer_reads(tmp_path):
    from llama3_np_b200.models import load_model
    cfg = config([layer(mlp=None), layer(mlp=MOE)], width=48, vocab=41)
    t = random_model(cfg, 32)
    t.update({"l0.norm2": np.ones(48, np.float32), "l0.norm2.b": np.zeros(48, np.float32), "l0.norm2.alpha": np.float32(1.0)})
    _write_folder(tmp_path, cfg, t)
    m = load_model(str(tmp_path), dtype="float32", max_seq_len=32)
    assert type(m).__name__ == "Vupitar"
    ids = toks(16, 41, seed=33)
    assert err(m.forward_rows(ids[None], 0, list(range(16))), Oracle(cfg, t).run(ids)) < FP32_BAR
    m.close()
    del t["l1.mix.right.f.b"]
    with pytest.raises(Exception, match="l1.mix.right.f.b"):
        build(cfg, tensors=t)


def test_trace_runner_replays_a_trace(tmp_path):
    """bin/trace_run as a user runs it: two requests after one another through the same slot, portions cut in odd
    places and longer than one forward call."""
    import os
    import subprocess
    import sys
    from conftest import ROOT
    cfg = config([layer(mlp=MOE), layer(), layer(mlp=None)], width=48, vocab=41, loop=(0, 2, 2))
    t = random_model(cfg, 34)
    _write_folder(tmp_path, cfg, t)
    o = Oracle(cfg, t)
    reqs = {"a": toks(23, 41, seed=35), "b": toks(9, 41, seed=36)}
    want = {k: fresh(o).run(v) for k, v in reqs.items()}
    steps, expect, n = [], {}, 0
    for rid, cuts in (("a", [11, 1, 2, 9]), ("b", [9])):
        pos = 0
        for c in cuts:
            w = [0, c - 1] if c > 1 else [0]
            steps.append({"step": n, "entries": [{"id": rid, "tokens": [int(x) for x in reqs[rid][pos:pos + c]], "want": w}],
                          "end": [rid] if pos + c == len(reqs[rid]) else []})
            expect[n] = want[rid][[pos + i for i in w]]
            pos += c
            n += 1
    steps.append({"step": n, "entries": [], "end": []})
    out = tmp_path / "out"
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32",
                        "--out", str(out), "--max-tokens", "64", "--piece", "5"],
                       input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done ")] == [f"done {i}" for i in range(n + 1)]
    for i, e in expect.items():
        got = np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(-1, 41)
        assert err(got, e) < FP32_BAR, i


def test_generate_command_prints_the_loop_s_tokens(tmp_path):
    import os
    import subprocess
    import sys
    from conftest import ROOT
    from llama3_np_b200.models import load_model
    cfg = config([layer(), layer(mlp=MOE)], width=48, vocab=47, loop=(1, 2, 2))
    _write_folder(tmp_path, cfg, random_model(cfg, 41))
    prompts = np.stack([toks(7, 47, seed=s) for s in (42, 43)])
    (tmp_path / "prompts.txt").write_text("\n".join(" ".join(str(int(x)) for x in p) for p in prompts) + "\n")
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "generate"), "--model", str(tmp_path), "--dtype", "float32",
                        "--batch-file", str(tmp_path / "prompts.txt"), "--new", "12"], capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    printed = np.array([[int(x) for x in line.split()] for line in r.stdout.strip().splitlines()[-2:]])
    m = load_model(str(tmp_path), dtype="float32", max_seq_len=19, max_batch_size=2)
    assert np.array_equal(printed, m.generate_all(prompts, 12))
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_wide_chunks_over_several_key_tiles(dtype):
    """Chunks of 150 and 70 positions over a prompt of 400: a query's keys span several tiles of keys, tiles of queries straddle
    chunk borders, and short portions split the keys over CTAs."""
    cfg = config([layer(l=left(heads=4, kv_heads=2, dim=32, vdim=16, size=150, dims=16, scale=0.2), mlp=None),
                  layer(l=left(heads=2, kv_heads=2, dim=16, vdim=48, size=70, dims=8, scale=0.3), mlp=None)], width=64, vocab=90)
    m, o = build(cfg, seed=44, dtype=dtype, max_seq_len=420)
    ids = toks(400, 90, seed=45)
    want = o.run(ids)
    assert close(m.forward_rows(ids[None], 0, list(range(400))), want, dtype)
    assert close(portions(m, ids, [130, 2, 64, 3, 100, 8, 1, 1, 50, 5, 1]), want, dtype)
    m.close()


def test_random_configurations():
    """Sizes, chunk lengths, feed-forwards and loops drawn at random; whole prompts, portions, decoded tokens."""
    rng = np.random.default_rng(37)
    for case in range(8):
        layers = []
        for _ in range(int(rng.integers(1, 4))):
            g = int(rng.choice([1, 2, 3]))
            dim = int(rng.choice([8, 16, 20, 32]))
            l = left(heads=g * int(rng.choice([1, 2, 4])), kv_heads=g, dim=dim, vdim=int(rng.choice([8, 24, 40])), size=int(rng.integers(1, 30)),
                     dims=int(rng.choice([0, 4, 8, dim])), base=float(rng.choice([100.0, 1e4, 1e6])), scale=float(rng.uniform(0.1, 0.5)))
            r = right(heads=int(rng.integers(1, 5)), dim=int(rng.choice([4, 8, 16, 64])), vdim=int(rng.choice([8, 16, 24, 64])), gate_cap=float(rng.uniform(3, 20)))
            kind = int(rng.integers(0, 4))
            mlp = [None, DENSE, MOE, {"kind": "moe", "router": {"experts": int(rng.integers(2, 20)), "top": 2}, "expert": {"ff": int(rng.choice([8, 24]))}}][kind]
            layers.append(layer(l=l, r=r, ls=float(rng.uniform(0.3, 1.5)), rs=float(rng.uniform(0.3, 1.5)), mlp=mlp))
        a = int(rng.integers(0, len(layers)))
        b = int(rng.integers(a + 1, len(layers) + 1))
        loop = (a, b, int(rng.integers(1, 4))) if rng.integers(0, 3) else None
        cfg = config(layers, width=int(rng.choice([48, 72, 96])), vocab=int(rng.integers(20, 90)), loop=loop, eps=float(rng.choice([1e-6, 1e-3])),
                     scale=float(rng.uniform(1, 8)))
        m, o = build(cfg, seed=40 + case)
        n = int(rng.integers(20, 60))
        ids = toks(n, cfg["vocab"], seed=50 + case)
        want = o.run(ids)
        assert err(m.forward_rows(ids[None], 0, list(range(n))), want) < FP32_BAR, case
        cuts = [int(x) for x in rng.integers(1, 9, 6)] + [1]
        assert err(portions(m, ids, cuts), want) < FP32_BAR, (case, cuts)
        m.close()


@pytest.mark.parametrize("moe", [False, True])
def test_larger_shapes_take_the_tensor_core_projections(moe):
    """Width 256 and 64 rows and more: bf16 mode runs the tcgen05 projections and the chunk-parallel matrix memory."""
    mlp = {"kind": "moe", "router": {"experts": 8, "top": 2}, "expert": {"ff": 128}, "shared": {"ff": 256}} if moe else {"kind": "dense", "ff": 512, "limit": 1.2}
    cfg = config([layer(l=left(heads=4, kv_heads=2, dim=64, vdim=64, size=80, dims=32, scale=0.15), r=right(heads=2, dim=64, vdim=128), mlp=mlp),
                  layer(l=left(heads=8, kv_heads=2, dim=32, vdim=32, size=48, dims=32, scale=0.18), r=right(heads=2, dim=128, vdim=128), mlp=mlp)],
                 width=256, vocab=300, loop=(0, 2, 2))
    m, o = build(cfg, seed=60, dtype="bfloat16", max_seq_len=200)
    ids = toks(170, 300, seed=61)
    want = o.run(ids)
    m.launch_count(reset=True)
    # a rounded router input may turn a close choice: rows whose scores are close are left out of the expert model's bar
    e = row_errs(m.forward_rows(ids[None], 0, list(range(170))), want)
    assert m.launch_count() > 0
    assert (np.quantile(e, 0.9) if moe else e.max()) < BF16_BAR
    e = row_errs(portions(m, ids, [140, 20, 2, 7, 1]), want)
    assert (np.quantile(e, 0.9) if moe else e.max()) < BF16_BAR
    m.close()


# ---- the new mechanisms in stacks of another make: the library's stack takes them as parameters
class _Sequential(Oracle):
    """x <- x + mixer(n1(x)); x <- x + ff(n2(x))"""

    def layer(self, i, x, st, pos):
        lc = self.c["layers"][i]
        only_mixer = dict(self.c, layers=[dict(l, mlp=None) for l in self.c["layers"]])
        full, self.c = self.c, only_mixer
        x = super().layer(i, x, st, pos)
        self.c = full
        if lc.get("mlp") is not None:
            from oracle import ref_vupitar as R
            P = self.layers[i]
            h, F = self.norm(x, P, "norm2"), R.sub(P, "mlp.")
            x = x + (R.mixture(h, lc["mlp"], F) if lc["mlp"]["kind"] == "moe" else R.clamped_unit(h, F, lc["mlp"]["limit"]))
        return x


class _Rms(Oracle):
    def norm(self, x, P, name):
        return x / np.sqrt((x * x).mean() + self.c["norm"]["eps"]) * P[name]


@pytest.mark.parametrize("make", ["tanh_sequential", "rms_dual"])
def test_the_mechanisms_combine_with_other_stacks(make):
    import dataclasses
    from llama3_np_b200.stack import StackDecoder
    from llama3_np_b200.vupitar import stack_config
    cfg = config([layer(), layer(mlp=MOE), layer(mlp=None)], width=64, vocab=60, loop=(0, 2, 2))
    t = random_model(cfg, 80)
    sc = stack_config(cfg, max_seq_len=64)
    if make == "tanh_sequential":
        sc, o = dataclasses.replace(sc, dual_norm=False), _Sequential(cfg, t)
    else:
        sc, o = dataclasses.replace(sc, norm_tanh=False), _Rms(cfg, t)
        t = {k: v for k, v in t.items() if not k.endswith(("norm1.b", "norm2.b", "final.norm.b", ".alpha"))}
    m = StackDecoder(sc)
    m.load_tensors(t)
    ids = toks(40, 60, seed=81)
    want = o.run(ids)
    assert err(m.forward_rows(ids[None], 0, list(range(40))), want) < FP32_BAR
    assert err(portions(m, ids, [13, 2, 1, 9]), want) < FP32_BAR
    m.close()


def test_unsupported_combinations_are_refused():
    import dataclasses
    from llama3_np_b200.stack import StackDecoder
    from llama3_np_b200.vupitar import stack_config
    sc = stack_config(config([layer()]))
    for bad in (dict(token_shift=True), dict(norm_groups=2), dict(streams=2), dict(layer_scale=True), dict(loop_x0=True)):
        with pytest.raises(ValueError):
            StackDecoder(dataclasses.replace(sc, **bad))
    spec = dataclasses.replace(sc.layers[0], pair=dataclasses.replace(sc.layers[0].pair, gate_cap=0.0))
    with pytest.raises(ValueError):
        StackDecoder(dataclasses.replace(sc, layers=[spec]))


@pytest.mark.parametrize("case", ["chunks", "wide_values", "off_the_grid"])
def test_prompts_of_wide_heads_attend_on_the_tensor_cores(case):
    """Heads of 64 and more in bf16 mode: portions of more than 8 tokens run the tensor-core kernel, shorter ones the exact one.
    Chunks end inside query tiles, key blocks start at a chunk's first position, portions start inside a chunk; a sharp
    softmax over few keys makes a wrong edge show."""
    l = {"chunks": left(heads=4, kv_heads=2, dim=64, vdim=64, size=75, dims=32, scale=0.3),
         "wide_values": left(heads=3, kv_heads=1, dim=128, vdim=128, size=190, dims=128, scale=0.2),
         "off_the_grid": left(heads=2, kv_heads=2, dim=72, vdim=88, size=33, dims=24, scale=0.25)}[case]
    cfg = config([layer(l=l, rs=0.2, mlp=None), layer(l=dict(l, mask={"size": 400}), rs=0.2, mlp=None)], width=128, vocab=150)
    m, o = build(cfg, seed=90, dtype="bfloat16", max_seq_len=420, max_batch_size=2)
    seqs = np.stack([toks(400, 150, seed=s) for s in (91, 92)])
    want = np.stack([fresh(o).run(s) for s in seqs])
    whole = m.forward_rows(seqs, 0, list(range(800))).reshape(2, 400, -1)
    assert err(whole[0], want[0]) < BF16_BAR and err(whole[1], want[1]) < BF16_BAR
    for cuts in ([130, 2, 64, 9, 100, 8, 1, 1, 50, 17, 1], [12], [399, 1]):
        assert err(portions(m, seqs[0], cuts), want[0]) < BF16_BAR, cuts
    m.close()


def test_planted_keys_at_chunk_edges_on_the_tensor_cores():
    """As the planted keys above, for heads the tensor-core kernel takes: the query ends a prompt, or a portion of 20 tokens."""
    size = 67
    l = left(heads=4, kv_heads=2, dim=64, vdim=64, size=size, dims=16, scale=0.5)
    cfg = config([layer(l=l, ls=2.0, rs=0.1, mlp=None)], vocab=40, width=256)
    KEY, QUERY = 38, 39
    m, o = build(cfg, dtype="bfloat16", tensors=planted(cfg, random_model(cfg, 19), KEY, QUERY), max_seq_len=300)
    for n in (4 * size - 9, 3 * size, 3 * size + 2):
        start = (n - 1) // size * size
        outs = {}
        for at in sorted({start, start - 1, n - 2, start - size + 1}):
            ids = toks(n, 38, seed=20)
            ids[at], ids[n - 1] = KEY, QUERY
            want = fresh(o).run(ids)
            outs[at] = want[-1]
            assert err(m.forward_rows(ids[None], 0, [n - 1]), want[-1:]) < BF16_BAR, ("prompt", n, at)
            assert err(portions(m, ids, [n - 20, 20])[-1:], want[-1:]) < BF16_BAR, ("portion", n, at)
            assert err(portions(m, ids, [n - 1, 1])[-1:], want[-1:]) < BF16_BAR, ("decoded", n, at)
        assert err(outs[start], outs[start - 1]) > 0.3
    m.close()
