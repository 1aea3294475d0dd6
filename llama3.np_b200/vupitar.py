"""Vupitar: a decoder whose sublayers both read the same residual stream, each through an element-wise norm of its own
(dynamic tanh, `tanh(alpha x) w + b`), and add their results to it at once.  The mixer of every layer is a pair, summed
with fixed weights: softmax attention inside chunks of the sequence - biased projections, an RMS norm with a weight per
query and key head, rotary pairs (i, i + dims / 2), a sigmoid gate per head - beside a matrix memory with exponential
gates (mLSTM).  The feed-forward is a clamped gated unit or a mixture of gated experts (softmax router, the best `top`
over their own sum) with a shared expert behind a sigmoid gate.  A block of layers may run several times with one set of
weights: ahead of every pass its step vector joins the stream, from the second pass on the embedding output, too.

The arithmetic lives in the library's layer-list path (csrc/layerlist.cu, attn_window.cu, mlstm.cu, recur_chunk.cu,
tanh_norm.cu, moe.cu); this file reads `config.json`, names the tensors and builds the `StackConfig`.  The reference has
one fixed block (llama3.py:238-262) and no counterpart of this.

A checkpoint folder holds `config.json` (keys: architecture, vocab, width, embedding.scale, norm.eps, loop.start / stop /
times, layers[].type / mixer / mlp) and `model.safetensors` (tensor names `embed`, `loop.step`, `l<i>.norm1`, `l<i>.norm2`
with `.b` and `.alpha`, `l<i>.mix.left.q / k / v / o` with `.b`, `l<i>.mix.left.q.norm / k.norm / g`, `l<i>.mix.right.q / k /
v / g / o / norm / i / i.b / f / f.b`, `l<i>.mlp.gate / up / down` or `l<i>.mlp.router`, `l<i>.mlp.e<j>.*`,
`l<i>.mlp.shared.*`, `l<i>.mlp.shared.sg`, `final.norm`, `head`).
"""
from __future__ import annotations

import json
import os
from typing import Mapping, Optional

import numpy as np

from .stack import ATTN_SOFTMAX, FF_CLAMP, MLSTM, ROUTE_SOFTMAX_GLU, WINDOW, LayerSpec, StackConfig, StackDecoder
from .utils import read_safetensors

FF_SLOPE = 1.702   # slope of the clamped unit's sigmoid, fixed by the design


def _left(mc: Mapping) -> LayerSpec:
    rot, mask = mc.get("rot") or {}, mc.get("mask") or {}
    return LayerSpec(mixer=WINDOW, heads=int(mc["heads"]), kv_heads=int(mc.get("kv_heads", mc["heads"])), dim=int(mc["dim"]),
                     vdim=int(mc["vdim"]), scale=float(mc["scale"]), window=int(mask.get("size", 0)), chunked=True,
                     rot_dims=int(rot.get("dims", 0)), rot_base=float(rot.get("base", 10000.0)), rot_layout=1,
                     attn_kind=ATTN_SOFTMAX, qk_norm=True, proj_bias=True, head_gate=True)


def _right(mc: Mapping) -> LayerSpec:
    return LayerSpec(mixer=MLSTM, heads=int(mc["heads"]), dim=int(mc["dim"]), vdim=int(mc["vdim"]), gate_cap=float(mc["gate_cap"]))


def stack_config(config: Mapping, *, max_seq_len: int = 256, max_batch_size: int = 1, dtype: str = "float32") -> StackConfig:
    """`config.json` (as a dict) -> StackConfig."""
    layers = []
    for i, lc in enumerate(config["layers"]):
        if lc["type"] != "parallel":
            raise ValueError(f"layer {i}: unknown layer type {lc['type']!r}")
        mc = lc["mixer"]
        spec = _left(mc["left"])
        spec.pair, spec.mix_scale, spec.pair_scale = _right(mc["right"]), float(mc["left_scale"]), float(mc["right_scale"])
        mlp = lc.get("mlp")
        if mlp is not None:
            kind = mlp.get("kind", "dense")
            if kind == "dense":
                spec.ff, spec.ff_kind, spec.ff_limit, spec.ff_slope = int(mlp["ff"]), FF_CLAMP, float(mlp["limit"]), FF_SLOPE
            elif kind == "moe":
                shared = mlp.get("shared")
                spec.ff, spec.router_kind = int(mlp["expert"]["ff"]), ROUTE_SOFTMAX_GLU
                spec.experts, spec.top = int(mlp["router"]["experts"]), int(mlp["router"]["top"])
                spec.shared_ff, spec.shared_gate = (int(shared["ff"]), True) if shared else (0, False)
            else:
                raise ValueError(f"layer {i}: unknown feed-forward kind {kind!r}")
        layers.append(spec)
    lp = config.get("loop")
    loop = (int(lp["start"]), int(lp["stop"]), int(lp["times"])) if lp and int(lp.get("times", 0)) > 0 else None
    return StackConfig(width=int(config["width"]), vocab=int(config["vocab"]), layers=layers,
                       norm_eps=float((config.get("norm") or {}).get("eps", 1e-6)), norm_one_plus=False, norm_input=True,
                       norm_tanh=True, dual_norm=True, loop=loop, loop_x0=loop is not None,
                       embed_scale=float((config.get("embedding") or {}).get("scale", 1.0)),
                       max_seq_len=max_seq_len, max_batch_size=max_batch_size, dtype=dtype)


class Vupitar(StackDecoder):
    architecture = "Vupitar"

    def __init__(self, config: Mapping, tensors: Optional[Mapping[str, np.ndarray]] = None, *, max_seq_len: int = 256,
                 max_batch_size: int = 1, dtype: str = "float32", device: int = 0, random_seed: Optional[int] = None,
                 flags: int = 0):
        """`tensors`: checkpoint name -> array; or None with `random_seed` for random weights on the device."""
        if tensors is None and random_seed is None:
            raise ValueError("tensors=None needs random_seed")
        self.config = dict(config)
        sc = stack_config(config, max_seq_len=max_seq_len, max_batch_size=max_batch_size, dtype=dtype)
        super().__init__(sc, device=device, flags=flags)
        if tensors is not None:
            # tensors no token ever reads, whether or not the checkpoint holds them: the second norm of a layer without a
            # feed-forward, the step vectors of a block that never runs
            unused = tuple(f"l{i}.norm2" for i, l in enumerate(sc.layers) if l.ff == 0) + (() if sc.loop else ("loop.step",))
            skip = {n + e for n in unused for e in ("", ".b", ".alpha")}
            self.load_tensors({k: v for k, v in tensors.items() if k not in skip} if skip else tensors)
        else:
            self.fill_random(random_seed)

    @classmethod
    def from_pretrained(cls, model_dir, **kw) -> "Vupitar":
        with open(os.path.join(model_dir, "config.json")) as f:
            config = json.load(f)
        return cls(config, read_safetensors(os.path.join(model_dir, "model.safetensors")), **kw)
