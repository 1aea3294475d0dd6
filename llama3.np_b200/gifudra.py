"""Gifudra: a pre-norm decoder with several residual streams per token (hyper-connections).  Every sublayer reads a
weighted sum of the streams, and its result - times a weight per channel (layer scale) - re-mixes all of them; the
final norm reads their sum.  The mixer is latent attention: one cached row per token (a normed latent and a rotated
key part shared by all heads), queries through a latent of their own, rotary pairs (i, i + dims / 2), a sink per head
in the softmax denominator, a sigmoid gate per value; a layer may attend over another layer's cached rows
(`kv_from`).  The feed-forward is `down(relu(up x)^2)`, the output projection is the embedding table.
The arithmetic lives in the library's layer-list path (csrc/layerlist.cu, attn_latent.cu, stream_ops.cu); this file
reads `config.json`, names the tensors and builds the `StackConfig`.  The reference has one fixed block
(llama3.py:238-262) and no counterpart of this.

A checkpoint folder holds `config.json` (keys: architecture, vocab, width, embedding.scale, norm.eps, streams,
logit_scale, layers[].type / mixer / mlp) and `model.safetensors` (tensor names `embed`, `l<i>.norm1`, `l<i>.norm2`,
`l<i>.ls1`, `l<i>.ls2`, `l<i>.hc1.in / out / mix`, `l<i>.hc2.*`, `l<i>.mix.*`, `l<i>.mlp.up / down`, `final.norm`).
"""
from __future__ import annotations

import json
import os
from typing import Mapping, Optional

import numpy as np

from .stack import FF_RELU2, LATENT, LayerSpec, StackConfig, StackDecoder
from .utils import read_safetensors


def stack_config(config: Mapping, *, max_seq_len: int = 256, max_batch_size: int = 1, dtype: str = "float32") -> StackConfig:
    """`config.json` (as a dict) -> StackConfig."""
    layers = []
    for i, lc in enumerate(config["layers"]):
        if lc["type"] != "latent_attention":
            raise ValueError(f"layer {i}: unknown mixer type {lc['type']!r}")
        mc = lc["mixer"]
        if mc.get("kv_from") is not None:  # what a shared cache fixes comes from its owner where the layer does not repeat it
            owner = config["layers"][int(mc["kv_from"])]["mixer"]
            mc = {**{k: owner[k] for k in ("kv_rank", "rot_dim", "rot") if k in owner}, **mc}
        rot, rot_dim = mc.get("rot") or {}, int(mc.get("rot_dim", 0))
        kv_from = mc.get("kv_from")
        spec = LayerSpec(mixer=LATENT, heads=int(mc["heads"]), dim=int(mc["dim"]), vdim=int(mc["vdim"]),
                         q_rank=int(mc["q_rank"]), kv_rank=int(mc["kv_rank"]), rot_dim=rot_dim,
                         rot_dims=int(rot.get("dims", rot_dim)), rot_base=float(rot.get("base", 10000.0)), rot_layout=1,
                         scale=float(mc["scale"]), kv_from=None if kv_from is None else int(kv_from), sink=True, gate_wide=True)
        mlp = lc.get("mlp")
        if mlp is not None:
            if mlp.get("kind", "dense") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
            spec.ff, spec.ff_kind = int(mlp["ff"]), FF_RELU2
        layers.append(spec)
    return StackConfig(width=int(config["width"]), vocab=int(config["vocab"]), layers=layers,
                       norm_eps=float(config["norm"]["eps"]), norm_one_plus=False, norm_input=True, layer_scale=True,
                       embed_scale=float((config.get("embedding") or {}).get("scale", 1.0)),
                       streams=int(config.get("streams") or 0), tied_head=True,
                       logit_scale=float(config.get("logit_scale", 1.0)),
                       max_seq_len=max_seq_len, max_batch_size=max_batch_size, dtype=dtype)


class Gifudra(StackDecoder):
    architecture = "Gifudra"

    def __init__(self, config: Mapping, tensors: Optional[Mapping[str, np.ndarray]] = None, *, max_seq_len: int = 256,
                 max_batch_size: int = 1, dtype: str = "float32", device: int = 0, random_seed: Optional[int] = None,
                 flags: int = 0):
        """`tensors`: checkpoint name -> array; or None with `random_seed` for random weights on the device."""
        if tensors is None and random_seed is None:
            raise ValueError("tensors=None needs random_seed")
        self.config = dict(config)
        super().__init__(stack_config(config, max_seq_len=max_seq_len, max_batch_size=max_batch_size, dtype=dtype),
                         device=device, flags=flags)
        if tensors is not None:
            # a layer without a feed-forward reads none of these, whether or not the checkpoint holds them
            unused = tuple(f"l{i}.{n}" for i, lc in enumerate(config["layers"]) if lc.get("mlp") is None for n in ("norm2", "ls2", "hc2."))
            self.load_tensors({k: v for k, v in tensors.items() if not k.startswith(unused)} if unused else tensors)
        else:
            self.fill_random(random_seed)

    @classmethod
    def from_pretrained(cls, model_dir, **kw) -> "Gifudra":
        with open(os.path.join(model_dir, "config.json")) as f:
            config = json.load(f)
        return cls(config, read_safetensors(os.path.join(model_dir, "model.safetensors")), **kw)
