"""Bigerax: a decoder of minGRU and sliding-window-attention layers with norms around every sublayer and a bigram embedding,
as a configuration of LayerListDecoder, and the reader of its config.json and tensor names."""
from __future__ import annotations

import torch

from . import _lib as L
from .layer_list import Bigram, FeedForward, GatedRecurrence, Layer, LayerListConfig, Rotation, WindowAttention

ARCHITECTURE = "Bigerax"


def parse_config(c: dict) -> LayerListConfig:
    layers = []
    for i, l in enumerate(c["layers"]):
        m = l["mixer"]
        if l["type"] == "mingru":
            mixer = GatedRecurrence(width=int(m["width"]))
        elif l["type"] == "attention":
            mixer = WindowAttention(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                                    window=int(m["mask"]["size"]), scale=float(m["scale"]),
                                    rot=Rotation(float(m["rot"]["base"]), int(m["rot"]["dims"]), L.ROT_NEIGHBOURS), sink=True,
                                    v_mix=bool(m.get("v_mix", False)))
        else:
            raise ValueError(f"layer {i}: unknown mixer {l['type']!r}")
        mlp = l.get("mlp")
        if mlp is not None:
            if mlp["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
            mlp = FeedForward(int(mlp["ff"]), L.UNARY_RELU_SQUARE)
        layers.append(Layer(mixer, mlp))
    b = c["embedding"]["bigram"]
    return LayerListConfig(width=int(c["width"]), vocab=int(c["vocab"]), layers=tuple(layers), norm_groups=int(c["norm"]["groups"]),
                           norm_eps=float(c["norm"]["eps"]), bigram=Bigram(int(b["buckets"]), int(b["mul_prev"]), int(b["mul_cur"])))


def gather_weights(cfg: LayerListConfig, get, has) -> dict:
    """Tensor names of the file -> the structure LayerListDecoder takes.  get(name) -> tensor, has(name) -> bool."""
    def linear(prefix, names):
        d = {}
        for n in names:
            d[n] = get(prefix + n)
            if has(prefix + n + ".b"):
                d[n + ".b"] = get(prefix + n + ".b")
        return d

    out = {"embed": get("embed"), "bigram": get("bigram"), "head": get("head"), "final_norm": get("final.norm"), "layers": []}
    for i, l in enumerate(cfg.layers):
        p = f"l{i}."
        d = {"norm1": get(p + "norm1"), "norm1b": get(p + "norm1b")}
        if isinstance(l.mixer, WindowAttention):
            d["mix"] = linear(p + "mix.", ["q", "k", "v", "o"])
            if l.mixer.v_mix and i != cfg.first_mixing:
                d["mix"]["vmix"] = float(get(p + "mix.vmix").to(torch.float32).reshape(-1)[0])
        else:
            d["mix"] = linear(p + "mix.", ["z", "x", "g", "o"])
        if l.mlp is not None:
            d["norm2"], d["norm2b"] = get(p + "norm2"), get(p + "norm2b")
            d["mlp"] = linear(p + "mlp.", ["up", "down"])
        out["layers"].append(d)
    return out
