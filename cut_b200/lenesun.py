"""Lenesun: a decoder of latent-attention layers with a mixture of experts beside each of them (one layer norm feeds both) and a
tied, scaled embedding, as a configuration of LayerListDecoder, and the reader of its config.json and tensor names."""
from __future__ import annotations

import torch

from . import _lib as L
from .layer_list import LatentAttention, Layer, LayerListConfig, MixtureOfExperts, Rotation

ARCHITECTURE = "Lenesun"
GLU_ALPHA, GLU_BETA = 1.702, 1.0    # g sigmoid(alpha g) (u + beta)


def parse_config(c: dict) -> LayerListConfig:
    layers = []
    for i, l in enumerate(c["layers"]):
        m = l["mixer"]
        if l["type"] != "latent_attention":
            raise ValueError(f"layer {i}: unknown mixer {l['type']!r}")
        if int(m["rot"]["dims"]) != int(m["rot_dim"]):
            raise ValueError(f"layer {i}: the rotated part of {m['rot_dim']} elements turns as a whole, not by {m['rot']['dims']}")
        mixer = LatentAttention(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), q_rank=int(m["q_rank"]), kv_rank=int(m["kv_rank"]),
                                scale=float(m["scale"]), rot=Rotation(float(m["rot"]["base"]), int(m["rot_dim"]), L.ROT_NEIGHBOURS), sink=True,
                                kv_from=None if m.get("kv_from") is None else int(m["kv_from"]))
        mlp = l.get("mlp")
        if mlp is not None:
            if mlp["kind"] != "moe":
                raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
            mlp = MixtureOfExperts(experts=int(mlp["router"]["experts"]), top=int(mlp["router"]["top"]), ff=int(mlp["expert"]["ff"]),
                                   limit=float(mlp["expert"]["limit"]), alpha=GLU_ALPHA, beta=GLU_BETA)
        layers.append(Layer(mixer, mlp))
    return LayerListConfig(width=int(c["width"]), vocab=int(c["vocab"]), layers=tuple(layers), norm_groups=1, norm_eps=float(c["norm"]["eps"]),
                           norm_center=True, parallel=True, residual_mult=float(c["residual_mult"]), embed_scale=float(c["embedding"]["scale"]),
                           tied_head=True)


def gather_weights(cfg: LayerListConfig, get, has) -> dict:
    """Tensor names of the file -> the structure LayerListDecoder takes.  get(name) -> tensor, has(name) -> bool."""
    out = {"embed": get("embed"), "final_norm": get("final.norm"), "layers": []}
    for i, l in enumerate(cfg.layers):
        p, m, f = f"l{i}.", l.mixer, l.mlp
        names = ["dq", "dq.norm", "uq", "uk", "uv", "sink", "o"] + (["dkv", "dkv.norm"] if m.kv_from is None else [])
        d = {"norm1": get(p + "norm1"), "mix": {n: get(p + "mix." + n) for n in names}}
        if f is not None:
            d["mlp"] = {n: torch.stack([get(f"{p}mlp.e{e}.{n}") for e in range(f.experts)]) for n in ("gate", "up", "down")}
            d["mlp"].update({"router": get(p + "mlp.router"), "router.b": get(p + "mlp.router.b")})
        out["layers"].append(d)
    return out
