"""Small random models of the layer-list kind for the tests: config.json-style dictionaries, bf16-exact weights, and their
reading by the product's own parser."""
from __future__ import annotations

import numpy as np


def bf16(a: np.ndarray) -> np.ndarray:
    """Nearest bf16 values, as float32."""
    u = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32).astype(np.uint64)
    u = (u + 0x7FFF + ((u >> 16) & 1)) & 0xFFFF0000
    return u.astype(np.uint32).view(np.float32).reshape(np.shape(a))


def attention(heads, kv_heads, dim, vdim, window, dims=None, base=10000.0, scale=None, v_mix=True):
    return {"type": "attention",
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window},
                      "rot": {"base": base, "dims": dim if dims is None else dims}, "scale": dim ** -0.5 if scale is None else scale,
                      "v_mix": v_mix}}


def mingru(width):
    return {"type": "mingru", "mixer": {"width": width}}


def with_mlp(layer, ff):
    return {**layer, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(width, vocab, layers, groups=1, eps=1e-6, bigram=(53, 7, 5)):
    return {"architecture": "Bigerax", "width": width, "vocab": vocab, "norm": {"groups": groups, "eps": eps}, "layers": layers,
            "embedding": {"bigram": {"buckets": bigram[0], "mul_prev": bigram[1], "mul_cur": bigram[2]}}}


# name -> configuration.  Odd sizes, grouped heads, partial rotation, layers without mixing or without feed-forward, a window of
# one token, windows around and above a tile, one norm group and several.
CONFIGS = {
    "gqa": config(96, 203, [with_mlp(attention(6, 2, 40, 24, 33, dims=16), 88), with_mlp(mingru(72), 0),
                            with_mlp(attention(4, 2, 32, 24, 7, base=500.0), 0), with_mlp(mingru(130), 56),
                            with_mlp(attention(2, 2, 24, 40, 64, v_mix=False), 40), with_mlp(attention(8, 2, 16, 24, 1), 24)], groups=3),
    "odd": config(70, 99, [with_mlp(mingru(33), 21), with_mlp(attention(3, 3, 18, 10, 130, dims=6), 35),
                           with_mlp(attention(6, 3, 10, 10, 65, dims=10, scale=0.6), 51)], groups=7, eps=1e-3, bigram=(101, 999983, 999979)),
    "one": config(128, 64, [with_mlp(attention(1, 1, 130, 200, 20, dims=64), 72)], groups=1),
    "wide": config(512, 640, [with_mlp(mingru(256), 0), with_mlp(attention(8, 1, 64, 64, 100), 768), with_mlp(attention(16, 1, 128, 64, 300, dims=32), 512)],
                   groups=4),
}


def random_weights(cfg: dict, seed: int) -> dict:
    """name -> float32 array of bf16 values; scaled so that attention scores, gates and biases all matter."""
    rng = np.random.default_rng(seed)
    W, w = cfg["width"], {}
    mat = lambda o, i, s=1.0: bf16(rng.standard_normal((o, i)) * s / np.sqrt(i))
    vec = lambda n, s=0.3: bf16(rng.standard_normal(n) * s)
    norm = lambda: bf16(1.0 + 0.2 * rng.standard_normal(W))
    w["embed"], w["bigram"] = bf16(rng.standard_normal((cfg["vocab"], W))), bf16(rng.standard_normal((cfg["embedding"]["bigram"]["buckets"] + 1, W)))
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        w[p + "norm1"], w[p + "norm1b"] = norm(), norm()
        if l["type"] == "mingru":
            for n in "zxg":
                w[p + "mix." + n] = mat(m["width"], W, 1.5)
            w[p + "mix.z.b"], w[p + "mix.x.b"] = vec(m["width"], 1.0), vec(m["width"])
            w[p + "mix.o"] = mat(W, m["width"])
        else:
            rows = {"q": m["heads"] * m["dim"], "k": m["kv_heads"] * m["dim"], "v": m["kv_heads"] * m["vdim"]}
            for n, r in rows.items():
                w[p + "mix." + n], w[p + "mix." + n + ".b"] = mat(r, W, 1.6 if n != "v" else 1.0), vec(r)
            w[p + "mix.o"], w[p + "mix.o.b"] = mat(W, m["heads"] * m["vdim"]), vec(W)
            if m["v_mix"]:
                w[p + "mix.vmix"] = bf16(rng.uniform(0.2, 0.8, ()))
        if l["mlp"]:
            ff = l["mlp"]["ff"]
            w[p + "norm2"], w[p + "norm2b"] = norm(), norm()
            w[p + "mlp.up"], w[p + "mlp.up.b"], w[p + "mlp.down"], w[p + "mlp.down.b"] = mat(ff, W), vec(ff), mat(W, ff), vec(W)
    w["final.norm"], w["head"] = norm(), mat(cfg["vocab"], W)
    return w


def torch_weights(w: dict) -> dict:
    import torch

    return {k: torch.from_numpy(np.array(v)).to(torch.bfloat16) for k, v in w.items()}


def build_decoder(cfg: dict, w: dict, dtype: str, **options):
    from cut_b200 import bigerax
    from cut_b200.layer_list import LayerListDecoder

    t = torch_weights(w)
    c = bigerax.parse_config(cfg)
    return LayerListDecoder(c, bigerax.gather_weights(c, t.__getitem__, t.__contains__), dtype=dtype, **options)


def save_model(folder, cfg: dict, w: dict) -> str:
    import json
    import os

    from cut_b200.safetensors_io import write_safetensors

    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(folder, "model.safetensors"), torch_weights(w))
    return str(folder)


def row_errors(got: np.ndarray, want: np.ndarray) -> np.ndarray:
    """Root-mean-square difference of every row, relative to the rms of the wanted logits."""
    return np.sqrt(((np.asarray(got, np.float64) - want) ** 2).mean(axis=-1)) / np.sqrt((want ** 2).mean())
