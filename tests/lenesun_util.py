"""Small random models with latent attention and mixtures of experts for the tests: config.json-style dictionaries, bf16-exact
weights, their reading by the product's own parser, and token sequences on which no router has a close call (a choice that
rounding may turn over says nothing about the arithmetic)."""
from __future__ import annotations

import numpy as np

from oracle import latent_ref as R
from tests.layer_list_util import bf16, save_model, torch_weights

__all__ = ["CONFIGS", "bf16", "config", "layer", "random_weights", "safe_tokens", "build_decoder", "save_model", "torch_weights",
           "SandwichReference", "sandwich_decoder"]


def layer(heads, dim, rot, vdim, q_rank, kv_rank, experts=0, top=0, ff=0, *, base=10000.0, scale=None, limit=2.0, kv_from=None):
    mixer = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
             "rot": {"base": base, "dims": rot}, "scale": (dim + rot) ** -0.5 if scale is None else scale}
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    mlp = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit}} if experts else None
    return {"type": "latent_attention", "mixer": mixer, "mlp": mlp}


def config(width, vocab, layers, eps=1e-5, mult=0.5, scale=1.5):
    return {"architecture": "Lenesun", "width": width, "vocab": vocab, "layers": layers, "norm": {"eps": eps}, "residual_mult": mult,
            "embedding": {"scale": scale}}


# name -> configuration.  Layers of unlike sizes, shared latents (not of the nearest layer, by layers with other head counts), odd
# widths and ranks that no vector width divides, one expert, all experts, layers without a feed-forward, head parts above and
# below the tile sizes, factors of one.
CONFIGS = {
    "mixed": config(136, 211, [layer(3, 24, 16, 40, 56, 48, 6, 2, 40), layer(5, 16, 8, 24, 40, 72, base=500.0),
                               layer(2, 40, 16, 16, 24, 48, 9, 3, 24, kv_from=0, limit=0.7), layer(7, 8, 8, 8, 72, 72, 4, 1, 88, kv_from=1, base=500.0)],
                    mult=0.4, scale=2.5),
    "odd": config(70, 99, [layer(3, 10, 6, 7, 21, 35, 5, 5, 13), layer(1, 9, 2, 30, 17, 35, 1, 1, 22), layer(4, 3, 6, 5, 33, 35, 7, 2, 9, kv_from=0)],
                  eps=1e-3, mult=1.0, scale=1.0),
    "big": config(128, 160, [layer(2, 128, 64, 128, 64, 256, 8, 2, 64, limit=1.0), layer(2, 192, 64, 200, 96, 160, 6, 2, 32), layer(1, 64, 0, 96, 64, 160)],
                  mult=0.7),
    "wide": config(512, 640, [layer(16, 64, 32, 64, 192, 256, 32, 4, 128), layer(16, 64, 32, 64, 192, 256, 32, 6, 96, kv_from=0)], eps=1e-6, mult=0.25,
                   scale=3.5),
}


def random_weights(cfg: dict, seed: int) -> dict:
    """name -> float32 array of bf16 values; scaled so that scores, sinks, clamps, biases and routers all matter."""
    rng = np.random.default_rng(seed)
    W, w = cfg["width"], {}
    mat = lambda o, i, s=1.0: bf16(rng.standard_normal((o, i)) * s / np.sqrt(i))
    norm = lambda n: bf16(1.0 + 0.25 * rng.standard_normal(n))
    w["embed"] = bf16(rng.standard_normal((cfg["vocab"], W)) + 0.4)  # (rows with a mean: a norm that does not take it off shows)
    for i, l in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", l["mixer"], l["mlp"]
        H, k = m["heads"], m["dim"] + m["rot_dim"]
        w[p + "norm1"] = norm(W)
        w[p + "mix.dq"], w[p + "mix.dq.norm"], w[p + "mix.uq"] = mat(m["q_rank"], W), norm(m["q_rank"]), mat(H * k, m["q_rank"], 2.0)
        if m.get("kv_from") is None:
            w[p + "mix.dkv"], w[p + "mix.dkv.norm"] = mat(m["kv_rank"] + m["rot_dim"], W, 1.5), norm(m["kv_rank"])
        w[p + "mix.uk"], w[p + "mix.uv"] = mat(H * m["dim"], m["kv_rank"], 1.5), mat(H * m["vdim"], m["kv_rank"])
        w[p + "mix.sink"], w[p + "mix.o"] = bf16(rng.standard_normal(H) * 1.5 + 2.0), mat(W, H * m["vdim"], 2.0)
        if f:
            E, n = f["router"]["experts"], f["expert"]["ff"]
            w[p + "mlp.router"], w[p + "mlp.router.b"] = mat(E, W), bf16(0.3 * rng.standard_normal(E))
            for e in range(E):
                q = f"{p}mlp.e{e}."
                w[q + "gate"], w[q + "up"], w[q + "down"] = mat(n, W, 1.5), mat(n, W, 1.5), mat(W, n)
    w["final.norm"] = norm(W)
    return w


def safe_tokens(ref, n: int, seed: int, margin: float = 0.06) -> np.ndarray:
    """n random tokens, each drawn again until every router's choice on it is clear; leaves `ref` reset."""
    rng, V, out = np.random.default_rng(seed), ref.cfg["vocab"], []
    ref.reset()
    while len(out) < n:
        at = ref.pos
        for _ in range(200):
            t = int(rng.integers(0, V))
            ref.run([t])
            if ref.margin[0] > margin:
                break
            ref.forget(at)
        else:
            raise RuntimeError("no token with clear choices")
        out.append(t)
    ref.reset()
    return np.array(out)


def build_decoder(cfg: dict, w: dict, dtype: str, **options):
    from cut_b200 import lenesun
    from cut_b200.layer_list import LayerListDecoder

    t = torch_weights(w)
    c = lenesun.parse_config(cfg)
    return LayerListDecoder(c, lenesun.gather_weights(c, t.__getitem__, t.__contains__), dtype=dtype, **options)


# ---- the same mechanisms between norms of their own (no model of the registry has this yet) ------------------------------------
class SandwichReference(R.LatentReference):
    """x <- x + RMS(f(RMS(x))) for the attention, then for the experts, with the weights' extra norms; untied head."""

    def run(self, tokens, layers_out=None):
        self.margin = np.full(len(tokens), np.inf)
        cfg, w, eps = self.cfg, self.w, self.cfg["norm"]["eps"]
        positions = np.arange(self.pos, self.pos + len(tokens))
        x = w["embed"][np.asarray(tokens)]
        for i, l in enumerate(cfg["layers"]):
            p = f"l{i}."
            x = x + R.rms_norm(self.attention(i, l["mixer"], R.rms_norm(x, w[p + "norm1"], eps), positions), w[p + "norm1b"], eps)
            if l["mlp"] is not None:
                x = x + R.rms_norm(self.experts(i, l["mlp"], R.rms_norm(x, w[p + "norm2"], eps)), w[p + "norm2b"], eps)
            if layers_out is not None:
                layers_out.append(x.copy())
        self.pos += len(tokens)
        return R.rms_norm(x, w["final.norm"], eps) @ w["head"].T


def sandwich_decoder(cfg: dict, w: dict, dtype: str, **options):
    from dataclasses import replace

    from cut_b200 import lenesun
    from cut_b200.layer_list import LayerListDecoder

    t = torch_weights(w)
    c = lenesun.parse_config(cfg)
    weights = lenesun.gather_weights(c, t.__getitem__, t.__contains__)
    weights["head"] = t["head"]
    for i, d in enumerate(weights["layers"]):
        d.update({n: t[f"l{i}.{n}"] for n in ("norm1b", "norm2", "norm2b")})
    c = replace(c, parallel=False, norm_center=False, residual_mult=1.0, embed_scale=1.0, tied_head=False)
    return LayerListDecoder(c, weights, dtype=dtype, **options)
