"""Plain CPU restatement of the parallel latent-attention / mixture-of-experts models (Lenesun): numpy, one function per
mechanism.

TEST INFRASTRUCTURE ONLY, like the rest of this folder: written from the equations, slow on purpose (attention looks at one
query at a time, the experts at one token at a time), and sharing nothing with the product package.  Every function works in
the dtype of the arrays it gets (float64 for a yardstick).

    x_0 = s E[token];   h = LN(x),  x <- x + m (A(h) + F(h));   logits = E LN(x)
    LN(x) = (x - mean x) / sqrt(mean (x - mean x)^2 + eps) * w          RMS(x) = x / sqrt(mean x^2 + eps) * w
    A:  q = W_uq RMS(W_dq h),  (a, r) = W_dkv h,  c = RMS(a),  r turned at its position
        s_ij = scale (q_i . W_uk c_j + turned q'_i . r_j),   o_i = sum_j e^s_ij (W_uv c_j) / (e^sink + sum_j e^s_ij),  j <= i
    F:  sum over the chosen experts of softmax weight * W_down(g sigmoid(1.702 g) (u + 1)),
        g = min(W_gate h, L), u = clip(W_up h, -L, L)
"""
from __future__ import annotations

import numpy as np


# ---- mechanisms ------------------------------------------------------------------------------------------------------
def layer_norm(x, w, eps):
    d = x - x.mean(axis=-1, keepdims=True)
    return d / np.sqrt((d * d).mean(axis=-1, keepdims=True) + eps) * w


def rms_norm(x, w, eps):
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps) * w


def turn_pairs(x, positions, base):
    """x [T, ..., n]: neighbours (2i, 2i + 1) turn by position * base^(-2i / n)."""
    n, out = x.shape[-1], np.empty_like(x)
    shape = (len(positions),) + (1,) * (x.ndim - 2)
    for i in range(n // 2):
        ang = np.asarray(positions, np.float64).reshape(shape) * float(base) ** (-2.0 * i / n)
        c, s = np.cos(ang).astype(x.dtype), np.sin(ang).astype(x.dtype)
        a, b = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = a * c - b * s, b * c + a * s
    return out


def sink_attention(q, k, v, first, scale, sink):
    """q [T, H, d] at positions first ..; k [n, H, d], v [n, H, e] from position 0; sink [H] or None -> [T, H * e]."""
    T, H, _ = q.shape
    out = np.zeros((T, H, v.shape[2]), q.dtype)
    for t in range(T):
        n = first + t + 1
        for h in range(H):
            s = k[:n, h] @ q[t, h] * scale
            m = s.max() if sink is None else max(s.max(), sink[h])
            e = np.exp(s - m)
            out[t, h] = (e / (e.sum() + (0.0 if sink is None else np.exp(sink[h] - m)))) @ v[:n, h]
    return out.reshape(T, -1)


def latent_keys_values(c, r, w_uk, w_uv, heads):
    """Every head's keys [n, H, dim + rot] and values [n, H, vdim] from the latents c [n, rank] and turned key parts r [n, rot]."""
    n = len(c)
    k = (c @ w_uk.T).reshape(n, heads, -1)
    return np.concatenate([k, np.repeat(r[:, None, :], heads, axis=1)], axis=2), (c @ w_uv.T).reshape(n, heads, -1)


def sigmoid(x):
    e = np.exp(-np.abs(x))
    return np.where(x >= 0, 1.0 / (1.0 + e), e / (1.0 + e))


def clamped_glu(g, u, limit):
    g, u = np.minimum(g, limit), np.clip(u, -limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


def choose_experts(z, top):
    """Indices of the `top` largest of z, and the softmax over them."""
    ids = np.argsort(-z, kind="stable")[:top]
    e = np.exp(z[ids] - z[ids].max())
    return ids, e / e.sum()


def choice_margin(logits, top):
    """How far the last chosen logit lies above the first one left out, in standard deviations of a token's logits."""
    z = -np.sort(-logits, axis=-1)
    return np.full(len(z), np.inf) if top == z.shape[1] else (z[:, top - 1] - z[:, top]) / z.std(axis=-1)


def mixture(h, logits, gate, up, down, top, limit):
    """h [T, W]; logits [T, E]; gate / up / down: lists of matrices."""
    out = np.zeros_like(h)
    for t in range(len(h)):
        for e, w in zip(*choose_experts(logits[t], top)):
            out[t] += w * (down[e] @ clamped_glu(gate[e] @ h[t], up[e] @ h[t], limit))
    return out


# ---- the model -------------------------------------------------------------------------------------------------------
class LatentReference:
    """Keeps every token's latent and turned key part; `run(tokens)` continues the sequence."""

    def __init__(self, config, weights, dtype=np.float64):
        self.cfg, self.dtype = config, dtype
        self.w = {k: np.asarray(v).astype(dtype) for k, v in weights.items()}
        self.reset()

    def reset(self):
        self.pos, self.c, self.r = 0, {}, {}

    def forget(self, n):
        """Back to the first n positions."""
        self.pos, self.c, self.r = n, {i: a[:n] for i, a in self.c.items()}, {i: a[:n] for i, a in self.r.items()}

    def attention(self, i, m, h, positions):
        w, p, eps, T = self.w, f"l{i}.mix.", self.cfg["norm"]["eps"], len(h)
        H, dim, rank = m["heads"], m["dim"], m["kv_rank"]
        q = (rms_norm(h @ w[p + "dq"].T, w[p + "dq.norm"], eps) @ w[p + "uq"].T).reshape(T, H, dim + m["rot_dim"])
        q = np.concatenate([q[:, :, :dim], turn_pairs(q[:, :, dim:], positions, m["rot"]["base"])], axis=2)
        j = m.get("kv_from")
        if j is None:
            j = i
            a = h @ w[p + "dkv"].T
            c, r = rms_norm(a[:, :rank], w[p + "dkv.norm"], eps), turn_pairs(a[:, rank:], positions, m["rot"]["base"])
            self.c[i] = np.concatenate([self.c[i], c]) if i in self.c else c
            self.r[i] = np.concatenate([self.r[i], r]) if i in self.r else r
        k, v = latent_keys_values(self.c[j], self.r[j], w[p + "uk"], w[p + "uv"], H)
        return sink_attention(q, k, v, self.pos, m["scale"], w[p + "sink"]) @ w[p + "o"].T

    def experts(self, i, f, h):
        w, p, E = self.w, f"l{i}.mlp.", f["router"]["experts"]
        part = lambda n: [w[f"{p}e{e}.{n}"] for e in range(E)]
        logits = h @ w[p + "router"].T + w[p + "router.b"]
        self.margin = np.minimum(self.margin, choice_margin(logits, f["router"]["top"]))
        return mixture(h, logits, part("gate"), part("up"), part("down"), f["router"]["top"], f["expert"]["limit"])

    def run(self, tokens, layers_out=None):
        """Logits [T, vocab] of the next tokens; appends the residual after every layer to `layers_out`.  `margin` [T] is left as the
        closest call any router had on each token."""
        self.margin = np.full(len(tokens), np.inf)
        cfg, w, eps = self.cfg, self.w, self.cfg["norm"]["eps"]
        positions = np.arange(self.pos, self.pos + len(tokens))
        x = w["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
        for i, layer in enumerate(cfg["layers"]):
            h = layer_norm(x, w[f"l{i}.norm1"], eps)
            y = self.attention(i, layer["mixer"], h, positions)
            if layer["mlp"] is not None:
                y = y + self.experts(i, layer["mlp"], h)
            x = x + cfg["residual_mult"] * y
            if layers_out is not None:
                layers_out.append(x.copy())
        self.pos += len(tokens)
        return layer_norm(x, w["final.norm"], eps) @ w["embed"].T
