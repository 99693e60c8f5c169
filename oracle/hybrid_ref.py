"""Plain CPU restatement of the layer-list models (minGRU and windowed-attention mixers): numpy, one function per mechanism.

TEST INFRASTRUCTURE ONLY, like the rest of this folder: written from the equations, slow on purpose (attention looks at
one query at a time), and sharing nothing with the product package.  `model` is {"config": dict as config.json holds it,
"weights": name -> array}; every function works in the dtype of the arrays it gets (float64 for a yardstick).

    y = (x / rms_g(x)) * w                      rms_g over each of `groups` equal parts, eps inside the root
    S_t = (1 - z_t) S_(t-1) + z_t c_t           c = u + 1/2 (u >= 0) | sigmoid(u) (u < 0)
    o_i = sum_j e_ij v_j / (1 + sum_j e_ij)     e_ij = exp(scale q_i . k_j) for 0 <= i - j < window
"""
from __future__ import annotations

import numpy as np


# ---- mechanisms ------------------------------------------------------------------------------------------------------
def sigmoid(x):
    return np.where(x >= 0, 1.0 / (1.0 + np.exp(-np.abs(x))), np.exp(-np.abs(x)) / (1.0 + np.exp(-np.abs(x))))


def grouped_norm(x, w, groups, eps):
    part = x.reshape(*x.shape[:-1], groups, x.shape[-1] // groups)
    rms = np.sqrt((part * part).mean(axis=-1, keepdims=True) + eps)
    return (part / rms).reshape(x.shape) * w


def bigram_rows(tokens, prev, mul_prev, mul_cur, buckets):
    """Table row of every token; `prev` is the token before the first one, None at the start of a sequence."""
    rows = []
    for t in tokens:
        rows.append(buckets if prev is None else (int(prev) * mul_prev + int(t) * mul_cur) % buckets)
        prev = t
    return np.array(rows)


def mingru_scan(z, u, state):
    """z (gates) and u (candidate pre-activations) [T, width] -> all states [T, width]."""
    cand = np.where(u >= 0, u + 0.5, sigmoid(u))
    out, s = np.empty_like(u), state
    for t in range(len(u)):
        s = (1.0 - z[t]) * s + z[t] * cand[t]
        out[t] = s
    return out


def rotate_pairs(x, positions, base, dims):
    """x [T, heads, dim]: neighbours (2i, 2i + 1) of the first `dims` elements turn by position * base^(-2i / dims)."""
    out = x.copy()
    for i in range(dims // 2):
        ang = np.asarray(positions, dtype=np.float64) * float(base) ** (-2.0 * i / dims)
        c, s = np.cos(ang)[:, None].astype(x.dtype), np.sin(ang)[:, None].astype(x.dtype)
        a, b = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        out[:, :, 2 * i], out[:, :, 2 * i + 1] = a * c - b * s, b * c + a * s
    return out


def window_attention(q, k, v, first, window, scale):
    """q [T, H, dim] at positions first ..; k [n, G, dim] / v [n, G, vdim] from position 0 -> [T, H * vdim]."""
    T, H, _ = q.shape
    rep = H // k.shape[1]
    out = np.zeros((T, H, v.shape[2]), q.dtype)
    for t in range(T):
        p = first + t
        lo = max(0, p - window + 1)
        for h in range(H):
            s = k[lo:p + 1, h // rep] @ q[t, h] * scale
            m = max(float(s.max()), 0.0)           # the sink's score is 0
            e = np.exp(s - m)
            out[t, h] = (e / (np.exp(-m) + e.sum())) @ v[lo:p + 1, h // rep]
    return out.reshape(T, -1)


def mix_values(v, v_first, lam):
    return (1.0 - lam) * v + lam * v_first


def squared_relu(x):
    return np.maximum(x, 0.0) ** 2


# ---- the model -------------------------------------------------------------------------------------------------------
class HybridReference:
    """Keeps every token's keys and values and each recurrence's state; `run(tokens)` continues the sequence."""

    def __init__(self, config, weights, dtype=np.float64):
        self.cfg = config
        self.w = {k: np.asarray(v).astype(dtype) for k, v in weights.items()}
        self.dtype = dtype
        self.reset()

    def reset(self):
        self.pos, self.prev = 0, None
        self.state, self.k, self.v = {}, {}, {}

    def linear(self, x, name):
        y = x @ self.w[name].T
        return y + self.w[name + ".b"] if name + ".b" in self.w else y

    def run(self, tokens, layers_out=None):
        """Logits [T, vocab] of the next tokens; appends the residual after every layer to `layers_out`."""
        cfg, w, eps, groups = self.cfg, self.w, self.cfg["norm"]["eps"], self.cfg["norm"]["groups"]
        T = len(tokens)
        positions = np.arange(self.pos, self.pos + T)
        x = w["embed"][np.asarray(tokens)]
        bg = cfg["embedding"]["bigram"]
        x = x + w["bigram"][bigram_rows(tokens, self.prev, bg["mul_prev"], bg["mul_cur"], bg["buckets"])]
        v_first = None
        for i, layer in enumerate(cfg["layers"]):
            p, m = f"l{i}.", layer["mixer"]
            h = grouped_norm(x, w[p + "norm1"], groups, eps)
            if layer["type"] == "mingru":
                z, u = sigmoid(self.linear(h, p + "mix.z")), self.linear(h, p + "mix.x")
                s = mingru_scan(z, u, self.state.get(i, np.zeros(m["width"], self.dtype)))
                self.state[i] = s[-1]
                g = self.linear(h, p + "mix.g")
                y = self.linear(s * (g * sigmoid(g)), p + "mix.o")
            else:
                H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
                q = self.linear(h, p + "mix.q").reshape(T, H, d)
                k = self.linear(h, p + "mix.k").reshape(T, G, d)
                v = self.linear(h, p + "mix.v").reshape(T, G, dv)
                q = rotate_pairs(q, positions, m["rot"]["base"], m["rot"]["dims"])
                k = rotate_pairs(k, positions, m["rot"]["base"], m["rot"]["dims"])
                if m["v_mix"]:
                    if v_first is None:
                        v_first = v
                    else:
                        v = mix_values(v, v_first, w[p + "mix.vmix"])
                self.k[i] = np.concatenate([self.k[i], k]) if i in self.k else k
                self.v[i] = np.concatenate([self.v[i], v]) if i in self.v else v
                y = self.linear(window_attention(q, self.k[i], self.v[i], self.pos, m["mask"]["size"], m["scale"]), p + "mix.o")
            x = x + grouped_norm(y, w[p + "norm1b"], groups, eps)
            if layer["mlp"] is not None:
                h = grouped_norm(x, w[p + "norm2"], groups, eps)
                y = self.linear(squared_relu(self.linear(h, p + "mlp.up")), p + "mlp.down")
                x = x + grouped_norm(y, w[p + "norm2b"], groups, eps)
            if layers_out is not None:
                layers_out.append(x.copy())
        self.pos, self.prev = self.pos + T, tokens[-1]
        return self.linear(grouped_norm(x, w["final.norm"], groups, eps), "head")
