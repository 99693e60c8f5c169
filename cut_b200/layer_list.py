"""Decoder for models whose configuration lists their layers: each layer has a mixer (windowed attention, latent attention or a
gated recurrence) and possibly a feed-forward (dense, or a mixture of experts) over dense bf16 weights.  Either every sublayer
has norms before and after it, or (parallel) one norm feeds the layer's mixer and feed-forward and their sum joins the residual.

Prefill runs a portion of a prompt as one batch: tensor-core GEMMs (bf16) or fp32 FMA GEMMs (the 32-bit mode), the scan of
the recurrence, the tiled attentions, the experts' grouped GEMMs over expert-sorted rows, and one launch per sublayer border that
adds the output (post-normed; the chosen experts' rows gathered and weighted) to the residual and norms it for the next
sublayer.  A decode step is recorded into a CUDA graph per sequence place: two launches for a recurrent layer's mixer (norms
and residual fused into the input staging of the projection, the state update and output gate into its epilogue), three for a
window-attention layer's, two for a feed-forward; a latent-attention layer takes six, in which its experts' matrices share the
launches of the query and the output projection.  The residual stream, the norms, the recurrence and its states, the rotation
angles, the scores, the softmax and the router are fp32 in both modes; decode mat-vecs use the fp32 activations as they are.

A sequence place holds, per window-attention layer, ring caches of keys and values (a position lives in row position %
ring_rows; the ring covers the window and one portion), per latent-attention layer that has its own a cache of latents and
rotated key parts (a row per position; layers with kv_from read another layer's), per recurrent layer its fp32 state, and
{token, previous token, position} on the device, so a recorded step replays for every token.
"""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass

import numpy as np
import torch

from . import _lib as L
from . import ops
from .decoding import RecordedStep


def pad(n: int, m: int) -> int:
    return (n + m - 1) // m * m


# ---- configuration ---------------------------------------------------------------------------------------------------
@dataclass(frozen=True)
class Rotation:
    base: float
    dims: int                       # leading elements of a head that rotate
    pairing: int = L.ROT_NEIGHBOURS


@dataclass(frozen=True)
class WindowAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    window: int
    scale: float
    rot: Rotation
    sink: bool = True
    v_mix: bool = False             # values mixed with those of the first layer that mixes

    @property
    def q_rows(self) -> int:
        return self.heads * self.dim

    @property
    def k_rows(self) -> int:
        return self.kv_heads * self.dim

    @property
    def v_rows(self) -> int:
        return self.kv_heads * self.vdim


@dataclass(frozen=True)
class LatentAttention:
    """Keys and values of all heads from one cached latent vector and one rotated key part per token."""
    heads: int
    dim: int                        # unrotated query / key elements of a head
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot: Rotation                   # of the rotated part, rot.dims elements, after the unrotated ones in a head's query
    sink: bool = True               # a learned logit per head in the softmax denominator
    kv_from: int | None = None      # the layer whose latents and key parts this one reads

    @property
    def q_rows(self) -> int:
        return self.heads * (self.dim + self.rot.dims)

    @property
    def kv_rows(self) -> int:
        return self.kv_rank + self.rot.dims if self.kv_from is None else 0

    @property
    def cache_row(self) -> int:
        return pad(self.kv_rank, 8) + pad(self.rot.dims, 8)


@dataclass(frozen=True)
class GatedRecurrence:
    width: int


@dataclass(frozen=True)
class FeedForward:
    ff: int
    unary: int = L.UNARY_RELU_SQUARE


@dataclass(frozen=True)
class MixtureOfExperts:
    """`top` of `experts` gated feed-forwards per token: g' sigmoid(alpha g') (u' + beta) with g' = min(g, limit), u' = clamp(u, +-limit),
    weighted by the softmax over the chosen router logits."""
    experts: int
    top: int
    ff: int
    limit: float
    alpha: float
    beta: float


@dataclass(frozen=True)
class Layer:
    mixer: WindowAttention | LatentAttention | GatedRecurrence
    mlp: FeedForward | MixtureOfExperts | None


@dataclass(frozen=True)
class Bigram:
    buckets: int
    mul_prev: int
    mul_cur: int


@dataclass(frozen=True)
class LayerListConfig:
    width: int
    vocab: int
    layers: tuple
    norm_groups: int
    norm_eps: float
    bigram: Bigram | None = None
    norm_center: bool = False       # layer norm instead of RMS norm
    parallel: bool = False          # x <- x + residual_mult * (mixer(h) + mlp(h)), h = N(x): one norm, none behind
    residual_mult: float = 1.0      # of what joins the residual
    embed_scale: float = 1.0
    tied_head: bool = False         # logits from the embedding table (unscaled)

    def __post_init__(self):
        def need(ok, what):
            if not ok:
                raise ValueError(what)

        need(self.width > 0 and self.vocab > 0 and self.layers, "width, vocab and the list of layers must not be empty")
        need(self.norm_groups > 0 and self.width % self.norm_groups == 0, "norm groups must divide the width")
        need(self.bigram is None or self.bigram.buckets > 0, "the bigram table needs buckets")
        mixed = set()
        for i, l in enumerate(self.layers):
            m = l.mixer
            if isinstance(m, WindowAttention):
                need(m.heads > 0 and m.kv_heads > 0 and m.heads % m.kv_heads == 0, f"layer {i}: heads must be a multiple of kv_heads")
                need(0 < m.dim <= 256 and 0 < m.vdim <= 256, f"layer {i}: head sizes up to 256")
                need(m.window >= 1, f"layer {i}: an empty window")
                need(m.rot.dims % 2 == 0 and 0 <= m.rot.dims <= m.dim, f"layer {i}: rotated elements must be even and fit the head")
                if m.v_mix:
                    mixed.add((m.kv_heads, m.vdim))
            elif isinstance(m, LatentAttention):
                need(min(m.heads, m.dim, m.vdim, m.q_rank) > 0 and 0 < m.kv_rank <= 1024, f"layer {i}: empty latent attention, or a latent above 1024")
                need(m.rot.dims % 2 == 0 and 0 <= m.rot.dims <= 1024 and m.rot.pairing == L.ROT_NEIGHBOURS,
                     f"layer {i}: rotated elements must be even, at most 1024, neighbours paired")
                if m.kv_from is not None:
                    need(0 <= m.kv_from < i, f"layer {i}: kv_from must name an earlier layer")
                    o = self.layers[m.kv_from].mixer
                    need(isinstance(o, LatentAttention) and o.kv_from is None and (o.kv_rank, o.rot) == (m.kv_rank, m.rot),
                         f"layer {i}: the layer of kv_from must have latents of its own, of the same rank and rotation")
            else:
                need(m.width > 0, f"layer {i}: empty recurrence")
            need(l.mlp is None or l.mlp.ff > 0, f"layer {i}: empty feed-forward")
            if isinstance(l.mlp, MixtureOfExperts):
                need(1 <= l.mlp.top <= min(l.mlp.experts, 64) and l.mlp.experts <= 1024, f"layer {i}: up to 64 of up to 1024 experts per token")
            need(not self.parallel or (isinstance(m, LatentAttention) and not isinstance(l.mlp, FeedForward)),
                 f"layer {i}: a parallel layer has a latent attention and a mixture of experts (or no feed-forward)")
        need(len(mixed) <= 1, "layers that mix values must have the same value heads")

    @property
    def first_mixing(self) -> int:
        """The layer whose values the later ones mix in, or -1."""
        return next((i for i, l in enumerate(self.layers) if isinstance(l.mixer, WindowAttention) and l.mixer.v_mix), -1)


def rotation_tables(rot: Rotation, n: int):
    """cos / sin [n, dims / 2] of position * base^(-2 i / dims), each rounded once to fp32."""
    i = np.arange(rot.dims // 2, dtype=np.float64)
    ang = np.arange(n, dtype=np.float64)[:, None] * np.power(float(rot.base), -2.0 * i / max(rot.dims, 1))[None, :]
    return np.cos(ang).astype(np.float32), np.sin(ang).astype(np.float32)


# ---- weights ---------------------------------------------------------------------------------------------------------
# What a model's loader hands over (CPU or device tensors; matrices [out, in], any float type that bf16 holds exactly):
#   {"embed", "bigram", "head", "final_norm", "layers": [{"norm1", "norm1b", "norm2", "norm2b", "mix": {...}, "mlp": {...}}]}
#   (no "head" when it is tied; parallel layers have "norm1" only)
#   mix of a recurrence: "z" "x" "g" "o" and biases "z.b" "x.b" ...;  of a window attention: "q" "k" "v" "o", biases, "vmix" (float);
#   of a latent attention: "dq" "dq.norm" "uq" "uk" "uv" "o", "sink" (if it has one), "dkv" "dkv.norm" (without kv_from)
#   mlp: "up", "down" and biases; of a mixture: "gate", "up" [experts, ff, width], "down" [experts, width, ff], "router", "router.b".
#   Missing biases are zero.
class Linear:
    """Stacked bf16 matrices with rows padded to 16 bytes, and their fp32 biases."""

    def __init__(self, mats, biases, device):
        self.K = mats[0].shape[1]
        self.N = sum(m.shape[0] for m in mats)
        self.ldw = pad(self.K, 8)
        self.w = torch.zeros((self.N, self.ldw), dtype=torch.bfloat16, device=device)
        at = 0
        for m in mats:
            if m.shape[1] != self.K:
                raise ValueError(f"stacked matrices read {self.K} and {m.shape[1]} inputs")
            self.w[at: at + m.shape[0], : self.K] = m.to(device)
            at += m.shape[0]
        self.bias = None
        if any(b is not None for b in biases):
            self.bias = torch.zeros(self.N, dtype=torch.float32, device=device)
            at = 0
            for m, b in zip(mats, biases):
                if b is not None:
                    self.bias[at: at + m.shape[0]] = b.to(device=device, dtype=torch.float32)
                at += m.shape[0]

    def rows(self, first: int, n: int) -> "Linear":
        """The matrix of rows first .. first + n - 1, over the same memory."""
        part = Linear.__new__(Linear)
        part.K, part.N, part.ldw, part.w = self.K, n, self.ldw, self.w[first: first + n]
        part.bias = self.bias[first: first + n] if self.bias is not None else None
        return part

    @property
    def nbytes(self) -> int:
        return self.w.numel() * 2


@dataclass(frozen=True)
class Addend:
    """A sublayer's output on its way into the residual: a row y, a post-norm's weight, gathered rows (matrix, numbers, weights)."""
    y: torch.Tensor | None = None
    post: torch.Tensor | None = None
    parts: tuple | None = None


LOG2_E = 1.4426950408889634

# Portions of at least this many tokens expand the cached latents into every head's keys and values; fewer stay in latent space.
EXPAND_TOKENS = 32


class Sequence:
    """One sequence's place: caches, recurrence states, position, and its recorded step."""

    def __init__(self):
        self.pos = 0            # host copy of the position
        self.open = False
        self.greedy_ready = False
        self.step = None        # RecordedStep of one token
        self.warm = False


class LayerListDecoder:
    """Device state of one model.  dtype "bfloat16": GEMM operands, activations between kernels and caches in bf16 with fp32
    accumulation; "float32": true 32-bit arithmetic everywhere (the weights are bf16 values).

    max_seq: longest sequence; max_portion: most tokens of a prompt that run as one batch (longer portions are cut); slots:
    sequences that may be open at the same time."""

    def __init__(self, cfg: LayerListConfig, weights: dict, device: torch.device | str = "cuda", dtype: str = "bfloat16",
                 max_seq: int = 4096, max_portion: int = 2048, slots: int = 1):
        if not torch.cuda.is_available():
            raise RuntimeError("LayerListDecoder needs a CUDA device: there is no CPU path")
        if dtype not in ("bfloat16", "float32"):
            raise ValueError("dtype must be bfloat16 or float32")
        L.lib()
        self.cfg, self.dev = cfg, torch.device(device)
        self.half = dtype == "bfloat16"
        self.act_t = torch.bfloat16 if self.half else torch.float32
        self.max_seq = max(1, int(max_seq))
        self.max_portion = max(1, min(int(max_portion), self.max_seq))
        self.ldx = pad(cfg.width, 8)
        self._load(weights)
        self._tables = {}
        for l in cfg.layers:
            if isinstance(l.mixer, (WindowAttention, LatentAttention)) and l.mixer.rot not in self._tables:
                self._tables[l.mixer.rot] = tuple(torch.from_numpy(t).to(self.dev) for t in rotation_tables(l.mixer.rot, self.max_seq))
        self.status = torch.zeros(1, dtype=torch.int32, device=self.dev)
        self._ws = torch.empty(0, dtype=torch.uint8, device=self.dev)
        self._batch = None      # activation buffers of the largest portion so far
        self._grown = {}        # further ones that grow with the context
        self._one = self._decode_buffers()
        self._free = [self._make_sequence() for _ in range(slots)]
        self.launches = 0       # kernels enqueued so far (a replayed step counts its recorded ones)

    # -- weights ------------------------------------------------------------------------------------------------------
    def _load(self, w: dict) -> None:
        cfg, dev = self.cfg, self.dev
        f32 = lambda t: t.to(device=dev, dtype=torch.float32).contiguous()

        def table(t, rows):
            if tuple(t.shape) != (rows, cfg.width):
                raise ValueError(f"embedding table of shape {tuple(t.shape)}, expected {(rows, cfg.width)}")
            return t.to(device=dev, dtype=torch.bfloat16).contiguous()

        def expect(d, n, *shape):
            if tuple(d[n].shape) != shape:
                raise ValueError(f"matrix {n} of shape {tuple(d[n].shape)}, expected {shape}")
            return d[n]

        def linear(d, names, rows, cols, more=()):
            parts = [(expect(d, n, r, cols), d.get(n + ".b")) for n, r in zip(names, rows)] + list(more)
            return Linear([m for m, _ in parts], [b for _, b in parts], dev)

        if cfg.tied_head:
            self.head = linear(w, ["embed"], [cfg.vocab], cfg.width)
            self.embed = self.head.w
        else:
            self.embed = table(w["embed"], cfg.vocab)
            self.head = linear(w, ["head"], [cfg.vocab], cfg.width)
        self.bigram = table(w["bigram"], cfg.bigram.buckets + 1) if cfg.bigram else None
        self.final_norm = f32(w["final_norm"])
        self.layers = []
        for l, lw in zip(cfg.layers, w["layers"], strict=True):
            d = {"norm1": f32(lw["norm1"])}
            m, mix, ff = l.mixer, lw["mix"], lw.get("mlp")
            router = [(expect(ff, "router", l.mlp.experts, cfg.width), ff.get("router.b"))] if isinstance(l.mlp, MixtureOfExperts) else []
            if not cfg.parallel:
                d["norm1b"] = f32(lw["norm1b"])
            if isinstance(m, WindowAttention):
                d["in"] = linear(mix, ["q", "k", "v"], [m.q_rows, m.k_rows, m.v_rows], cfg.width)
                d["out"] = linear(mix, ["o"], [cfg.width], m.heads * m.vdim)
                d["vmix"] = float(mix["vmix"]) if m.v_mix and "vmix" in mix else 0.0
            elif isinstance(m, LatentAttention):
                H = m.heads
                own = m.kv_from is None
                # (parallel: the router reads the same normed row)
                d["in"] = linear(mix, ["dq"] + ["dkv"] * own, [m.q_rank] + [m.kv_rows] * own, cfg.width, router if cfg.parallel else ())
                d["router_at"] = m.q_rank + m.kv_rows
                d["cq_norm"], d["c_norm"] = f32(expect(mix, "dq.norm", m.q_rank)), f32(expect(mix, "dkv.norm", m.kv_rank)) if own else None
                d["sink"] = f32(expect(mix, "sink", H)) if m.sink else None
                d["uq"] = linear(mix, ["uq"], [m.q_rows], m.q_rank)
                d["expand"] = linear(mix, ["uk", "uv"], [H * m.dim, H * m.vdim], m.kv_rank)
                d["uv"] = d["expand"].rows(H * m.dim, H * m.vdim)
                # a query's way into latent space: per head the transpose of its key matrix
                d["absorb"] = Linear([mix["uk"].reshape(H, m.dim, m.kv_rank).transpose(1, 2).reshape(H * m.kv_rank, m.dim)], [None], dev)
                d["out"] = linear(mix, ["o"], [cfg.width], H * m.vdim)
            else:
                d["in"] = linear(mix, ["z", "x", "g"], [m.width] * 3, cfg.width)
                d["out"] = linear(mix, ["o"], [cfg.width], m.width)
            if l.mlp is not None and not cfg.parallel:
                d["norm2"], d["norm2b"] = f32(lw["norm2"]), f32(lw["norm2b"])
            if isinstance(l.mlp, MixtureOfExperts):
                E, n = l.mlp.experts, l.mlp.ff
                if not cfg.parallel:
                    d["router"] = linear(ff, ["router"], [E], cfg.width)
                    d["router_at"] = 0
                pairs = torch.stack([expect(ff, "gate", E, n, cfg.width), expect(ff, "up", E, n, cfg.width)], dim=2)
                d["gate_up"] = Linear([pairs.reshape(E * 2 * n, cfg.width)], [None], dev)  # rows 2 j and 2 j + 1: gate and up of element j
                d["e_down"] = Linear([expect(ff, "down", E, cfg.width, n).reshape(E * cfg.width, n)], [None], dev)
            elif l.mlp is not None:
                d["up"] = linear(ff, ["up"], [l.mlp.ff], cfg.width)
                d["down"] = linear(ff, ["down"], [cfg.width], l.mlp.ff)
            self.layers.append(d)

    def weight_bytes_per_token(self) -> int:
        """Bytes of matrices one decoded token streams."""
        total = self.head.nbytes
        for l, d in zip(self.cfg.layers, self.layers):
            total += sum(d[k].nbytes for k in ("in", "uq", "absorb", "uv", "out", "router", "up", "down") if k in d)
            if isinstance(l.mlp, MixtureOfExperts):
                total += (d["gate_up"].nbytes + d["e_down"].nbytes) * l.mlp.top // l.mlp.experts
        return total

    # -- sequence places ----------------------------------------------------------------------------------------------
    def _make_sequence(self) -> Sequence:
        cfg, s = self.cfg, Sequence()
        s.state = torch.zeros(4, dtype=torch.int32, device=self.dev)  # cutb_sequence_state
        s.kv, s.gru = {}, {}
        for i, l in enumerate(cfg.layers):
            m = l.mixer
            if isinstance(m, WindowAttention):
                rows = min(pad(min(m.window, self.max_seq) + self.max_portion - 1, 64), pad(self.max_seq, 64))
                s.kv[i] = tuple(torch.zeros((rows, m.kv_heads * pad(n, 8)), dtype=self.act_t, device=self.dev) for n in (m.dim, m.vdim))
            elif isinstance(m, LatentAttention):
                if m.kv_from is None:
                    s.kv[i] = (torch.zeros((pad(self.max_seq, 64), m.cache_row), dtype=self.act_t, device=self.dev),)
            else:
                s.gru[i] = torch.zeros(m.width, dtype=torch.float32, device=self.dev)
        return s

    def open(self) -> Sequence:
        if not self._free:
            raise RuntimeError("no free sequence place: close one first, or construct the decoder with more slots")
        s = self._free.pop()
        # Only what a new sequence would read: the position masks whatever the caches still hold.
        s.state.copy_(torch.tensor([0, -1, 0, 0], dtype=torch.int32))  # -1: no previous token
        for t in s.gru.values():
            t.zero_()
        s.pos, s.open, s.greedy_ready = 0, True, False
        return s

    def close(self, s: Sequence) -> None:
        if not s.open:
            raise RuntimeError("this sequence is not open")
        s.open = False
        self._free.append(s)

    def cache_bytes(self) -> int:
        """Bytes of caches and states one sequence place holds."""
        s = self._free[0] if self._free else self._make_sequence()
        return sum(t.numel() * t.element_size() for kv in s.kv.values() for t in kv) + sum(t.numel() * 4 for t in s.gru.values())

    # -- launches -----------------------------------------------------------------------------------------------------
    @staticmethod
    def _stream() -> int:
        return torch.cuda.current_stream().cuda_stream

    def _call(self, name: str, d) -> None:
        self.launches += 1
        L.check(getattr(L.lib(), name)(C.byref(d), self._stream()))

    def _dense_desc(self, lin: Linear, M: int, a, c, unary: int = 0):
        return ops.dense_desc(a, lin.w, lin.K, c, bias=lin.bias, unary=unary, status=self.status, M=M)

    def _dense(self, lin: Linear, M: int, a, c, unary: int = 0, matvec: bool = False) -> None:
        """c[:M] = unary(a[:M] W^T + bias) on the batch kernels (a single row on the mat-vec if `matvec`)."""
        d = self._dense_desc(lin, M, a, c, unary)
        if not (matvec and M == 1):
            d.variant = L.DENSE_TC if self.half else L.DENSE_SIMT
        need = int(L.lib().cutb_dense_workspace_bytes(C.byref(d)))
        if need:
            if self._ws.numel() < need:
                self._ws = torch.empty(need, dtype=torch.uint8, device=self.dev)
            d.workspace, d.workspace_bytes = self._ws.data_ptr(), self._ws.numel()
            self.launches += 1
        self._call("cutb_dense_matmul", d)

    def _embed_desc(self, n: int, tokens_ptr: int, prev_ptr: int, out):
        cfg, d = self.cfg, L.EmbedDesc()
        d.tokens, d.prev, d.embed, d.ld_embed = tokens_ptr, prev_ptr, self.embed.data_ptr(), self.embed.stride(0)
        if self.bigram is not None:
            d.bigram, d.ld_bigram = self.bigram.data_ptr(), self.bigram.stride(0)
            d.buckets, d.mul_prev, d.mul_cur = cfg.bigram.buckets, cfg.bigram.mul_prev, cfg.bigram.mul_cur
        d.out, d.ldo, d.n, d.dim, d.vocab, d.status = out.data_ptr(), out.stride(0), n, cfg.width, cfg.vocab, self.status.data_ptr()
        d.scale = cfg.embed_scale
        return d

    def _norm(self, rows: int, x, add: "Addend", pre, h, keep: bool, row_index=None) -> None:
        cfg = self.cfg
        self.launches += 1
        ops.residual_norm(x[:rows] if row_index is None else x, pre, cfg.norm_groups, cfg.norm_eps, dim=cfg.width, y=add.y, post_w=add.post,
                          x_out=x if keep else None, out=h, row_index=row_index, center=cfg.norm_center, y_scale=cfg.residual_mult, parts=add.parts)

    def _attn_desc(self, i: int, seq: Sequence, n: int, qkv, out, v_first):
        m, (kc, vc) = self.cfg.layers[i].mixer, seq.kv[i]
        cos_t, sin_t = self._tables[m.rot]
        mix = {}
        if m.v_mix and i == self.cfg.first_mixing:
            mix = {"v_first_out": v_first}
        elif m.v_mix:
            mix = {"v_first": v_first, "v_mix": self.layers[i]["vmix"]}
        return ops.window_desc(qkv[:n], m.heads, m.kv_heads, m.dim, m.vdim, kc, vc, window=m.window, scale=m.scale, out=out, cos_t=cos_t,
                               sin_t=sin_t, rot_dims=m.rot.dims, pairing=m.rot.pairing, max_pos=self.max_seq, sink=m.sink, pos=seq.pos,
                               pos_ptr=seq.state.data_ptr() + 8, status=self.status, **mix)

    def _latent_desc(self, i: int, seq: Sequence, T: int, **tensors):
        m = self.cfg.layers[i].mixer
        (cache,) = seq.kv[i if m.kv_from is None else m.kv_from]
        cos_t, sin_t = self._tables[m.rot]
        return ops.latent_desc(cache, m.heads, m.dim, m.rot.dims, m.vdim, m.kv_rank, scale=m.scale, eps=self.cfg.norm_eps, max_pos=self.max_seq,
                               n_tokens=T, cos_t=cos_t, sin_t=sin_t, sink=self.layers[i]["sink"], pos=seq.pos, pos_ptr=seq.state.data_ptr() + 8,
                               status=self.status, **tensors)

    # -- a portion of a prompt ----------------------------------------------------------------------------------------
    def _sizes(self) -> dict:
        """Columns of the activation buffers: what any layer needs of each."""
        cfg, n = self.cfg, dict.fromkeys(("pre", "mid", "first", "q", "lat", "lat_split", "cq", "logits", "top", "experts", "act", "workspace"), 0)

        def need(**sizes):
            for k, v in sizes.items():
                n[k] = max(n[k], v)

        for l, d in zip(cfg.layers, self.layers):
            need(pre=d["in"].N, mid=max(d["out"].K, d["up"].N if "up" in d else 0))  # pre-activations of a mixer, fp32; its output
            if isinstance(l.mixer, LatentAttention):
                m = l.mixer
                need(q=m.q_rows, lat=m.heads * m.kv_rank, lat_split=m.heads * pad(m.kv_rank, 8), cq=m.q_rank)
                cos_t, sin_t = self._tables[m.rot]
                need(workspace=ops.latent_workspace_bytes(ops.latent_desc(
                    torch.empty((1, m.cache_row)), m.heads, m.dim, m.rot.dims, m.vdim, m.kv_rank, scale=m.scale, eps=cfg.norm_eps,
                    max_pos=self.max_seq, n_tokens=1, cos_t=cos_t, sin_t=sin_t)))
            if isinstance(l.mlp, MixtureOfExperts):
                need(logits=l.mlp.experts, top=l.mlp.top, experts=l.mlp.experts, act=l.mlp.top * pad(l.mlp.ff, 8))
        if cfg.first_mixing >= 0:
            n["first"] = cfg.layers[cfg.first_mixing].mixer.v_rows
        return {k: v if k in ("top", "experts", "workspace") else pad(v, 8) for k, v in n.items()}

    def _buffers(self, T: int) -> dict:
        if self._batch is None or self._batch["rows"] < T:
            n, rows, f32, i32 = self._sizes(), min(self.max_portion, pad(T, 256)), torch.float32, torch.int32
            e = lambda cols, t, per=1: torch.zeros((rows * per, cols), dtype=t, device=self.dev) if cols and per else None
            self._batch = None
            self._batch = {"rows": rows, "x": e(self.ldx, f32), "y": e(self.ldx, f32), "h": e(self.ldx, self.act_t), "pre": e(n["pre"], f32),
                           "mid": e(n["mid"], self.act_t), "first": e(n["first"], f32), "q": e(n["q"], f32), "cq": e(n["cq"], self.act_t),
                           "logits": e(n["logits"], f32)}
            if n["top"]:  # rows sorted by expert: inputs, inner activations, outputs
                ff = max(pad(l.mlp.ff, 8) for l in self.cfg.layers if isinstance(l.mlp, MixtureOfExperts))
                self._batch.update({"sorted": e(self.ldx, self.act_t, n["top"]), "act": e(ff, self.act_t, n["top"]), "moe": e(self.ldx, self.act_t, n["top"]),
                                    "offsets": torch.zeros(n["experts"] + 1, dtype=i32, device=self.dev)})
                for k, t in (("slots", i32), ("ids", i32), ("weights", f32)):
                    self._batch[k] = torch.zeros(rows * n["top"], dtype=t, device=self.dev)
        return self._batch

    def _scratch(self, name: str, rows: int, cols: int, dtype) -> torch.Tensor:
        """A buffer [rows, cols] that grows on demand and lives until a larger one is asked for."""
        t = self._grown.get(name)
        if t is None or t.numel() < rows * cols or t.dtype != dtype:
            self._grown[name] = None
            t = self._grown[name] = torch.zeros(pad(rows, 512) * cols, dtype=dtype, device=self.dev)
        return t[: rows * cols].view(rows, cols)

    def _latent_batch(self, i: int, seq: Sequence, T: int, pre, b: dict) -> None:
        """Latent attention of T tokens, from the pre-activations of the stacked input projection to `mid`."""
        m, d = self.cfg.layers[i].mixer, self.layers[i]
        q, cq, mid = b["q"][:T], b["cq"][:T], b["mid"]
        own = {"lat": pre[:T, m.q_rank:], "lat_norm_w": d["c_norm"]} if m.kv_from is None else {}
        self._call("cutb_latent_kv_write", self._latent_desc(i, seq, T, cq=pre[:T], cq_norm_w=d["cq_norm"], cq_out=cq, **own))
        self._dense(d["uq"], T, cq, q)
        n = seq.pos + T
        if self.half and T >= EXPAND_TOKENS:
            (cache,) = seq.kv[i if m.kv_from is None else m.kv_from]
            exp = self._scratch("expand", n, pad(d["expand"].N, 8), torch.bfloat16)
            a = self._latent_desc(i, seq, T, q=q, k_exp=exp, v_exp=exp[:, m.heads * m.dim:], out=mid)
            if L.lib().cutb_latent_prefill_supported(C.byref(a)):
                self._dense(d["expand"], n, cache[:n], exp)
                self._call("cutb_latent_prefill", a)
                return
        qa, lat = self._scratch("qa", T, m.heads * m.kv_rank, torch.float32), self._scratch("lat", T, m.heads * m.kv_rank, torch.float32)
        self._dense_heads(d["absorb"], T, q, qa, m.heads, m.dim + m.rot.dims, m.kv_rank)
        if T == 1:
            self._call("cutb_latent_attention", self._latent_desc(i, seq, 1, q=q, qa=qa, workspace=self._one["workspace"]))
            self._call("cutb_latent_values", self._latent_desc(i, seq, 1, out=mid, workspace=self._one["workspace"], w_uv=d["uv"].w))
            return
        self._call("cutb_latent_attention", self._latent_desc(i, seq, T, q=q, qa=qa, out=lat))
        self._dense_heads(d["uv"], T, lat, mid, m.heads, m.kv_rank, m.vdim)

    def _dense_heads(self, lin: Linear, T: int, a, c, heads: int, a_step: int, c_step: int) -> None:
        d = ops.batch_desc(a[:T], lin.w, lin.K, c, heads, a_step, c_step, status=self.status)
        self._call("cutb_dense_matmul", d)

    def _experts_batch(self, l: Layer, d: dict, T: int, h, logits, b: dict):
        """The mixture for T tokens; returns what the next norm gathers: (rows sorted by expert, their numbers, their weights)."""
        f, K = l.mlp, self.cfg.width
        slots, ids, weights = (b[k][: T * f.top].view(T, f.top) for k in ("slots", "ids", "weights"))
        rows, variant = T * f.top, L.DENSE_TC if self.half else L.DENSE_SIMT
        group = dict(offsets=b["offsets"], experts=f.experts, tokens=T, top=f.top, variant=variant, status=self.status)
        self._call("cutb_moe_route", ops.moe_route_desc(logits[:T], f.experts, f.top, weights, ids, slots, b["offsets"]))
        self.launches += 1  # (the choice and the sort)
        self._call("cutb_moe_scatter", ops.moe_scatter_desc(h[:T], K, slots, f.experts, b["sorted"][:rows]))
        self._call("cutb_moe_matmul", ops.moe_matmul_desc(b["sorted"], d["gate_up"].w, K, out=b["act"], glu=L.GLU_CLAMPED, alpha=f.alpha,
                                                          beta=f.beta, limit=f.limit, **group))
        self._call("cutb_moe_matmul", ops.moe_matmul_desc(b["act"], d["e_down"].w, f.ff, out=b["moe"], **group))
        return b["moe"], slots, weights

    def _portion(self, seq: Sequence, tokens: torch.Tensor, want, trace=None):
        """Runs tokens (device, int32) as one batch; returns the logits of the places in `want`, or None."""
        cfg, T = self.cfg, tokens.numel()
        b = self._buffers(T)
        x, y, h, pre, mid, first = b["x"], b["y"], b["h"], b["pre"], b["mid"], b["first"]
        self._call("cutb_embedding_bigram", self._embed_desc(T, tokens.data_ptr(), seq.state.data_ptr() + 4, x))
        add = Addend()  # the previous sublayer's output, not yet added to x
        for i, (l, d) in enumerate(zip(cfg.layers, self.layers)):
            m = l.mixer
            self._norm(T, x, add, d["norm1"], h, True)
            if trace is not None and i:
                trace.append(x[:T, : cfg.width].clone())
            rows = pre[:, : pad(d["in"].N, 8)]
            self._dense(d["in"], T, h, rows)
            if isinstance(m, WindowAttention):
                a = self._attn_desc(i, seq, T, rows, mid, first)
                self._call("cutb_window_kv_write", a)
                self._call("cutb_window_attention", a)
            elif isinstance(m, LatentAttention):
                self._latent_batch(i, seq, T, rows, b)
            else:
                self.launches += 1
                ops.mingru_scan(rows[:T], m.width, seq.gru[i], mid)
            self._dense(d["out"], T, mid, y)
            if cfg.parallel:
                add = Addend(y, None, self._experts_batch(l, d, T, h, rows[:, d["router_at"]:], b) if l.mlp is not None else None)
                continue
            add = Addend(y, d["norm1b"])
            if l.mlp is not None:
                self._norm(T, x, add, d["norm2"], h, True)
                if isinstance(l.mlp, MixtureOfExperts):
                    self._dense(d["router"], T, h, b["logits"])
                    add = Addend(None, d["norm2b"], self._experts_batch(l, d, T, h, b["logits"], b))
                else:
                    self._dense(d["up"], T, h, mid, l.mlp.unary)
                    self._dense(d["down"], T, mid, y)
                    add = Addend(y, d["norm2b"])
        logits = None
        if want or trace is not None:
            rows = list(want) if trace is None else list(range(T))
            idx = torch.tensor(rows, dtype=torch.int32).to(self.dev)
            hs = torch.zeros((len(rows), self.ldx), dtype=self.act_t, device=self.dev)
            if trace is not None:
                self._norm(T, x, add, self.final_norm, h, True)
                trace.append(x[:T, : cfg.width].clone())
                hs = h[:T].clone()
            else:
                self._norm(len(rows), x, add, self.final_norm, hs, False, idx)
            full = torch.empty((len(rows), pad(cfg.vocab, 8)), dtype=torch.float32, device=self.dev)
            self._dense(self.head, len(rows), hs, full, matvec=True)
            logits = full[:, : cfg.vocab] if trace is None else full[list(want), : cfg.vocab]
        nxt = None
        if want and want[-1] == T - 1:
            nxt = self._one["next"]
            self.launches += 1
            L.check(L.lib().cutb_argreduce(1, logits[-1].data_ptr(), nxt.data_ptr(), cfg.vocab, self._stream()))
        self.launches += 1
        L.check(L.lib().cutb_sequence_advance(seq.state.data_ptr(), tokens.data_ptr(), T, nxt.data_ptr() if nxt is not None else None,
                                              self._stream()))
        seq.pos += T
        seq.greedy_ready = nxt is not None
        return logits

    # -- one token ----------------------------------------------------------------------------------------------------
    def _decode_buffers(self) -> dict:
        n = self._sizes()
        e = lambda cols: torch.zeros((1, cols), dtype=torch.float32, device=self.dev) if cols else None
        return {"x": [e(self.ldx), e(self.ldx)], "y": e(self.ldx), "h": e(self.ldx), "pre": e(n["pre"]), "mid": e(n["mid"]), "first": e(n["first"]),
                "q": e(n["q"]), "lat": e(n["lat"]), "lat_split": torch.zeros(2 * n["lat_split"], dtype=torch.bfloat16, device=self.dev), "router": e(n["logits"]), "act": e(n["act"]),
                "ids": torch.zeros(max(1, n["top"]), dtype=torch.int32, device=self.dev),
                "workspace": torch.zeros(max(4, n["workspace"] // 4), dtype=torch.float32, device=self.dev),
                "logits": e(pad(self.cfg.vocab, 8)), "next": torch.zeros(1, dtype=torch.float32, device=self.dev)}

    def _plan_step(self, seq: Sequence) -> RecordedStep:
        """The launches of one token, as closures over prepared descriptors."""
        cfg, b, lib, seqd = self.cfg, self._one, L.lib(), []
        keep = []

        def call(name, d):
            keep.append(d)
            fn, ref = getattr(lib, name), C.byref(d)
            seqd.append(lambda: L.check(fn(ref, self._stream())))

        cur = 0

        def staged(lin, add, pre, c, unary=0, h=None):
            """The projection behind a sublayer border: residual add and norms while its input is staged; h: where the normed row goes too."""
            nonlocal cur
            d = self._dense_desc(lin, 1, None, c, unary)
            norm = dict(center=cfg.norm_center, y_scale=cfg.residual_mult, norm_out=h)
            if add.y is None:
                return ops.stage_input(d, b["x"][cur], pre, cfg.norm_groups, cfg.norm_eps, **norm)
            cur ^= 1
            return ops.stage_input(d, b["x"][cur ^ 1], pre, cfg.norm_groups, cfg.norm_eps, add.y, add.post, b["x"][cur], **norm)

        def dense(lin, a, c, unary=0):
            call("cutb_dense_matmul", self._dense_desc(lin, 1, a, c, unary))

        def experts(f, d, name, logits=None, **companion):
            """One of a mixture's two mat-vecs, perhaps with a dense matrix beside it."""
            up = name == "cutb_expert_up"
            more = dict(logits=logits, x=b["h"], alpha=f.alpha, beta=f.beta, limit=f.limit) if up else {}
            call(name, ops.expert_desc(f.experts, f.top, cfg.width, f.ff, d["gate_up" if up else "e_down"].w, b["ids"], b["act"], **more, **companion))

        def latent(i, d, m, f, pre):
            """From the input projection's pre-activations to `y`; a mixture f that reads the same input shares two of the launches."""
            if f is not None:
                experts(f, d, "cutb_expert_up", pre[:, d["router_at"]:], dense=d["uq"].w, dense_K=m.q_rank, xd=pre, xd_norm_w=d["cq_norm"],
                        eps=cfg.norm_eps, out=b["q"])
            else:
                call("cutb_dense_matmul", ops.stage_input(self._dense_desc(d["uq"], 1, None, b["q"]), pre, d["cq_norm"], 1, cfg.norm_eps))
            own = {"lat": pre[:, m.q_rank:], "lat_norm_w": d["c_norm"]} if m.kv_from is None else {}
            attention = self._latent_desc(i, seq, 1, q=b["q"], qa=b["lat"], workspace=b["workspace"], **own)
            if m.heads > 1 and ops.latent_takes_split_queries(attention):  # the absorbed queries as the tensor cores read them
                row = pad(m.kv_rank, 8)
                high, low = b["lat_split"][: 2 * m.heads * row].view(2, m.heads, row)
                attention = self._latent_desc(i, seq, 1, q=b["q"], qa_split=(high, low), workspace=b["workspace"], **own)
                call("cutb_dense_matmul", ops.batch_desc(b["q"], d["absorb"].w, m.dim, high, m.heads, m.dim + m.rot.dims, row, status=self.status,
                                                         low=low, scale=m.scale * LOG2_E))
            else:
                call("cutb_dense_matmul", ops.batch_desc(b["q"], d["absorb"].w, m.dim, b["lat"], m.heads, m.dim + m.rot.dims, m.kv_rank, status=self.status))
            call("cutb_latent_attention", attention)
            call("cutb_latent_values", self._latent_desc(i, seq, 1, out=b["mid"], workspace=b["workspace"], w_uv=d["uv"].w))
            if f is not None:
                experts(f, d, "cutb_expert_down", dense=d["out"].w, dense_K=d["out"].K, xd=b["mid"], out=b["y"])
            else:
                dense(d["out"], b["mid"], b["y"])

        call("cutb_embedding_bigram", self._embed_desc(1, seq.state.data_ptr(), seq.state.data_ptr() + 4, b["x"][0]))
        add = Addend()
        for i, (l, d) in enumerate(zip(cfg.layers, self.layers)):
            m = l.mixer
            if isinstance(m, LatentAttention):
                beside = l.mlp if cfg.parallel else None
                call("cutb_dense_matmul", staged(d["in"], add, d["norm1"], b["pre"], h=b["h"] if beside is not None else None))
                latent(i, d, m, beside, b["pre"])
            elif isinstance(m, WindowAttention):
                call("cutb_dense_matmul", staged(d["in"], add, d["norm1"], b["pre"]))
                call("cutb_window_attention_decode", self._attn_desc(i, seq, 1, b["pre"], b["mid"], b["first"]))
                dense(d["out"], b["mid"], b["y"])
            else:
                q = staged(d["in"], add, d["norm1"], b["mid"])
                q.gru_state = seq.gru[i].data_ptr()
                call("cutb_dense_matmul", q)
                dense(d["out"], b["mid"], b["y"])
            if cfg.parallel:
                add = Addend(b["y"])
                continue
            add = Addend(b["y"], d["norm1b"])
            if l.mlp is not None:
                if isinstance(l.mlp, MixtureOfExperts):
                    call("cutb_dense_matmul", staged(d["router"], add, d["norm2"], b["router"], h=b["h"]))
                    experts(l.mlp, d, "cutb_expert_up", b["router"])
                    experts(l.mlp, d, "cutb_expert_down", out=b["y"])
                else:
                    call("cutb_dense_matmul", staged(d["up"], add, d["norm2"], b["mid"], l.mlp.unary))
                    dense(d["down"], b["mid"], b["y"])
                add = Addend(b["y"], d["norm2b"])
        call("cutb_dense_matmul", staged(self.head, add, self.final_norm, b["logits"]))
        seqd.append(lambda: L.check(lib.cutb_argreduce(1, b["logits"].data_ptr(), b["next"].data_ptr(), cfg.vocab, self._stream())))
        seqd.append(lambda: L.check(lib.cutb_sequence_advance(seq.state.data_ptr(), None, 1, b["next"].data_ptr(), self._stream())))
        step = RecordedStep(seqd, self.dev)
        step.keep, step.launches = keep, len(seqd)
        return step

    def _one_token(self, seq: Sequence) -> torch.Tensor:
        """Runs the token in seq.state; the first time eagerly, then from the recorded graph."""
        if seq.step is None:
            seq.step = self._plan_step(seq)
        if seq.step.graph is None and seq.warm:
            seq.step.capture()
        if seq.step.graph is not None:
            seq.step.replay(1)
        else:
            seq.step.run()
            seq.warm = True
        self.launches += seq.step.launches
        seq.pos += 1
        seq.greedy_ready = True
        return self._one["logits"][:, : self.cfg.vocab]

    # -- the interface of decoding.py -----------------------------------------------------------------------------------
    def _check(self, seq: Sequence, n: int) -> None:
        if not seq.open:
            raise RuntimeError("this sequence is not open")
        if n < 1 or seq.pos + n > self.max_seq:
            raise ValueError(f"1 .. {self.max_seq - seq.pos} further tokens fit this sequence, got {n}")

    def forward(self, seq: Sequence, tokens, want=(), batched: bool = False, trace=None):
        """The next tokens of a sequence; returns the logits at the places `want` (ascending, among these tokens) as a device
        tensor [len(want), vocab] (a single token's is overwritten by the next step), or None.  One token runs the recorded
        decode step unless `batched`.  `trace` (a list) receives the residual stream after every layer."""
        tokens = np.asarray(list(tokens), dtype=np.int64)
        want = [int(w) for w in want]
        self._check(seq, len(tokens))
        if ((tokens < 0) | (tokens >= self.cfg.vocab)).any():
            raise ValueError("token id past the vocabulary")
        if any(not 0 <= w < len(tokens) for w in want) or sorted(set(want)) != want:
            raise ValueError("wanted places must be ascending and among the tokens")
        if len(tokens) == 1 and not batched and trace is None:
            seq.state[0].fill_(int(tokens[0]))
            logits = self._one_token(seq)
            return logits if want else None
        dev_tokens = torch.from_numpy(tokens.astype(np.int32)).to(self.dev)
        parts = []
        for at in range(0, len(tokens), self.max_portion):
            n = min(self.max_portion, len(tokens) - at)
            part = self._portion(seq, dev_tokens[at: at + n], [w - at for w in want if at <= w < at + n], trace)
            if part is not None:
                parts.append(part)
        if not parts:
            return None
        return parts[0] if len(parts) == 1 else torch.cat(parts)

    def decode_greedy(self, seq: Sequence, n: int) -> list:
        """n tokens: the arg-max of the last wanted logits first, then one recorded step per further token; the picks stay on
        the device until the end."""
        if not seq.greedy_ready:
            raise RuntimeError("ask for the logits of the last token first: the continuation starts from their arg-max")
        if n > 1:
            self._check(seq, n - 1)
        picks = torch.empty(n, dtype=torch.int32, device=self.dev)
        for i in range(n):
            picks[i].copy_(seq.state[0])
            if i + 1 < n:
                self._one_token(seq)
        ids = picks.cpu().tolist()
        self.check_status()
        return ids

    def check_status(self) -> None:
        st = int(self.status.item())
        if st:
            self.status.zero_()
            raise L.CutbError(st, "a kernel reported an error (position past the tables, token past the vocabulary, or an expired "
                                  "bounded wait)")
