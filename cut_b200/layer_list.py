"""Decoder for models whose configuration lists their layers: each layer has a mixer (windowed attention or a gated
recurrence) and possibly a feed-forward, with norms before and after each of them, over dense bf16 weights.

Prefill runs a portion of a prompt as one batch: tensor-core GEMMs (bf16) or fp32 FMA GEMMs (the 32-bit mode), the scan of
the recurrence, the tiled window attention, and one launch per sublayer border that adds the post-normed output to the
residual and norms it for the next sublayer.  A decode step is recorded into a CUDA graph per sequence place: two launches for
a recurrent layer's mixer (norms and residual fused into the input staging of the projection, the state update and output
gate into its epilogue), three for an attention layer's, two for a feed-forward.  The residual stream, the norms, the
recurrence and its states, the rotation angles, the scores and the softmax are fp32 in both modes; decode mat-vecs use the
fp32 activations as they are.

A sequence place holds, per attention layer, ring caches of keys and values (a position lives in row position % ring_rows;
the ring covers the window and one portion), per recurrent layer its fp32 state, and {token, previous token, position} on the
device, so a recorded step replays for every token.
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
class GatedRecurrence:
    width: int


@dataclass(frozen=True)
class FeedForward:
    ff: int
    unary: int = L.UNARY_RELU_SQUARE


@dataclass(frozen=True)
class Layer:
    mixer: WindowAttention | GatedRecurrence
    mlp: FeedForward | None


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
            else:
                need(m.width > 0, f"layer {i}: empty recurrence")
            need(l.mlp is None or l.mlp.ff > 0, f"layer {i}: empty feed-forward")
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
#   mix of a recurrence: "z" "x" "g" "o" and biases "z.b" "x.b" ...;  of an attention: "q" "k" "v" "o", biases, "vmix" (float)
#   mlp: "up", "down" and biases.  Missing biases are zero.
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

    @property
    def nbytes(self) -> int:
        return self.w.numel() * 2


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
            if isinstance(l.mixer, WindowAttention) and l.mixer.rot not in self._tables:
                self._tables[l.mixer.rot] = tuple(torch.from_numpy(t).to(self.dev) for t in rotation_tables(l.mixer.rot, self.max_seq))
        self.status = torch.zeros(1, dtype=torch.int32, device=self.dev)
        self._ws = torch.empty(0, dtype=torch.uint8, device=self.dev)
        self._batch = None      # activation buffers of the largest portion so far
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

        def linear(d, names, rows, cols):
            for n, r in zip(names, rows):
                if tuple(d[n].shape) != (r, cols):
                    raise ValueError(f"matrix {n} of shape {tuple(d[n].shape)}, expected {(r, cols)}")
            return Linear([d[n] for n in names], [d.get(n + ".b") for n in names], dev)

        self.embed = table(w["embed"], cfg.vocab)
        self.bigram = table(w["bigram"], cfg.bigram.buckets + 1) if cfg.bigram else None
        self.head = linear(w, ["head"], [cfg.vocab], cfg.width)
        self.final_norm = f32(w["final_norm"])
        self.layers = []
        for l, lw in zip(cfg.layers, w["layers"], strict=True):
            d = {"norm1": f32(lw["norm1"]), "norm1b": f32(lw["norm1b"])}
            m, mix = l.mixer, lw["mix"]
            if isinstance(m, WindowAttention):
                d["in"] = linear(mix, ["q", "k", "v"], [m.q_rows, m.k_rows, m.v_rows], cfg.width)
                d["out"] = linear(mix, ["o"], [cfg.width], m.heads * m.vdim)
                d["vmix"] = float(mix["vmix"]) if m.v_mix and "vmix" in mix else 0.0
            else:
                d["in"] = linear(mix, ["z", "x", "g"], [m.width] * 3, cfg.width)
                d["out"] = linear(mix, ["o"], [cfg.width], m.width)
            if l.mlp is not None:
                d["norm2"], d["norm2b"] = f32(lw["norm2"]), f32(lw["norm2b"])
                d["up"] = linear(lw["mlp"], ["up"], [l.mlp.ff], cfg.width)
                d["down"] = linear(lw["mlp"], ["down"], [cfg.width], l.mlp.ff)
            self.layers.append(d)

    def weight_bytes_per_token(self) -> int:
        """Bytes of matrices one decoded token streams."""
        return self.head.nbytes + sum(d[k].nbytes for d in self.layers for k in ("in", "out", "up", "down") if k in d)

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
            else:
                s.gru[i] = torch.zeros(m.width, dtype=torch.float32, device=self.dev)
        return s

    def open(self) -> Sequence:
        if not self._free:
            raise RuntimeError("no free sequence place: close one first, or construct the decoder with more slots")
        s = self._free.pop()
        # Only what a new sequence would read: the position masks whatever the rings still hold.
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
        return d

    def _norm(self, rows: int, x, y, post, pre, h, keep: bool, row_index=None) -> None:
        self.launches += 1
        ops.residual_norm(x[:rows] if row_index is None else x, pre, self.cfg.norm_groups, self.cfg.norm_eps, dim=self.cfg.width, y=y,
                          post_w=post, x_out=x if keep else None, out=h, row_index=row_index)

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

    # -- a portion of a prompt ----------------------------------------------------------------------------------------
    def _sizes(self):
        cfg = self.cfg
        pre = max(d["in"].N for d in self.layers)                                # pre-activations of a mixer, fp32
        mid = max([d["out"].K for d in self.layers] + [d["up"].N for d in self.layers if "up" in d])
        first = cfg.layers[cfg.first_mixing].mixer.v_rows if cfg.first_mixing >= 0 else 0
        return pad(pre, 8), pad(mid, 8), pad(first, 8)

    def _buffers(self, T: int) -> dict:
        if self._batch is None or self._batch["rows"] < T:
            pre, mid, first = self._sizes()
            rows = min(self.max_portion, pad(T, 256))
            e = lambda n, t: torch.zeros((rows, n), dtype=t, device=self.dev)
            self._batch = None
            self._batch = {"rows": rows, "x": e(self.ldx, torch.float32), "y": e(self.ldx, torch.float32), "h": e(self.ldx, self.act_t),
                           "pre": e(pre, torch.float32), "mid": e(mid, self.act_t), "first": e(first, torch.float32) if first else None}
        return self._batch

    def _portion(self, seq: Sequence, tokens: torch.Tensor, want, trace=None):
        """Runs tokens (device, int32) as one batch; returns the logits of the places in `want`, or None."""
        cfg, T = self.cfg, tokens.numel()
        b = self._buffers(T)
        x, y, h, pre, mid, first = b["x"], b["y"], b["h"], b["pre"], b["mid"], b["first"]
        self._call("cutb_embedding_bigram", self._embed_desc(T, tokens.data_ptr(), seq.state.data_ptr() + 4, x))
        out, post = None, None  # the previous sublayer's output and its norm, not yet added to x
        for i, (l, d) in enumerate(zip(cfg.layers, self.layers)):
            m = l.mixer
            self._norm(T, x, out, post, d["norm1"], h, True)
            if trace is not None and i:
                trace.append(x[:T, : cfg.width].clone())
            rows = pre[:, : pad(d["in"].N, 8)]
            self._dense(d["in"], T, h, rows)
            if isinstance(m, WindowAttention):
                a = self._attn_desc(i, seq, T, rows, mid, first)
                self._call("cutb_window_kv_write", a)
                self._call("cutb_window_attention", a)
            else:
                self.launches += 1
                ops.mingru_scan(rows[:T], m.width, seq.gru[i], mid)
            self._dense(d["out"], T, mid, y)
            out, post = y, d["norm1b"]
            if l.mlp is not None:
                self._norm(T, x, out, post, d["norm2"], h, True)
                self._dense(d["up"], T, h, mid, l.mlp.unary)
                self._dense(d["down"], T, mid, y)
                out, post = y, d["norm2b"]
        logits = None
        if want or trace is not None:
            rows = list(want) if trace is None else list(range(T))
            idx = torch.tensor(rows, dtype=torch.int32).to(self.dev)
            hs = torch.zeros((len(rows), self.ldx), dtype=self.act_t, device=self.dev)
            if trace is not None:
                self._norm(T, x, out, post, self.final_norm, h, True)
                trace.append(x[:T, : cfg.width].clone())
                hs = h[:T].clone()
            else:
                self._norm(len(rows), x, out, post, self.final_norm, hs, False, idx)
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
        pre, mid, first = self._sizes()
        e = lambda n: torch.zeros((1, n), dtype=torch.float32, device=self.dev)
        return {"x": [e(self.ldx), e(self.ldx)], "y": e(self.ldx), "pre": e(pre), "mid": e(mid), "first": e(first) if first else None,
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

        def staged(lin, out, post, pre, c, unary=0):
            """The projection behind a sublayer border: residual add and norms while its input is staged."""
            nonlocal cur
            d = self._dense_desc(lin, 1, None, c, unary)
            if out is None:
                return ops.stage_input(d, b["x"][cur], pre, cfg.norm_groups, cfg.norm_eps)
            cur ^= 1
            return ops.stage_input(d, b["x"][cur ^ 1], pre, cfg.norm_groups, cfg.norm_eps, out, post, b["x"][cur])

        call("cutb_embedding_bigram", self._embed_desc(1, seq.state.data_ptr(), seq.state.data_ptr() + 4, b["x"][0]))
        out, post = None, None
        for i, (l, d) in enumerate(zip(cfg.layers, self.layers)):
            if isinstance(l.mixer, WindowAttention):
                call("cutb_dense_matmul", staged(d["in"], out, post, d["norm1"], b["pre"]))
                call("cutb_window_attention_decode", self._attn_desc(i, seq, 1, b["pre"], b["mid"], b["first"]))
            else:
                q = staged(d["in"], out, post, d["norm1"], b["mid"])
                q.gru_state = seq.gru[i].data_ptr()
                call("cutb_dense_matmul", q)
            call("cutb_dense_matmul", self._dense_desc(d["out"], 1, b["mid"], b["y"]))
            out, post = b["y"], d["norm1b"]
            if l.mlp is not None:
                call("cutb_dense_matmul", staged(d["up"], out, post, d["norm2"], b["mid"], l.mlp.unary))
                call("cutb_dense_matmul", self._dense_desc(d["down"], 1, b["mid"], b["y"]))
                out, post = b["y"], d["norm2b"]
        call("cutb_dense_matmul", staged(self.head, out, post, self.final_norm, b["logits"]))
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
