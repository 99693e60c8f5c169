"""Measurements of the layer-list models (bench.py --layer-list): every kernel alone against its roofline, beside the like
kernel of another model path at equal shape, and prefill / decode throughput of whole models of equal size: Bigerax beside the
llama path, Lenesun (--layer-list-model lenesun) beside Bigerax.

Device time from CUDA events around replays of a graph of launches that walk through enough distinct operands (>= 400 MB)
that L2 does not serve them.  Roofline time = max(bytes / copy bandwidth, FLOPs / bf16 GEMM rate); bytes count every operand
once.  The llama kernels read Q4_K blocks (0.5625 byte per weight), these bf16 weights (2 bytes), so times are compared as
fractions of their own rooflines."""
from __future__ import annotations

import ctypes as C

import numpy as np
import torch

from . import _lib as L
from . import ops
from .layer_list import (Bigram, FeedForward, GatedRecurrence, LatentAttention, Layer, LayerListConfig, LayerListDecoder, MixtureOfExperts, Rotation,
                         WindowAttention, pad, rotation_tables)


def time_us(launches, reps: int = 5, warm: int = 3) -> float:
    """Best device time per launch over `reps` replays of one graph of all launches."""
    for f in launches:
        f()
    torch.cuda.synchronize()
    g = torch.cuda.CUDAGraph()
    with torch.cuda.graph(g):
        for f in launches:
            f()
    for _ in range(warm):
        g.replay()
    best = float("inf")
    for _ in range(reps):
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        g.replay()
        b.record()
        torch.cuda.synchronize()
        best = min(best, a.elapsed_time(b) * 1e3 / len(launches))
    return best


class Roofline:
    def __init__(self, hbm_gbs: float, tflops: float):
        self.hbm, self.tf = hbm_gbs, tflops

    def entry(self, us: float, nbytes: float, flops: float = 0.0) -> dict:
        ideal = max(nbytes / self.hbm / 1e3, flops / self.tf / 1e6)
        return {"us": round(us, 2), "roofline_us": round(ideal, 2), "fraction": round(ideal / us, 3)}


def _copies(nbytes: int, lo: int = 2, hi: int = 64) -> int:
    return max(lo, min(hi, int(400e6 // max(nbytes, 1)) + 1))


def _bf16(*shape):
    return torch.randn(shape, device="cuda", dtype=torch.float32).mul_(shape[-1] ** -0.5).to(torch.bfloat16)


def matvec_us(N: int, K: int, norm: bool = False, gru: bool = False, unary: int = 0) -> float:
    n = _copies(N * K * 2)
    Ws, out = [_bf16(N, K) for _ in range(n)], torch.zeros((1, pad(N, 8)), device="cuda")
    x, y, w = (torch.randn((1, K), device="cuda") for _ in range(3))
    x2, st, keep = torch.zeros_like(x), torch.zeros(N, device="cuda"), []
    for W in Ws:
        d = ops.dense_desc(None if norm else x, W, K, out, unary=unary)
        if norm:
            ops.stage_input(d, x, w, 1, 1e-6, y, w, x2)
        if gru:
            d.gru_state = st.data_ptr()
        keep.append(d)
    us = time_us([lambda d=d: L.check(L.lib().cutb_dense_matmul(C.byref(d), ops._stream_ptr())) for d in keep * max(1, 32 // n)])
    return us


def gemm_us(M: int, N: int, K: int, unary: int = 0, out_t=torch.float32) -> float:
    n = _copies(N * K * 2 + M * K * 2, hi=16)
    sets = [(_bf16(M, K), _bf16(N, K)) for _ in range(n)]
    out = torch.zeros((M, pad(N, 8)), device="cuda", dtype=out_t)
    ds = [ops.dense_desc(A, W, K, out, unary=unary, variant=L.DENSE_TC) for A, W in sets]
    need = int(L.lib().cutb_dense_workspace_bytes(C.byref(ds[0])))
    ws = torch.empty(max(need, 16), dtype=torch.uint8, device="cuda")
    for d in ds:
        d.workspace, d.workspace_bytes = ws.data_ptr(), need
    return time_us([lambda d=d: L.check(L.lib().cutb_dense_matmul(C.byref(d), ops._stream_ptr())) for d in ds])


def _llama_qmm_us(M: int, N: int, K: int, norm: bool = False, glu: bool = False) -> float:
    """The llama path's projection at this shape: Q4_K blocks, fp32 activations, as LlamaDecoder launches it."""
    from . import synth

    rb = synth.row_bytes(L.Q4_K, K)
    n = _copies(N * rb, hi=32)
    base = torch.from_numpy(synth.make_weights(L.Q4_K, N, K, seed=3)).cuda()
    A = torch.randn((M, K), device="cuda")
    w = torch.ones(K, device="cuda")
    ds, keep = [], []
    for r in range(n):
        W = torch.roll(base, 144 * 7 * r)
        d, out, k = ops.make_desc(A, W, L.Q4_K, N, flags=L.FLAG_ACT_16BIT | (0 if norm else L.FLAG_NO_OVERLAP))
        if norm:
            d.flags |= L.FLAG_A_RMSNORM
            d.a_norm_weight, d.a_norm_eps = w.data_ptr(), 1e-5
        need = ops.workspace_bytes(d)
        if need:
            ws = torch.empty(need, dtype=torch.uint8, device="cuda")
            d.workspace, d.workspace_bytes = ws.data_ptr(), need
            k = k + (ws,)
        ds.append(d)
        keep.append((k, out))
    return time_us([lambda d=d: ops.launch(d) for d in ds * max(1, 32 // n)])


def window_us(T: int, H: int, G: int, dim: int, window: int, decode: bool, pos: int) -> float:
    ring = pad(min(window, pos + T) + T, 64)
    cos_t, sin_t = (torch.from_numpy(t).cuda() for t in rotation_tables(Rotation(10000.0, dim), pos + T))
    per = 2 * ring * G * dim * 2
    n = _copies(per + T * (H + 2 * G) * dim * 4, hi=64)
    launches, keep = [], []
    for _ in range(n):
        qkv = torch.randn((T, (H + 2 * G) * dim), device="cuda")
        kc, vc = (torch.randn((ring, G * dim), device="cuda").to(torch.bfloat16) for _ in range(2))
        out = torch.zeros((T, H * dim), device="cuda", dtype=torch.float32 if decode else torch.bfloat16)
        d = ops.window_desc(qkv, H, G, dim, dim, kc, vc, window=window, scale=dim ** -0.5, out=out, cos_t=cos_t, sin_t=sin_t, rot_dims=dim,
                            max_pos=pos + T, sink=True, pos=pos)
        keep.append((qkv, kc, vc, out, d))
        launches.append((lambda d=d: ops.window_attention_decode(d)) if decode else (lambda d=d: ops.window_attention(d)))
    return time_us(launches)


def kv_write_us(T: int, H: int, G: int, dim: int) -> float:
    cos_t, sin_t = (torch.from_numpy(t).cuda() for t in rotation_tables(Rotation(10000.0, dim), T))
    keep, launches = [], []
    for _ in range(_copies(T * (H + 2 * G) * dim * 4, hi=16)):
        qkv = torch.randn((T, (H + 2 * G) * dim), device="cuda")
        kc, vc = (torch.zeros((pad(T, 64), G * dim), device="cuda", dtype=torch.bfloat16) for _ in range(2))
        d = ops.window_desc(qkv, H, G, dim, dim, kc, vc, window=T, scale=1.0, out=qkv, cos_t=cos_t, sin_t=sin_t, rot_dims=dim, max_pos=T)
        keep.append((qkv, kc, vc, d))
        launches.append(lambda d=d: ops.window_kv_write(d))
    return time_us(launches)


def llama_attention_us(T: int, H: int, G: int, dim: int, decode: bool, pos: int) -> float:
    max_seq = pos + T
    half = dim // 2
    cos_t, sin_t = torch.randn((max_seq, half), device="cuda"), torch.randn((max_seq, half), device="cuda")
    n = _copies(2 * max_seq * G * dim * 2 + T * H * dim * 4, hi=64)
    keep, launches = [], []
    st = torch.zeros(1, dtype=torch.int32, device="cuda")
    for _ in range(n):
        q, k, v = (torch.randn((T, m * dim), device="cuda") for m in (H, G, G))
        kc, vc = (torch.randn((max_seq, G * dim), device="cuda").half() for _ in range(2))
        out = torch.zeros((T, H * dim), device="cuda")
        if decode:
            params = torch.tensor([pos, pos + 1], dtype=torch.int32, device="cuda")
            ws = ops.attention_workspace(H, G, dim, max_seq, "cuda")
            launches.append(lambda a=(q, k, v, params, kc, vc, ws, out): ops.rope_attention_decode(
                a[0], a[1], a[2], a[3], cos_t, sin_t, a[4], a[5], H, G, dim, a[6], out=a[7], status=st))
        else:
            params = torch.arange(pos, pos + T, dtype=torch.int32, device="cuda")
            launches.append(lambda a=(q, params, kc, vc, out): ops.batched_attention(a[0], a[2], a[3], a[1], cos_t, sin_t, H, G, dim, out=a[4]))
        keep.append((q, k, v, kc, vc, out, params))
    return time_us(launches)


def norm_us(T: int, dim: int) -> float:
    keep, launches = [], []
    w = torch.ones(dim, device="cuda")
    for _ in range(_copies(T * dim * 14, hi=64)):
        x, y = torch.randn((T, dim), device="cuda"), torch.randn((T, dim), device="cuda")
        h = torch.zeros((T, dim), device="cuda", dtype=torch.bfloat16)
        keep.append((x, y, h))
        launches.append(lambda x=x, y=y, h=h: ops.residual_norm(x, w, 2, 1e-6, y=y, post_w=w, x_out=x, out=h))
    return time_us(launches)


def llama_norm_us(T: int, dim: int) -> float:
    keep, launches = [], []
    w = torch.ones(dim, device="cuda")
    for _ in range(_copies(T * dim * 8, hi=64)):
        x, y = torch.randn((T, dim), device="cuda"), torch.zeros((T, dim), device="cuda")
        keep.append((x, y))
        launches.append(lambda x=x, y=y: L.check(L.lib().cutb_rmsnorm(L.F32, x.data_ptr(), w.data_ptr(), y.data_ptr(), T, dim, dim, 1e-5,
                                                                      ops._stream_ptr())))
    return time_us(launches)


def scan_us(T: int, width: int) -> float:
    keep, launches = [], []
    for _ in range(_copies(T * width * 14, hi=16)):
        zxg, st = torch.randn((T, 3 * width), device="cuda"), torch.zeros(width, device="cuda")
        out = torch.zeros((T, width), device="cuda", dtype=torch.bfloat16)
        keep.append((zxg, st, out))
        launches.append(lambda a=(zxg, st, out): ops.mingru_scan(a[0], width, a[1], a[2]))
    return time_us(launches)


def embed_us(T: int, dim: int, vocab: int) -> float:
    e, bg = _bf16(vocab, dim), _bf16(vocab + 1, dim)
    keep = [torch.randint(0, vocab, (T,), dtype=torch.int32, device="cuda") for _ in range(8)]
    return time_us([lambda t=t: ops.embedding_bigram(t, e, bigram=bg, mul_prev=31, mul_cur=17) for t in keep])


def kernel_table(roof: Roofline, hidden: int, ff: int, H: int, G: int, dim: int, window: int, context: int, T: int, vocab: int) -> dict:
    """Every kernel of a decode step and of a T-token prefill at one layer size, with the llama path's like kernel."""
    qkv = (H + 2 * G) * dim
    out = {}

    def mv(name, N, K, like_norm, **kw):
        ours = roof.entry(matvec_us(N, K, **kw), N * K * 2 + 4 * (N + K))
        like = roof.entry(_llama_qmm_us(1, N, K, norm=like_norm), N * K * 0.5625 + 4 * (N + K))
        out[f"decode {name} {N}x{K}"] = {"ours": ours, "llama": like}

    mv("qkv mat-vec (norms fused)", qkv, hidden, True, norm=True)
    mv("recurrence mat-vec (norms, state update fused)", 3 * hidden, hidden, True, norm=True, gru=True)
    mv("output mat-vec", hidden, H * dim, False)
    mv("up mat-vec (norms, relu^2 fused)", ff, hidden, True, norm=True, unary=L.UNARY_RELU_SQUARE)
    mv("down mat-vec", hidden, ff, False)
    mv("head mat-vec (norms fused)", vocab, hidden, True, norm=True)
    kvb = min(window, context) * G * dim * 2 * 2
    out[f"decode attention, window {window}, context {context}"] = {
        "ours": roof.entry(window_us(1, H, G, dim, window, True, context), kvb + 4 * (H + 2 * G) * dim + 4 * H * dim),
        "llama": roof.entry(llama_attention_us(1, H, G, dim, True, context - 1), context * G * dim * 4 + 4 * (H + 2 * G) * dim + 4 * H * dim)}

    def gm(name, M, N, K, **kw):
        o = 2 if kw.get("out_t") == torch.bfloat16 else 4
        ours = roof.entry(gemm_us(M, N, K, **kw), N * K * 2 + M * K * 2 + M * N * o, 2.0 * M * N * K)
        like = roof.entry(_llama_qmm_us(M, N, K), N * K * 0.5625 + M * K * 4 + M * N * 4, 2.0 * M * N * K)
        out[f"prefill {name} {M}x{N}x{K}"] = {"ours": ours, "llama": like}

    for M in sorted({32, 128, 512, T}):
        gm("qkv GEMM", M, qkv, hidden)
        gm("output GEMM", M, hidden, H * dim)
        gm("up GEMM (relu^2 fused)", M, ff, hidden, unary=L.UNARY_RELU_SQUARE, out_t=torch.bfloat16)
        gm("down GEMM", M, hidden, ff)
    gm("recurrence GEMM", T, 3 * hidden, hidden)
    seen = sum(min(window, i + 1) for i in range(T))  # score entries the mask leaves, per head
    full = T * (T + 1) / 2
    out[f"prefill attention, window {window}, {T} tokens"] = {
        "ours": roof.entry(window_us(T, H, G, dim, window, False, 0), T * (H * dim * 6 + 2 * G * dim * 2), 4.0 * seen * H * dim),
        "llama": roof.entry(llama_attention_us(T, H, G, dim, False, 0), T * (H * dim * 8 + 2 * G * dim * 2), 4.0 * full * H * dim)}
    out[f"prefill cache write, {T} tokens"] = {"ours": roof.entry(kv_write_us(T, H, G, dim), T * 2 * G * dim * 6)}
    out[f"prefill residual + norms, {T} x {hidden}"] = {"ours": roof.entry(norm_us(T, hidden), T * hidden * 14.0),
                                                        "llama": roof.entry(llama_norm_us(T, hidden), T * hidden * 8.0)}
    out[f"prefill recurrence scan, {T} x {hidden}"] = {"ours": roof.entry(scan_us(T, hidden), T * hidden * 14.0)}
    out[f"prefill embedding + bigram, {T} x {hidden}"] = {"ours": roof.entry(embed_us(T, hidden, vocab), T * hidden * 8.0)}
    return out


def model_config(hidden: int, ff: int, H: int, G: int, dim: int, window: int, n_layers: int, vocab: int) -> LayerListConfig:
    att = WindowAttention(H, G, dim, dim, window, dim ** -0.5, Rotation(10000.0, dim), True, True)
    layers = [Layer(GatedRecurrence(hidden), None) if i % 4 == 0 else Layer(att, FeedForward(ff)) for i in range(n_layers)]
    return LayerListConfig(hidden, vocab, tuple(layers), 2, 1e-6, Bigram(65521, 36313, 27191))


# ---- latent attention and mixtures of experts -----------------------------------------------------------------------------------
def _graph_calls(name: str, ds, min_calls: int = 32):
    return [lambda d=d: L.check(getattr(L.lib(), name)(C.byref(d), ops._stream_ptr())) for d in ds * max(1, min_calls // len(ds))]


def head_matvec_us(H: int, N: int, K: int) -> float:
    Ws, x, out = [_bf16(H * N, K) for _ in range(_copies(H * N * K * 2))], torch.randn((1, H * K), device="cuda"), torch.zeros((1, H * N), device="cuda")
    return time_us(_graph_calls("cutb_dense_matmul", [ops.batch_desc(x, W, K, out, H, K, N) for W in Ws]))


class _LatentShapes:
    """Tensors of one latent-attention layer whose context is `ctx` tokens, the last T of them new."""

    def __init__(self, H, dim, rot, vdim, rank, q_rank, T, ctx):
        self.p, self.T, self.ctx = (H, dim, rot, vdim, rank), T, ctx
        self.tables = tuple(torch.from_numpy(t).cuda() for t in rotation_tables(Rotation(10000.0, rot), ctx))
        f = lambda *s: torch.randn(s, device="cuda")
        self.cache = f(ctx, pad(rank, 8) + pad(rot, 8)).to(torch.bfloat16)
        self.q, self.qa, self.lat, self.cq = f(T, H * (dim + rot)), _bf16(2, H, pad(rank, 8)), f(T, rank + rot), f(T, q_rank)
        self.one, self.sink = torch.ones(max(rank, q_rank), device="cuda"), torch.zeros(H, device="cuda")
        self.cq_out = torch.zeros((T, q_rank), device="cuda", dtype=torch.bfloat16)
        self.out = torch.zeros((T, H * vdim), device="cuda", dtype=torch.bfloat16)

    def desc(self, T=None, pos=None, **more):
        H, dim, rot, vdim, rank = self.p
        T = self.T if T is None else T
        return ops.latent_desc(self.cache, H, dim, rot, vdim, rank, scale=(dim + rot) ** -0.5, eps=1e-6, max_pos=self.ctx, n_tokens=T, cos_t=self.tables[0],
                               sin_t=self.tables[1], sink=self.sink, pos=self.ctx - T if pos is None else pos, **more)


def latent_decode_us(H, dim, rot, vdim, rank, ctx):
    """(attention over the cached latents, the values' mat-vec behind it) of one token, each launch timed alone."""
    n = _copies(ctx * (rank + rot) * 2)
    sets = [_LatentShapes(H, dim, rot, vdim, rank, 64, 1, ctx) for _ in range(n)]
    ws = torch.zeros(ops.latent_workspace_bytes(sets[0].desc()) // 4, device="cuda")
    att = [s.desc(q=s.q, qa_split=(s.qa[0], s.qa[1]), workspace=ws, lat=s.lat, lat_norm_w=s.one) for s in sets]
    a = time_us(_graph_calls("cutb_latent_attention", att))
    Ws, out = [_bf16(H * vdim, rank) for _ in range(_copies(H * vdim * rank * 2))], torch.zeros((1, H * vdim), device="cuda")
    v = time_us(_graph_calls("cutb_latent_values", [sets[0].desc(out=out, workspace=ws, w_uv=W) for W in Ws]))
    return a, v


def latent_prefill_us(H, dim, rot, vdim, rank, T) -> float:
    n, keep, ds = _copies(T * H * (dim + vdim) * 2 + T * H * (dim + rot) * 4, hi=16), [], []
    for _ in range(n):
        s, exp = _LatentShapes(H, dim, rot, vdim, rank, 64, T, T), _bf16(T, H * (dim + vdim))
        keep.append((s, exp))
        ds.append(s.desc(q=s.q, k_exp=exp, v_exp=exp[:, H * dim:], out=s.out))
    return time_us(_graph_calls("cutb_latent_prefill", ds, 1))


def latent_write_us(H, dim, rot, vdim, rank, q_rank, T) -> float:
    keep = [_LatentShapes(H, dim, rot, vdim, rank, q_rank, T, T) for _ in range(_copies(T * (rank + rot + q_rank) * 6, hi=32))]
    return time_us(_graph_calls("cutb_latent_kv_write", [s.desc(lat=s.lat, lat_norm_w=s.one, cq=s.cq, cq_norm_w=s.one[:q_rank], cq_out=s.cq_out) for s in keep], 1))


class _Experts:
    def __init__(self, width, ff, E, top, T, sets):
        self.p = (width, ff, E, top)
        self.gu, self.dn = [_bf16(E * 2 * ff, width) for _ in range(sets)], [_bf16(E * width, ff) for _ in range(sets)]
        z = torch.randn((T, E), device="cuda")
        i32 = lambda *s: torch.zeros(s, dtype=torch.int32, device="cuda")
        self.z, self.weights, self.ids, self.slots, self.offsets = z, torch.zeros((T, top), device="cuda"), i32(T, top), i32(T, top), i32(E + 1)
        self.route = ops.moe_route_desc(z, E, top, self.weights, self.ids, self.slots, self.offsets)
        ops.launch_layer_op("cutb_moe_route", self.route)
        torch.cuda.synchronize()


def expert_prefill_us(width, ff, E, top, T) -> dict:
    n = _copies(E * 3 * ff * width * 2 + T * top * (width + ff) * 4, hi=8)
    e, rows = _Experts(width, ff, E, top, T, n), T * top
    bf = lambda r, c: torch.zeros((r, c), device="cuda", dtype=torch.bfloat16)
    x, srt, act, out = [_bf16(T, width) for _ in range(4)], [_bf16(rows, width) for _ in range(n)], [_bf16(rows, ff) for _ in range(n)], bf(rows, width)
    group = dict(offsets=e.offsets, experts=E, tokens=T, top=top, variant=L.DENSE_TC)
    aout = bf(rows, ff)
    up = [ops.moe_matmul_desc(a, W, width, out=aout, glu=L.GLU_CLAMPED, alpha=1.702, beta=1.0, limit=7.0, **group) for a, W in zip(srt, e.gu)]
    down = [ops.moe_matmul_desc(a, W, ff, out=out, **group) for a, W in zip(act, e.dn)]
    scatter = [ops.moe_scatter_desc(a, width, e.slots, E, b) for a, b in zip(x, srt)]
    return {"route": time_us(_graph_calls("cutb_moe_route", [e.route], 16)), "scatter": time_us(_graph_calls("cutb_moe_scatter", scatter, 8)),
            "up": time_us(_graph_calls("cutb_moe_matmul", up, 1)), "down": time_us(_graph_calls("cutb_moe_matmul", down, 1))}


def expert_decode_us(width, ff, E, top, Nd, Kd, Ko):
    """(up with the query projection beside it, down with the output projection beside it) of one token."""
    active = top * 3 * ff * width * 2
    n = _copies(active // 2, hi=16)
    e = _Experts(width, ff, E, top, 1, n)
    wd, wo = [_bf16(Nd, Kd) for _ in range(n)], [_bf16(width, Ko) for _ in range(n)]
    f = lambda c: torch.randn(c, device="cuda")
    x, xd, one, xo, act, q, y = f(width), f(Kd), torch.ones(Kd, device="cuda"), f(Ko), f(top * ff), f(Nd), f(width)
    ids = torch.zeros(top, dtype=torch.int32, device="cuda")
    up = [ops.expert_desc(E, top, width, ff, W, ids, act, logits=e.z, x=x, alpha=1.702, beta=1.0, limit=7.0, dense=D, dense_K=Kd, xd=xd, xd_norm_w=one,
                          eps=1e-6, out=q) for W, D in zip(e.gu, wd)]
    down = [ops.expert_desc(E, top, width, ff, W, ids, act, dense=D, dense_K=Ko, xd=xo, out=y) for W, D in zip(e.dn, wo)]
    return time_us(_graph_calls("cutb_expert_up", up)), time_us(_graph_calls("cutb_expert_down", down))


def parallel_norm_us(T: int, dim: int, top: int) -> float:
    keep, launches, w = [], [], torch.ones(dim, device="cuda")
    for _ in range(_copies(T * dim * (14 + 2 * top), hi=32)):
        x, y, m = torch.randn((T, dim), device="cuda"), torch.randn((T, dim), device="cuda"), _bf16(T * top, dim)
        h, rows = torch.zeros((T, dim), device="cuda", dtype=torch.bfloat16), torch.randperm(T * top, device="cuda").to(torch.int32).view(T, top)
        pw = torch.rand((T, top), device="cuda")
        keep.append((x, y, m, h, rows, pw))
        launches.append(lambda a=keep[-1]: ops.residual_norm(a[0], w, 1, 1e-6, y=a[1], x_out=a[0], out=a[3], center=True, y_scale=0.4, parts=(a[2], a[4], a[5])))
    return time_us(launches)


def latent_table(roof: Roofline, hidden, H, dim, rot, vdim, q_rank, rank, E, top, ff, context, T, vocab, kv_heads) -> dict:
    """Every kernel of a Lenesun decode step and of a T-token prefill at one layer size, with Bigerax's like kernel."""
    out, mv_bytes = {}, lambda N, K: N * K * 2 + 4 * (N + K)
    n_in, n_uq, wide = q_rank + rank + rot + E, H * (dim + rot), dim + rot

    def put(name, us, nbytes, flops=0.0, like=None):
        out[name] = {"ours": roof.entry(us, nbytes, flops), **({"bigerax": roof.entry(*like)} if like else {})}

    dense_like = lambda N, K, **kw: (matvec_us(N, K, **kw), mv_bytes(N, K))
    put(f"decode input mat-vec (layer norm fused) {n_in}x{hidden}", matvec_us(n_in, hidden, norm=True), mv_bytes(n_in, hidden), like=dense_like(n_in, hidden, norm=True))
    up, down = expert_decode_us(hidden, ff, E, top, n_uq, q_rank, H * vdim)
    ub = mv_bytes(n_uq, q_rank) + mv_bytes(top * 2 * ff, hidden)
    db = mv_bytes(hidden, H * vdim + top * ff)
    put(f"decode experts up {top}x{2 * ff}x{hidden} + queries {n_uq}x{q_rank}", up, ub, like=dense_like(ub // (2 * hidden), hidden, norm=True))
    put(f"decode experts down {hidden}x{top}x{ff} + output {hidden}x{H * vdim}", down, db, like=dense_like(hidden, H * vdim + top * ff))
    put(f"decode queries into latent space {H}x{rank}x{dim}", head_matvec_us(H, rank, dim), mv_bytes(H * rank, dim), like=dense_like(H * dim, rank))
    for c in (context, 8 * context):
        att, val = latent_decode_us(H, dim, rot, vdim, rank, c)
        put(f"decode latent attention, context {c}", att, c * (rank + rot) * 2 + 4 * H * (rank + wide), 2.0 * H * c * (2 * rank + rot),
            like=(window_us(1, H, kv_heads, dim, c, True, c), c * kv_heads * dim * 4 + 8 * H * dim))
    put(f"decode values out of latent space {H}x{vdim}x{rank}", val, mv_bytes(H * vdim, rank), like=dense_like(H * vdim, rank))
    put(f"decode head mat-vec (layer norm fused) {vocab}x{hidden}", matvec_us(vocab, hidden, norm=True), mv_bytes(vocab, hidden), like=dense_like(vocab, hidden, norm=True))

    gemm_bytes = lambda M, N, K, o: N * K * 2 + M * K * 2 + M * N * o
    for M in sorted({128, 512, T}):
        rows = M * top
        e = expert_prefill_us(hidden, ff, E, top, M)
        used = min(E, rows)
        for k, N, K, o in (("up", 2 * ff, hidden, 1), ("down", hidden, ff, 2)):
            like = (gemm_us(rows, N, K, out_t=torch.bfloat16), gemm_bytes(rows, N, K, 2), 2.0 * rows * N * K)
            put(f"prefill experts {k}, {M} tokens, {E} x {N}x{K}", e[k], used * N * K * 2 + rows * K * 2 + rows * N * o, 2.0 * rows * N * K, like=like)
    e = expert_prefill_us(hidden, ff, E, top, T)
    put(f"prefill routing (choice, sort), {T} tokens", e["route"], T * E * 4 + T * top * 16)
    put(f"prefill expert order (row copies), {T} x {top} x {hidden}", e["scatter"], T * hidden * 2 + T * top * hidden * 2)
    for name, N, K in (("input", n_in, hidden), ("queries", n_uq, q_rank), ("expansion", H * (dim + vdim), rank), ("output", hidden, H * vdim)):
        us = gemm_us(T, N, K)
        put(f"prefill {name} GEMM {T}x{N}x{K}", us, gemm_bytes(T, N, K, 4), 2.0 * T * N * K)
    pairs = T * (T + 1) / 2
    put(f"prefill latent attention (expanded), {T} tokens", latent_prefill_us(H, dim, rot, vdim, rank, T), T * H * (wide * 4 + (dim + vdim) * 2 + vdim * 2) + T * rot * 2,
        2.0 * pairs * H * (wide + vdim), like=(window_us(T, H, kv_heads, dim, T, False, 0), T * (H * dim * 6 + 2 * kv_heads * dim * 2), 4.0 * pairs * H * dim))
    put(f"prefill cache write and query norm, {T} tokens", latent_write_us(H, dim, rot, vdim, rank, q_rank, T), T * (rank + rot + q_rank) * 6,
        like=(kv_write_us(T, H, kv_heads, dim), T * 2 * kv_heads * dim * 6))
    put(f"prefill residual + gathered experts + layer norm, {T} x {hidden}", parallel_norm_us(T, hidden, top), T * hidden * (14.0 + 2 * top),
        like=(norm_us(T, hidden), T * hidden * 14.0))
    put(f"prefill embedding, {T} x {hidden}", embed_us(T, hidden, vocab), T * hidden * 8.0)
    return out


def latent_model_config(hidden, H, dim, rot, vdim, q_rank, rank, E, top, ff, n_layers, vocab) -> LayerListConfig:
    """Every other layer reads the latents of the one before it."""
    att = lambda j: LatentAttention(H, dim, vdim, q_rank, rank, (dim + rot) ** -0.5, Rotation(10000.0, rot), True, j)
    layers = tuple(Layer(att(None if i % 2 == 0 else i - 1), MixtureOfExperts(E, top, ff, 7.0, 1.702, 1.0)) for i in range(n_layers))
    return LayerListConfig(hidden, vocab, layers, 1, 1e-6, norm_center=True, parallel=True, residual_mult=0.4, embed_scale=2.0, tied_head=True)


def latent_random_weights(cfg: LayerListConfig) -> dict:
    layers = []
    for l in cfg.layers:
        m, f, one = l.mixer, l.mlp, lambda n: torch.ones(n, device="cuda")
        mix = {"dq": _bf16(m.q_rank, cfg.width), "dq.norm": one(m.q_rank), "uq": _bf16(m.q_rows, m.q_rank), "uk": _bf16(m.heads * m.dim, m.kv_rank),
               "uv": _bf16(m.heads * m.vdim, m.kv_rank), "o": _bf16(cfg.width, m.heads * m.vdim), "sink": torch.zeros(m.heads, device="cuda")}
        if m.kv_from is None:
            mix.update({"dkv": _bf16(m.kv_rows, cfg.width), "dkv.norm": one(m.kv_rank)})
        layers.append({"norm1": one(cfg.width), "mix": mix, "mlp": {
            "gate": _bf16(f.experts, f.ff, cfg.width), "up": _bf16(f.experts, f.ff, cfg.width), "down": _bf16(f.experts, cfg.width, f.ff),
            "router": _bf16(f.experts, cfg.width), "router.b": torch.zeros(f.experts, device="cuda")}})
    return {"embed": _bf16(cfg.vocab, cfg.width), "final_norm": torch.ones(cfg.width, device="cuda"), "layers": layers}


def decoder_throughput(roof: Roofline, dec: LayerListDecoder, vocab: int, T: int, steps: int, matmul_flops: float) -> dict:
    """Prefill of T tokens (best of 4) and the following `steps` tokens."""
    prompt = np.random.default_rng(1).integers(0, vocab, T)
    ev = lambda: torch.cuda.Event(enable_timing=True)
    best = float("inf")
    for turn in range(4):
        s = dec.open()
        torch.cuda.synchronize()
        a, b = ev(), ev()
        a.record()
        dec.forward(s, prompt, [T - 1])
        b.record()
        torch.cuda.synchronize()
        best = min(best, a.elapsed_time(b))
        if turn < 3:
            dec.close(s)
    dec.decode_greedy(s, 4)
    torch.cuda.synchronize()
    a, b = ev(), ev()
    a.record()
    for _ in range(steps):
        dec._one_token(s)
    b.record()
    torch.cuda.synchronize()
    dec.check_status()
    ms = a.elapsed_time(b) / steps
    return {"prefill_tokens": T, "prefill_ms": round(best, 3), "prefill_tok/s": round(T / best * 1e3),
            "prefill_GEMM_roofline_fraction": round(matmul_flops / roof.tf / 1e9 / best, 3), "decode_ms": round(ms, 4), "decode_tok/s": round(1e3 / ms, 1),
            "weight_GB_per_token": round(dec.weight_bytes_per_token() / 1e9, 3),
            "decode_roofline_fraction": round(dec.weight_bytes_per_token() / roof.hbm / 1e6 / ms, 3), "launches_per_token": s.step.launches}


def latent_throughput(roof: Roofline, hidden, H, dim, rot, vdim, q_rank, rank, E, top, ff, n_layers, vocab, T, kv_heads, steps: int = 128) -> dict:
    cfg = latent_model_config(hidden, H, dim, rot, vdim, q_rank, rank, E, top, ff, n_layers, vocab)
    dec = LayerListDecoder(cfg, latent_random_weights(cfg), max_seq=T + steps + 16)
    per_token = sum(d["in"].K * d["in"].N + d["uq"].K * d["uq"].N + d["expand"].K * d["expand"].N + d["out"].K * d["out"].N + top * 3 * ff * hidden for d in dec.layers)
    res = {"lenesun": decoder_throughput(roof, dec, vocab, T, steps, 2.0 * T * per_token)}
    del dec
    torch.cuda.empty_cache()
    # Bigerax with as many layers, all of them attention with a window over the whole context, and as much feed-forward per token
    ff_like = top * ff * 3 // 2
    att = WindowAttention(H, kv_heads, dim, dim, T + steps + 16, dim ** -0.5, Rotation(10000.0, dim), True, True)
    like = LayerListConfig(hidden, vocab, tuple(Layer(att, FeedForward(ff_like)) for _ in range(n_layers)), 2, 1e-6, Bigram(65521, 36313, 27191))
    dec = LayerListDecoder(like, random_weights(like), max_seq=T + steps + 16)
    per_token = (dec.weight_bytes_per_token() - dec.head.nbytes) / 2
    res["bigerax"] = decoder_throughput(roof, dec, vocab, T, steps, 2.0 * T * per_token)
    del dec
    torch.cuda.empty_cache()
    return res


def random_weights(cfg: LayerListConfig) -> dict:
    lin = lambda d, names, rows, cols, bias: {**{n: _bf16(r, cols) for n, r in zip(names, rows)},
                                              **({n + ".b": torch.zeros(r, device="cuda") for n, r in zip(names, rows)} if bias else {})}
    one = lambda: torch.ones(cfg.width, device="cuda")
    layers = []
    for l in cfg.layers:
        m, d = l.mixer, {"norm1": one(), "norm1b": one()}
        if isinstance(m, WindowAttention):
            d["mix"] = lin(d, ["q", "k", "v"], [m.q_rows, m.k_rows, m.v_rows], cfg.width, True)
            d["mix"].update(lin(d, ["o"], [cfg.width], m.heads * m.vdim, True), vmix=0.3)
        else:
            d["mix"] = {**lin(d, ["z", "x", "g"], [m.width] * 3, cfg.width, False), **lin(d, ["o"], [cfg.width], m.width, False)}
        if l.mlp:
            d["norm2"], d["norm2b"] = one(), one()
            d["mlp"] = {**lin(d, ["up"], [l.mlp.ff], cfg.width, True), **lin(d, ["down"], [cfg.width], l.mlp.ff, True)}
        layers.append(d)
    return {"embed": _bf16(cfg.vocab, cfg.width), "bigram": _bf16(cfg.bigram.buckets + 1, cfg.width), "head": _bf16(cfg.vocab, cfg.width),
            "final_norm": one(), "layers": layers}


def model_throughput(roof: Roofline, hidden: int, ff: int, H: int, G: int, dim: int, window: int, n_layers: int, vocab: int, T: int,
                     steps: int = 128) -> dict:
    cfg = model_config(hidden, ff, H, G, dim, window, n_layers, vocab)
    dec = LayerListDecoder(cfg, random_weights(cfg), max_seq=T + steps + 16)
    prompt = np.random.default_rng(1).integers(0, vocab, T)
    ours = decoder_throughput(roof, dec, vocab, T, steps, 2.0 * T * (dec.weight_bytes_per_token() - dec.head.nbytes) / 2)
    del dec
    torch.cuda.empty_cache()

    from .llama_decode import LlamaConfig, LlamaDecoder, synthetic_weights

    lc = LlamaConfig(n_layers=n_layers, hidden=hidden, n_heads=H, n_kv_heads=G, head_dim=dim, ffn=ff, vocab=vocab, max_seq=T + steps + 16)
    ll = LlamaDecoder(lc, synthetic_weights(lc, seed=41, distinct_layers=False, scale_shift=7))
    ev = lambda: torch.cuda.Event(enable_timing=True)
    best = float("inf")
    for _ in range(4):
        torch.cuda.synchronize()
        a, b = ev(), ev()
        a.record()
        ll.prefill(prompt)
        b.record()
        torch.cuda.synchronize()
        best = min(best, a.elapsed_time(b))
    ll.set_position(1, T)
    ll.step(1, T)
    ll.capture()
    ll.replay(4)
    ll.set_position(1, T)
    torch.cuda.synchronize()
    a, b = ev(), ev()
    a.record()
    ll.replay(steps)
    b.record()
    torch.cuda.synchronize()
    ll.check_status()
    ms = a.elapsed_time(b) / steps
    lin = sum(p * q for p, q in ((lc.q_dim + 2 * lc.kv_dim, hidden), (hidden, lc.q_dim), (2 * ff, hidden), (hidden, ff))) * n_layers
    like = {"prefill_ms": round(best, 3), "prefill_tok/s": round(T / best * 1e3), "prefill_GEMM_roofline_fraction": round(2.0 * T * lin / roof.tf / 1e9 / best, 3),
            "decode_ms": round(ms, 4), "decode_tok/s": round(1e3 / ms, 1), "weight_GB_per_token": round(ll.weight_bytes_per_token() / 1e9, 3),
            "decode_roofline_fraction": round(ll.weight_bytes_per_token() / roof.hbm / 1e6 / ms, 3), "launches_per_token": ll.launches_per_step}
    return {"bigerax": ours, "llama_q4_k": like}


SIZES = {  # hidden, ff, query heads, KV heads, head, window, layers, vocabulary
    "2048": (2048, 8192, 16, 4, 128, 1024, 16, 32000),
    "4096": (4096, 14336, 32, 8, 128, 1024, 16, 32000),
}


LATENT_SIZES = {  # hidden, heads, unrotated, rotated and value parts, query and latent ranks, experts, top, ff, layers, vocabulary, KV heads beside it
    "2048": (2048, 16, 128, 64, 128, 768, 512, 32, 4, 1024, 16, 32000, 4),
    "4096": (4096, 32, 128, 64, 128, 1536, 512, 16, 4, 2048, 8, 32000, 8),
}


def measure(hbm_gbs: float, tflops: float, source: str, tables=("4096",), models=("2048", "4096"), T: int = 2048, design: str = "bigerax") -> dict:
    roof = Roofline(hbm_gbs, tflops)
    res = {"roofline": {"hbm_GB/s": hbm_gbs, "bf16_TFLOP/s": tflops, "source": source},
           "timing": "CUDA-graph chains over >= 400 MB of distinct operands, best of 5", "kernels": {}, "models": {}}
    for s in tables:
        if design == "lenesun":
            hidden, H, dim, rot, vdim, q_rank, rank, E, top, ff, _, vocab, kv = LATENT_SIZES[s]
            res["kernels"][s] = latent_table(roof, hidden, H, dim, rot, vdim, q_rank, rank, E, top, ff, 2048, T, vocab, kv)
        else:
            hidden, ff, H, G, dim, window, _, vocab = SIZES[s]
            res["kernels"][s] = kernel_table(roof, hidden, ff, H, G, dim, window, 2048, T, vocab)
        torch.cuda.empty_cache()
    for s in models:
        res["models"][s] = (latent_throughput(roof, *LATENT_SIZES[s][:-1], T, LATENT_SIZES[s][-1]) if design == "lenesun"
                            else model_throughput(roof, *SIZES[s], T=T))
        torch.cuda.empty_cache()
    return res
