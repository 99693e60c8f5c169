"""Measurements of the layer-list models (bench.py --layer-list): every kernel alone against its roofline, beside the like
kernel of the llama path at equal shape, and prefill / decode throughput of whole models of equal size.

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
from .layer_list import (Bigram, FeedForward, GatedRecurrence, Layer, LayerListConfig, LayerListDecoder, Rotation, WindowAttention, pad,
                         rotation_tables)


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
    ev = lambda: torch.cuda.Event(enable_timing=True)
    best = float("inf")
    for _ in range(4):
        s = dec.open()
        torch.cuda.synchronize()
        a, b = ev(), ev()
        a.record()
        dec.forward(s, prompt, [T - 1])
        b.record()
        torch.cuda.synchronize()
        best = min(best, a.elapsed_time(b))
        if _ < 3:
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
    n_lin = (dec.weight_bytes_per_token() - dec.head.nbytes) / 2
    pre_roof = 2.0 * T * n_lin / roof.tf / 1e9
    ours = {"prefill_tokens": T, "prefill_ms": round(best, 3), "prefill_tok/s": round(T / best * 1e3), "prefill_GEMM_roofline_fraction": round(pre_roof / best, 3),
            "decode_ms": round(ms, 4), "decode_tok/s": round(1e3 / ms, 1), "weight_GB_per_token": round(dec.weight_bytes_per_token() / 1e9, 3),
            "decode_roofline_fraction": round(dec.weight_bytes_per_token() / roof.hbm / 1e6 / ms, 3), "launches_per_token": s.step.launches}
    del dec, s
    torch.cuda.empty_cache()

    from .llama_decode import LlamaConfig, LlamaDecoder, synthetic_weights

    lc = LlamaConfig(n_layers=n_layers, hidden=hidden, n_heads=H, n_kv_heads=G, head_dim=dim, ffn=ff, vocab=vocab, max_seq=T + steps + 16)
    ll = LlamaDecoder(lc, synthetic_weights(lc, seed=41, distinct_layers=False, scale_shift=7))
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


def measure(hbm_gbs: float, tflops: float, source: str, tables=("4096",), models=("2048", "4096"), T: int = 2048) -> dict:
    roof = Roofline(hbm_gbs, tflops)
    res = {"roofline": {"hbm_GB/s": hbm_gbs, "bf16_TFLOP/s": tflops, "source": source},
           "timing": "CUDA-graph chains over >= 400 MB of distinct operands, best of 5", "kernels": {}, "models": {}}
    for s in tables:
        hidden, ff, H, G, dim, window, _, vocab = SIZES[s]
        res["kernels"][s] = kernel_table(roof, hidden, ff, H, G, dim, window, 2048, T, vocab)
        torch.cuda.empty_cache()
    for s in models:
        res["models"][s] = model_throughput(roof, *SIZES[s], T=T)
        torch.cuda.empty_cache()
    return res
