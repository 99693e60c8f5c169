"""Layer-list models on the device: every mechanism alone against its oracle, then whole models in both element types --
prompts, token-by-token decoding, portions, places that are used again, sequences that alternate -- and greedy generation
through the queue, the trace replay and the command line.

Limits are relative to the rms of the wanted values: 32-bit mode 3e-5, bf16 mode 3e-2 for whole models (a handful of
layers of bf16 operands)."""
import ctypes as C
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from cut_b200 import _lib as L
from cut_b200 import ops
from cut_b200.decoding import RequestQueue
from cut_b200.layer_list import Rotation, pad, rotation_tables
from cut_b200.models import load_model
from cut_b200.trace import replay
from oracle import hybrid_ref as R
from tests.layer_list_util import CONFIGS, attention, bf16, build_decoder, config, mingru, random_weights, row_errors, save_model, with_mlp

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
LIMIT = {"float32": 3e-5, "bfloat16": 3e-2}


def dev(a, dtype=torch.float32):
    return torch.from_numpy(np.ascontiguousarray(a)).to(device="cuda", dtype=dtype)


def rel(got, want):
    got, want = np.asarray(got.float().cpu() if torch.is_tensor(got) else got, np.float64), np.asarray(want, np.float64)
    return float(np.linalg.norm(got - want) / np.linalg.norm(want))


def padded(a, m=8):
    out = np.zeros((a.shape[0], pad(a.shape[1], m)), np.float32)
    out[:, : a.shape[1]] = a
    return out


def cuts_of(T, sizes):
    cuts = [0]
    while cuts[-1] < T:
        cuts.append(min(T, cuts[-1] + sizes[(len(cuts) - 1) % len(sizes)]))
    return cuts


# ---- dense products --------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("M,K,N", [(2, 72, 40), (7, 333, 130), (64, 64, 64), (129, 200, 257), (300, 1024, 384), (33, 4096, 320), (1, 96, 48),
                                   (513, 96, 1000)])
@pytest.mark.parametrize("unary", [0, L.UNARY_RELU_SQUARE, 133])
def test_dense_gemm(M, K, N, unary):
    rng = np.random.default_rng(M + K)
    A, W, b = bf16(rng.standard_normal((M, K))), bf16(rng.standard_normal((N, K)) / np.sqrt(K)), rng.standard_normal(N).astype(np.float32)
    y = A.astype(np.float64) @ W.T.astype(np.float64) + b
    want = {0: y, L.UNARY_RELU_SQUARE: np.maximum(y, 0) ** 2, 133: y * R.sigmoid(y)}[unary]
    w, bias, status = dev(padded(W), torch.bfloat16), dev(b), torch.zeros(1, dtype=torch.int32, device="cuda")
    for a_t, variant in ((torch.bfloat16, L.DENSE_TC), (torch.float32, L.DENSE_SIMT), (torch.bfloat16, L.DENSE_SIMT)):
        a = dev(padded(A), a_t)
        for c_t, lim in ((torch.float32, 2e-6), (torch.bfloat16, 4e-3)):
            out = torch.full((M, pad(N, 8)), 7.0, device="cuda", dtype=c_t)
            ops.dense_matmul(ops.dense_desc(a, w, K, out, bias=bias, unary=unary, variant=variant, status=status, N=N))
            assert rel(out[:, :N], want) < lim, (a_t, variant, c_t)
            assert bool((out[:, N:] == 7.0).all())  # nothing is written past the row
    assert int(status.item()) == 0


def test_dense_gemm_with_odd_row_strides_and_split_k_without_workspace():
    rng = np.random.default_rng(8)
    M, K, N = 20, 4096, 130
    A, W = bf16(rng.standard_normal((M, K))), bf16(rng.standard_normal((N, K)) / 64)
    a, w = dev(A, torch.bfloat16), dev(W, torch.bfloat16)
    d = ops.dense_desc(a, w, K, torch.empty((M, 136), device="cuda"), variant=L.DENSE_TC, N=N)
    assert int(L.lib().cutb_dense_workspace_bytes(C.byref(d))) > 0  # K is shared out over the SMs
    for ld in (130, 131, 136):
        outs = []
        for split in (True, False):
            out = torch.zeros((M, ld), device="cuda")
            d = ops.dense_desc(a, w, K, out, variant=L.DENSE_TC, N=N)
            if split:
                ops.dense_matmul(d)
            else:  # the plain launch runs the shape in one pass
                L.check(L.lib().cutb_dense_matmul(C.byref(d), ops._stream_ptr()))
            assert rel(out[:, :N], A.astype(np.float64) @ W.T.astype(np.float64)) < 1e-5
            outs.append(out)
        assert rel(outs[0][:, :N], outs[1][:, :N].cpu().numpy()) < 1e-5


@pytest.mark.parametrize("K,N", [(64, 48), (96, 203), (333, 130), (1000, 7), (4096, 4500), (2048, 9000), (14336, 512), (40, 1)])
def test_dense_matvec(K, N):
    rng = np.random.default_rng(K)
    x, W, b = rng.standard_normal(K).astype(np.float32), bf16(rng.standard_normal((N, K)) / np.sqrt(K)), rng.standard_normal(N).astype(np.float32)
    want = np.maximum(W.astype(np.float64) @ x + b, 0) ** 2
    out = torch.full((1, pad(N, 8)), 7.0, device="cuda")
    w, bias = dev(padded(W), torch.bfloat16), dev(b)
    for flags in (0, L.FLAG_NO_OVERLAP):
        d = ops.dense_desc(dev(x).view(1, -1), w, K, out, bias=bias, unary=L.UNARY_RELU_SQUARE, N=N)
        d.flags = flags
        ops.dense_matmul(d)
        assert rel(out[0, :N], want) < 2e-6 and bool((out[0, N:] == 7.0).all())
    xb = dev(bf16(x), torch.bfloat16).view(1, -1)
    o16 = torch.zeros((1, pad(N, 8)), device="cuda", dtype=torch.bfloat16)
    ops.dense_matmul(ops.dense_desc(xb, w, K, o16, bias=bias, N=N))
    assert rel(o16[0, :N], W.astype(np.float64) @ bf16(x).astype(np.float64) + b) < 4e-3


NORM_SHAPES = [(128, 1), (256, 2), (96, 3), (70, 7), (35, 5), (4096, 2), (4096, 32), (8192, 4), (1000, 125), (5000, 1)]


@pytest.mark.parametrize("dim,groups", NORM_SHAPES)
@pytest.mark.parametrize("with_y", [True, False])
def test_residual_norm_and_the_matvec_that_stages_it(dim, groups, with_y):
    rng = np.random.default_rng(dim)
    rows, eps = 5, 1e-3
    # parts of very different size: a norm over the whole row, or over wrong parts, shows
    size = np.repeat(10.0 ** rng.uniform(-2, 2, groups), dim // groups)
    x, y = rng.standard_normal((rows, dim)) * size, rng.standard_normal((rows, dim)) * size[::-1]
    wp, wn = 1 + 0.3 * rng.standard_normal(dim), 1 + 0.3 * rng.standard_normal(dim)
    nx = x + R.grouped_norm(y, wp, groups, eps) if with_y else x
    want = R.grouped_norm(nx, wn, groups, eps)
    ld = pad(dim, 8)
    tx, ty, twp, twn = dev(padded(x)), dev(padded(y)), dev(wp), dev(wn)
    kw = dict(dim=dim, y=ty if with_y else None, post_w=twp)
    for dt, lim in ((torch.float32, 2e-6), (torch.bfloat16, 4e-3)):
        h = torch.zeros((rows, ld), device="cuda", dtype=dt)
        keep = tx.clone()
        ops.residual_norm(keep, twn, groups, eps, x_out=keep, out=h, **kw)  # in place
        assert rel(h[:, :dim], want) < lim and rel(keep[:, :dim], nx) < 1e-6
    idx = torch.tensor([4, 0, 4], dtype=torch.int32, device="cuda")
    h = ops.residual_norm(tx, twn, groups, eps, row_index=idx, **kw)
    assert rel(h[:, :dim], want[[4, 0, 4]]) < 2e-6 and rel(tx[:, :dim], x) < 1e-7
    N = 24
    W = bf16(rng.standard_normal((N, dim)) / np.sqrt(dim))
    out, xo = torch.zeros((1, N), device="cuda"), torch.zeros(ld, device="cuda")
    d = ops.dense_desc(None, dev(padded(W), torch.bfloat16), dim, out, N=N)
    ops.stage_input(d, tx[3], twn, groups, eps, ty[3] if with_y else None, twp if with_y else None, xo if with_y else None)
    ops.dense_matmul(d)
    assert rel(out[0], W.astype(np.float64) @ want[3]) < 5e-6
    if with_y:
        assert rel(xo[:dim], nx[3]) < 1e-6


def test_embedding_with_bigrams():
    rng = np.random.default_rng(1)
    V, B = 61, 37
    for dim in (40, 30):
        e, b = bf16(rng.standard_normal((V, dim))), bf16(rng.standard_normal((B + 1, dim)))
        toks = rng.integers(0, V, 50)
        te, tb, tt = dev(e, torch.bfloat16), dev(b, torch.bfloat16), torch.tensor(toks, dtype=torch.int32, device="cuda")
        for prev in (None, 17):
            p = torch.tensor([-1 if prev is None else prev], dtype=torch.int32, device="cuda")
            got = ops.embedding_bigram(tt, te, prev=p, bigram=tb, mul_prev=4294967291, mul_cur=3999999979)
            rows = R.bigram_rows(toks, prev, 4294967291, 3999999979, B)
            assert np.array_equal(got.cpu().numpy(), e[toks] + b[rows])
        assert np.array_equal(ops.embedding_bigram(tt, te).cpu().numpy(), e[toks])
        status = torch.zeros(1, dtype=torch.int32, device="cuda")
        bad = torch.tensor([3, V, 5], dtype=torch.int32, device="cuda")
        got = ops.embedding_bigram(bad, te, bigram=tb, mul_prev=3, mul_cur=5, status=status)
        assert int(status.item()) == L.ERR_INVALID and not got[1:].any() and got[0].any()


@pytest.mark.parametrize("width", [16, 33, 200])
def test_recurrence_scan_and_step(width):
    rng = np.random.default_rng(width)
    T = 700
    pre = rng.standard_normal((T, 3 * width)) * 2
    pre[:, :width] -= 2.0  # slow gates: states remember hundreds of tokens
    s0 = rng.standard_normal(width)
    states = R.mingru_scan(R.sigmoid(pre[:, :width]), pre[:, width:2 * width], s0)
    g = pre[:, 2 * width:]
    want = states * g * R.sigmoid(g)
    t = dev(padded(pre))
    for cuts in ([0, T], [0, 1, 3, 128, 129, 300, 556, T]):
        st, out = dev(s0), torch.zeros((T, pad(width, 8)), device="cuda")
        for a, b in zip(cuts, cuts[1:]):
            ops.mingru_scan(t[a:b], width, st, out[a:b])
        assert rel(out[:, :width], want) < 3e-6 and rel(st, states[-1]) < 3e-6
    o16 = torch.zeros((T, width), device="cuda", dtype=torch.bfloat16)
    ops.mingru_scan(t, width, dev(s0), o16)
    assert rel(o16, want) < 4e-3
    # one token through the mat-vec's epilogue: an input row that picks row 0 of the pre-activations out of the weight
    W, st, out = np.zeros((3 * width, 8), np.float32), dev(s0), torch.zeros((1, pad(width, 8)), device="cuda")
    W[:, 0], bias = bf16(pre[0]), pre[0] - bf16(pre[0])
    x = dev(np.eye(1, 8))
    d = ops.dense_desc(x, dev(W, torch.bfloat16), 8, out, bias=dev(bias), N=3 * width)
    d.gru_state = st.data_ptr()
    ops.dense_matmul(d)
    assert rel(out[0, :width], want[0]) < 3e-6 and rel(st, states[0]) < 3e-6


# ---- windowed attention ------------------------------------------------------------------------------------------------
class Attn:
    """Random q / k / v rows of one layer, its oracle, and the device side over a ring."""

    def __init__(self, H, G, dim, vdim, window, T, dtype, *, dims=None, sink=True, pairing=L.ROT_NEIGHBOURS, mix=0.0, ring=None, seed=0, base=1000.0):
        self.p = (H, G, dim, vdim)
        self.window, self.T, self.dtype, self.sink, self.pairing, self.mix = window, T, dtype, sink, pairing, mix
        self.dims = dim if dims is None else dims
        rng = np.random.default_rng(seed)
        self.qkv = bf16(rng.standard_normal((T, H * dim + G * (dim + vdim))))
        self.first = rng.standard_normal((T, G * vdim)).astype(np.float32)
        self.scale = 1.3 * dim ** -0.5
        self.rot = Rotation(base, self.dims, pairing)
        self.ring = pad(window + T, 64) if ring is None else ring
        self.cos, self.sin = (torch.from_numpy(t).cuda() for t in rotation_tables(self.rot, T))
        self.kc = torch.zeros((self.ring, G * pad(dim, 8)), device="cuda", dtype=dtype)
        self.vc = torch.zeros((self.ring, G * pad(vdim, 8)), device="cuda", dtype=dtype)
        self.status = torch.zeros(1, dtype=torch.int32, device="cuda")

    def parts(self):
        H, G, dim, vdim = self.p
        q, k, v = np.split(self.qkv.astype(np.float64), [H * dim, (H + G) * dim], axis=1)
        return q.reshape(self.T, H, dim), k.reshape(self.T, G, dim), v.reshape(self.T, G, vdim)

    def want(self, window=None, sink=None):
        q, k, v = self.parts()
        pos = np.arange(self.T)

        def turn(x):
            if self.pairing == L.ROT_NEIGHBOURS:
                return R.rotate_pairs(x, pos, self.rot.base, self.dims)
            y, half = x.copy(), self.dims // 2  # half-split: reorder, rotate neighbours, reorder back
            order = np.arange(self.dims).reshape(2, half).T.reshape(-1)
            y[:, :, : self.dims] = x[:, :, order]
            y = R.rotate_pairs(y, pos, self.rot.base, self.dims)
            z = x.copy()
            z[:, :, order] = y[:, :, : self.dims]
            return z

        v = R.mix_values(v, self.first.reshape(v.shape), self.mix) if self.mix else v
        q, k, w = turn(q), turn(k), self.window if window is None else window
        sink = self.sink if sink is None else sink
        if sink:
            return R.window_attention(q, k, v, 0, w, self.scale)
        # no sink: the same weights without the extra one
        ones = R.window_attention(q, k, np.ones(v.shape[:2] + (1,)), 0, w, self.scale)
        out = R.window_attention(q, k, v, 0, w, self.scale).reshape(self.T, q.shape[1], -1)
        return (out / ones.reshape(self.T, -1, 1)).reshape(self.T, -1)

    def desc(self, a, b, out, pos_ptr=None):
        H, G, dim, vdim = self.p
        self.rows = dev(self.qkv[a:b])
        self.vf = dev(self.first[a:b])
        mix = {"v_first": self.vf, "v_mix": self.mix} if self.mix else {}
        return ops.window_desc(self.rows, H, G, dim, vdim, self.kc, self.vc, window=self.window, scale=self.scale, out=out[a:b], cos_t=self.cos,
                               sin_t=self.sin, rot_dims=self.dims, pairing=self.pairing, max_pos=self.T, sink=self.sink, pos=a,
                               pos_ptr=pos_ptr, status=self.status, **mix)

    def run(self, cuts, decode_from=None):
        H, G, dim, vdim = self.p
        out = torch.zeros((self.T, H * vdim), device="cuda")
        for a, b in zip(cuts, cuts[1:]):
            d = self.desc(a, b, out)
            ops.window_kv_write(d)
            ops.window_attention(d)
        for a in range(decode_from if decode_from is not None else self.T, self.T):
            ops.window_attention_decode(self.desc(a, a + 1, out))
        torch.cuda.synchronize()
        assert int(self.status.item()) == 0
        return out.cpu().numpy().astype(np.float64)


ATTN = [(4, 2, 32, 24, 33, 150), (1, 1, 10, 7, 1, 40), (6, 2, 64, 64, 64, 200), (8, 1, 128, 128, 100, 260), (3, 3, 48, 96, 65, 130),
        (2, 1, 130, 200, 50, 90), (16, 1, 24, 72, 700, 300), (5, 1, 100, 20, 200, 330),
        (56, 4, 16, 8, 20, 40), (100, 2, 24, 24, 30, 50)]  # (many heads: two and four per block in decoding)


@pytest.mark.parametrize("H,G,dim,vdim,window,T", ATTN)
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_window_attention_prefill_portions_and_decode(H, G, dim, vdim, window, T, dtype):
    lim = 5e-6 if dtype == torch.float32 else 8e-3
    for sink, mix, dims, pairing in ((True, 0.4, dim // 4 * 2, L.ROT_NEIGHBOURS), (False, 0.0, dim // 2 * 2, L.ROT_HALVES)):
        a = Attn(H, G, dim, vdim, window, T, dtype, sink=sink, mix=mix, dims=dims, pairing=pairing, seed=T)
        want = a.want()
        whole = a.run([0, T])
        assert rel(whole, want) < lim
        # a ring that is as small as it may be: it wraps again and again, a new key takes the row of one outside the window
        small = Attn(H, G, dim, vdim, window, T, dtype, sink=sink, mix=mix, dims=dims, pairing=pairing, seed=T, ring=pad(window + 39, 64))
        cuts = cuts_of(T, [2, 40, 1, 3, 17, 40, 2])
        assert rel(small.run(cuts), want) < lim
        tail = Attn(H, G, dim, vdim, window, T, dtype, sink=sink, mix=mix, dims=dims, pairing=pairing, seed=T, ring=pad(window + 39, 64))
        cuts = [c for c in cuts if c < T // 3] + [T // 3]
        assert rel(tail.run(cuts, decode_from=T // 3), want) < lim


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("window", [1, 2, 17, 63, 64, 65, 128, 200])
def test_one_key_that_stands_out_is_seen_exactly_inside_the_window(window, dtype):
    """Keys whose score is far above all others, at positions around tile borders: a query one token further than the window
    must not see them, one at its edge must; the same in prompts and in decoding, and with the window one off in the oracle."""
    T, H, G, dim = 330, 2, 1, 32
    def make():
        a = Attn(H, G, dim, 32, window, T, dtype, dims=0, seed=window)
        q, k = slice(0, H * dim), slice(H * dim, (H + G) * dim)
        a.qkv[:, q] = bf16(0.05 * a.qkv[:, q])
        a.qkv[:, 0] = a.qkv[:, dim] = 4.0
        a.qkv[:, k.start] = 0.0
        for p in (0, 1, 62, 63, 64, 100, 128):
            a.qkv[p, k.start] = 16.0
        a.scale = 0.25  # their scores: 16; the others': about 0
        return a
    lim = 5e-6 if dtype == torch.float32 else 8e-3
    a = make()
    want = a.want()
    assert rel(a.want(window=window + 1), want) > 0.05  # the mistake would show
    assert rel(a.run([0, T]), want) < lim
    assert rel(make().run([0, 2, 63, 65, 128, 130, T]), want) < lim
    assert rel(make().run([0, 5], decode_from=5), want) < lim


def test_sink_takes_the_weight_of_keys_that_score_low():
    a = Attn(2, 1, 16, 16, 20, 60, torch.float32, dims=0)
    a.qkv[:, :32], a.qkv[:, 32:48] = 2.0, -1.0  # every score about -8
    want = a.want()
    assert np.abs(want).max() < 0.05 and rel(a.want(sink=False), want) > 10
    assert rel(a.run([0, 60]), want) < 1e-5 and rel(a.run([0, 3], decode_from=3), want) < 1e-5


def test_positions_past_the_tables_are_reported_and_touch_nothing():
    a = Attn(2, 1, 16, 16, 20, 60, torch.bfloat16)
    out = torch.zeros((60, 32), device="cuda")
    d = a.desc(0, 4, out)
    d.max_pos, d.pos = 50, 48
    for f in (ops.window_kv_write, ops.window_attention):
        a.status.zero_()
        f(d)
        torch.cuda.synchronize()
        assert int(a.status.item()) == L.ERR_INVALID
    assert bool(a.kc[48:50].any()) and not a.kc[50:].any() and not out.any()
    d = a.desc(0, 1, out)
    d.max_pos, d.pos = 50, 50
    a.status.zero_()
    ops.window_attention_decode(d)
    torch.cuda.synchronize()
    assert int(a.status.item()) == L.ERR_INVALID and not out.any() and not a.kc[50:].any()


# ---- whole models --------------------------------------------------------------------------------------------------------
_MODELS = {}


def model(name, dtype, **options):
    """(reference logits of a fixed token sequence, tokens, decoder)."""
    if name not in _MODELS:
        cfg = CONFIGS[name]
        w = random_weights(cfg, sum(map(ord, name)))
        toks = np.random.default_rng(9).integers(0, cfg["vocab"], 230)
        trace = []
        _MODELS[name] = (cfg, w, toks, R.HybridReference(cfg, w).run(toks, trace), trace)
    cfg, w, toks, want, trace = _MODELS[name]
    return toks, want, trace, build_decoder(cfg, w, dtype, **{"max_seq": 256, **options})


def feed(dec, toks, cuts, seq=None, batched=False):
    s = dec.open() if seq is None else seq
    rows = []
    for a, b in zip(cuts, cuts[1:]):
        rows.append(dec.forward(s, toks[a:b], list(range(b - a)), batched=batched).cpu().numpy())
    dec.check_status()
    if seq is None:
        dec.close(s)
    return np.concatenate(rows)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_model_whole_portions_and_token_by_token(name, dtype):
    toks, want, trace, dec = model(name, dtype)
    T, lim = len(toks), LIMIT[dtype]
    got = []
    s = dec.open()
    whole = dec.forward(s, toks, list(range(T)), trace=got).cpu().numpy()
    dec.close(s)
    assert len(got) == len(trace)
    for i, (g, t) in enumerate(zip(got, trace)):
        assert rel(g, t) < lim, f"residual after layer {i}"
    assert row_errors(whole, want).max() < lim
    assert row_errors(feed(dec, toks, list(range(T + 1))), want).max() < lim           # the recorded step
    assert row_errors(feed(dec, toks, list(range(21)), batched=True), want[:20]).max() < lim  # single tokens on the batch kernels
    for sizes in ([2], [3, 2, 64, 1, 31], [100, 1, 1], [33]):
        assert row_errors(feed(dec, toks, cuts_of(T, sizes)), want).max() < lim, sizes
    # only some places wanted, none wanted, and the first token alone
    s = dec.open()
    assert dec.forward(s, toks[:1], []) is None
    some = dec.forward(s, toks[1:200], [0, 5, 198]).cpu().numpy()
    assert row_errors(some, want[[1, 6, 199]]).max() < lim
    assert dec.forward(s, toks[200:210], []) is None and dec.forward(s, toks[210:211], []) is None
    assert row_errors(dec.forward(s, toks[211:213], [1]).cpu().numpy(), want[[212]]).max() < lim
    dec.close(s)
    dec.check_status()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_portions_are_cut_and_rings_wrap(dtype):
    toks, want, _, dec = model("gqa", dtype, max_portion=48)  # rings of 128 rows under 230 tokens
    assert all(kc.shape[0] < 200 for kc, _ in dec._free[0].kv.values())
    assert row_errors(feed(dec, toks, [0, len(toks)]), want).max() < LIMIT[dtype]
    assert row_errors(feed(dec, toks, [0, 100] + list(range(101, len(toks) + 1))), want).max() < LIMIT[dtype]
    s = dec.open()
    sparse = dec.forward(s, toks, [3, 47, 48, 229]).cpu().numpy()  # wanted places in several of the inner portions
    assert row_errors(sparse, want[[3, 47, 48, 229]]).max() < LIMIT[dtype]
    dec.close(s)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_places_are_reused_and_sequences_do_not_mix(dtype):
    toks, want, _, dec = model("gqa", dtype, slots=2)
    lim = LIMIT[dtype]
    other = np.random.default_rng(4).integers(0, 203, 120)
    ref = R.HybridReference(_MODELS["gqa"][0], _MODELS["gqa"][1])
    other_want = ref.run(other)
    a, b = dec.open(), dec.open()
    with pytest.raises(RuntimeError, match="no free sequence place"):
        dec.open()
    ga, gb = [], []
    for i in range(0, 120, 10):  # alternate: portions of one, tokens of the other
        ga.append(dec.forward(a, toks[i:i + 10], list(range(10))).cpu().numpy())
        gb += [dec.forward(b, other[j:j + 1], [0]).cpu().numpy() for j in range(i, i + 10)]
    assert row_errors(np.concatenate(ga), want[:120]).max() < lim and row_errors(np.concatenate(gb), other_want).max() < lim
    dec.close(a)
    with pytest.raises(RuntimeError, match="not open"):
        dec.forward(a, [1], [])
    with pytest.raises(RuntimeError, match="not open"):
        dec.close(a)
    c = dec.open()  # the place of `a`, with its old keys and states underneath
    assert c is a
    assert row_errors(feed(dec, other, [0, 1, 3, 60, 120], seq=c), other_want).max() < lim
    assert row_errors(feed(dec, toks[:1], [0, 1], seq=(dec.close(c), dec.open())[1]), want[:1]).max() < lim
    dec.check_status()


def test_same_tokens_give_the_same_bits_whatever_ran_before():
    toks, _, _, dec = model("odd", "bfloat16")
    first = feed(dec, toks, [0, 100, 101, 102, 230])
    feed(dec, toks[::-1], [0, 7, 90])
    assert np.array_equal(first, feed(dec, toks, [0, 100, 101, 102, 230]))


def test_refusals():
    toks, _, _, dec = model("one", "float32", max_seq=20)
    s = dec.open()
    for bad in ([], [64], [-1], list(range(21))):
        with pytest.raises(ValueError):
            dec.forward(s, bad, [])
    with pytest.raises(ValueError):
        dec.forward(s, [1, 2], [2])
    with pytest.raises(RuntimeError, match="logits of the last token"):
        dec.decode_greedy(s, 2)
    dec.forward(s, [1, 2, 3], [0])
    with pytest.raises(RuntimeError, match="logits of the last token"):
        dec.decode_greedy(s, 2)
    dec.forward(s, [1], [0])
    with pytest.raises(ValueError, match="further tokens fit"):
        dec.decode_greedy(s, 30)
    assert len(dec.decode_greedy(s, 17)) == 17 and s.pos == 20  # the last pick needs no step of its own
    assert dec.cache_bytes() > 0 and dec.weight_bytes_per_token() > 0 and dec.launches > 0


# ---- generation ------------------------------------------------------------------------------------------------------------
def oracle_greedy(cfg, w, prompt, n):
    """The oracle's continuation and the smallest margin between its first and second choice."""
    ref, out, margin = R.HybridReference(cfg, w), [], np.inf
    logits = ref.run(prompt)[-1]
    for _ in range(n):
        top = np.sort(logits)[-2:]
        margin = min(margin, top[1] - top[0])
        out.append(int(np.argmax(logits)))
        logits = ref.run([out[-1]])[-1]
    return out, margin


def test_greedy_generation_through_the_queue():
    cfg = CONFIGS["gqa"]
    w = random_weights(cfg, 77)
    dec = build_decoder(cfg, w, "float32", max_seq=300)
    rng = np.random.default_rng(2)
    prompts = [rng.integers(0, cfg["vocab"], n).tolist() for n in (1, 2, 40, 90)]
    for portion in (None, 7, 1):
        q = RequestQueue(dec, portion)
        reqs = [q.submit(p, 200 if len(p) == 40 else 30) for p in prompts]
        q.run()
        for r in reqs:
            want, margin = oracle_greedy(cfg, w, r.prompt, r.n_new)
            assert margin > 1e-4 and r.tokens == want  # (a margin the 32-bit mode resolves)
    bf = build_decoder(cfg, w, "bfloat16", max_seq=300)
    q = RequestQueue(bf, 16)
    reqs = [q.submit(p, 20) for p in prompts]
    q.run()
    for r in reqs:  # every pick is the arg-max, to bf16 accuracy, of the oracle's logits after the same tokens
        logits = R.HybridReference(cfg, w).run(r.prompt + r.tokens[:-1])[len(r.prompt) - 1:]
        picked = logits[np.arange(20), r.tokens]
        assert (logits.max(axis=1) - picked).max() < 0.15 * logits.std()


def test_trace_replay_generate_and_runner_from_a_model_folder(tmp_path):
    cfg = CONFIGS["wide"]
    w = random_weights(cfg, 5)
    folder = save_model(tmp_path / "model", cfg, w)
    toks = [int(t) for t in np.random.default_rng(3).integers(0, cfg["vocab"], 60)]
    want = R.HybridReference(cfg, w).run(toks)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:50], "want": [49, 3]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": toks[50:52], "want": []}], "end": []}]
    steps += [{"step": i - 50, "entries": [{"id": "x", "tokens": [toks[i]], "want": [0]}], "end": ["x"] if i == 59 else []} for i in range(52, 60)]
    steps.append({"step": 10, "entries": [{"id": "y", "tokens": toks[:1], "want": [0]}], "end": ["y"]})
    out = tmp_path / "out"
    out.mkdir()
    for dtype in ("float32", "bfloat16"):
        lines = [json.dumps(s) for s in steps]
        if dtype == "float32":
            r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", str(out), "--max-tokens", "64"],
                               input="\n".join(lines), capture_output=True, text=True, timeout=600)
            assert r.returncode == 0, r.stderr[-2000:]
            said = r.stdout.splitlines()
        else:
            said = []
            replay(load_model(folder, dtype, max_seq=64), lines, str(out), said.append)
        assert [x for x in said if x.startswith("done")] == [f"done {i}" for i in range(11)]
        got = np.concatenate([np.fromfile(out / f"{i}.f32", "<f4").reshape(-1, cfg["vocab"]) for i in [0, *range(2, 11)]])
        assert row_errors(got, want[[49, 3, *range(52, 60), 0]]).max() < LIMIT[dtype] and not (out / "1.f32").exists()
    r = subprocess.run([sys.executable, "-m", "cut_b200.generate", "--model", folder, "--tokens", "5,6,7;9", "--n", "6", "--dtype", "float32",
                        "--portion", "2"], capture_output=True, text=True, timeout=600, cwd=ROOT)
    assert r.returncode == 0, r.stderr[-2000:]
    lines = [json.loads(x) for x in r.stdout.splitlines()]
    for line in lines:
        picks, margin = oracle_greedy(cfg, w, line["prompt"], 6)
        assert margin > 1e-4 and line["tokens"] == picks
    assert [x["prompt"] for x in lines] == [[5, 6, 7], [9]]


@pytest.mark.parametrize("layers", [[with_mlp(mingru(40), 0)], [with_mlp(mingru(8), 16), with_mlp(mingru(24), 0)],
                                    [with_mlp(attention(2, 2, 16, 16, 3), 0)]])
def test_models_of_one_kind_of_layer(layers):
    cfg = config(24, 31, layers, groups=2, bigram=(3, 1, 1))
    w = random_weights(cfg, 6)
    toks = np.random.default_rng(1).integers(0, 31, 90)
    want = R.HybridReference(cfg, w).run(toks)
    dec = build_decoder(cfg, w, "float32", max_seq=90)
    assert row_errors(feed(dec, toks, [0, 90]), want).max() < LIMIT["float32"]
    assert row_errors(feed(dec, toks, list(range(91))), want).max() < LIMIT["float32"]
