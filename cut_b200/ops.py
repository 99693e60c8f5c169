"""Python harness over the C ABI: torch supplies device memory and streams only.

These wrappers mirror the reference's operator entry points for the path
(runtime/Operations.h:65-93 matmul / matmulUnary / matmulBinary, :459
transposeQ4, :467 dequantize): outputs are allocated by the op, shape errors
raise, and nothing here computes on the CPU.
"""
from __future__ import annotations

import ctypes as C

import torch

from . import _lib as L


def _stream_ptr() -> int:
    return torch.cuda.current_stream().cuda_stream


def _pad4(n: int) -> int:
    return (n + 3) & ~3


def make_desc(A: torch.Tensor, W: torch.Tensor, fmt: int, N: int, *, layout=L.LAYOUT_GGUF_BLOCKS, scales=None,
              affine=False, ldb=0, lds=0, C_out: torch.Tensor | None = None, D: torch.Tensor | None = None,
              fusion_type=L.FUSION_NONE, fusion_op=0, variant=L.VARIANT_AUTO, workspace: torch.Tensor | None = None,
              status: torch.Tensor | None = None, flags: int = 0):
    """Builds a cutb_qmatmul_desc over torch CUDA tensors; returns (desc, C, keepalive)."""
    if A.dim() == 1:
        A = A.unsqueeze(0)
    if A.dim() != 2:
        raise RuntimeError("matmul: A must be 1D or 2D")
    if A.dtype not in (torch.float32, torch.float16):
        raise RuntimeError("matmul: A must be float32 or float16")
    if A.stride(1) != 1:
        A = A.contiguous()
    M, K = A.shape
    if C_out is None:  # paired gate / up rows give one output column per pair
        C_out = torch.empty((M, N // 2 if flags & L.FLAG_GLU_PAIRS else N), dtype=torch.float32, device=A.device)
    d = L.QMatmulDesc()
    d.format, d.layout, d.affine = fmt, layout, int(affine)
    d.a_dtype = L.F32 if A.dtype == torch.float32 else L.F16
    d.M, d.K, d.N = M, K, N
    d.A, d.lda = A.data_ptr(), A.stride(0) if M > 1 else max(A.stride(0), K)
    d.W, d.W_bytes = W.data_ptr(), W.numel() * W.element_size()
    d.scales = scales.data_ptr() if scales is not None else None
    d.ldb, d.lds = ldb, lds
    d.C, d.ldc = C_out.data_ptr(), C_out.stride(0)
    d.D, d.ldd = (D.data_ptr(), D.stride(0)) if D is not None else (None, 0)
    d.fusion_type, d.fusion_op, d.variant = fusion_type, fusion_op, variant
    d.workspace, d.workspace_bytes = (workspace.data_ptr(), workspace.numel() * workspace.element_size()) \
        if workspace is not None else (None, 0)
    d.status = status.data_ptr() if status is not None else None
    d.flags = flags
    return d, C_out, (A, W, scales, D, workspace, status)


def workspace_bytes(desc) -> int:
    return int(L.lib().cutb_qmatmul_workspace_bytes(C.byref(desc)))


def select_variant(desc) -> int:
    return int(L.lib().cutb_qmatmul_select_variant(C.byref(desc)))


def qmatmul(A, W, fmt, N, **kw) -> torch.Tensor:
    """C[M,N] = epilogue(A[M,K] * dequant(W)); allocates C and, if needed, the workspace."""
    d, C_out, keep = make_desc(A, W, fmt, N, **kw)
    need = workspace_bytes(d)
    if need and not d.workspace:
        ws = torch.empty(need, dtype=torch.uint8, device=A.device)
        d.workspace, d.workspace_bytes = ws.data_ptr(), need
        keep = keep + (ws,)
    L.check(L.lib().cutb_qmatmul(C.byref(d), _stream_ptr()))
    return C_out


def launch(desc) -> None:
    """Re-launch a prepared descriptor on the current stream (benchmark inner loop)."""
    L.check(L.lib().cutb_qmatmul(C.byref(desc), _stream_ptr()))


def dequantize(raw: torch.Tensor, fmt: int, rows: int, cols: int, out: torch.Tensor | None = None) -> torch.Tensor:
    """Raw GGUF bytes -> float32 [rows, cols]; the row stride is padded to 4 as the
    reference's DequantOpNode does (operators/impl/dequant/DequantOp.cpp:15-17)."""
    ldo = _pad4(cols)
    if out is None:
        out = torch.empty((rows, ldo), dtype=torch.float32, device=raw.device)
    L.check(L.lib().cutb_dequant(fmt, raw.data_ptr(), raw.numel() * raw.element_size(), out.data_ptr(), rows, cols,
                                 out.stride(0), _stream_ptr()))
    return out[:, :cols]


def transpose_q4(packed: torch.Tensor, N: int, K: int) -> torch.Tensor:
    """[N, pad4(K/2)] GGML nibbles -> [K, pad4(N/2)] with even n in the low nibble."""
    if packed.dim() != 2:
        raise RuntimeError("TransposeQ4: input must be 2D")
    out = torch.zeros((K, _pad4(N // 2)), dtype=torch.uint8, device=packed.device)
    L.check(L.lib().cutb_transpose_q4(packed.data_ptr(), out.data_ptr(), N, K, packed.stride(0), out.stride(0),
                                      _stream_ptr()))
    return out


# ---- load-time repacks on the device (bit-exact with the reference's CPU loader / runner) ----
def separate_blocks(raw: torch.Tensor, fmt: int, rows: int, cols: int):
    """Q8_0 / Q4_0 blocks -> (values [rows, cols] int8 or packed nibbles [rows, cols / 2] uint8, scales [rows, cols / 32]
    as int16 bit patterns of f16), as the reference's read_tensor_q8/q4_separated return them."""
    vals = torch.empty((rows, cols if fmt == L.Q8_0 else cols // 2), dtype=torch.int8 if fmt == L.Q8_0 else torch.uint8,
                       device=raw.device)
    scales = torch.empty((rows, cols // 32), dtype=torch.int16, device=raw.device)
    L.check(L.lib().cutb_separate_blocks(fmt, raw.data_ptr(), raw.numel() * raw.element_size(), vals.data_ptr(), scales.data_ptr(),
                                         rows, cols, _stream_ptr()))
    return vals, scales


def transpose_2d(x: torch.Tensor, ldo: int | None = None) -> torch.Tensor:
    """[R, C] of 1- or 2-byte elements -> [C, ldo >= R] (padding zero-filled)."""
    R, Cc = x.shape
    ldo = R if ldo is None else ldo
    out = torch.zeros((Cc, ldo), dtype=x.dtype, device=x.device)
    L.check(L.lib().cutb_transpose_2d(x.element_size(), x.data_ptr(), out.data_ptr(), R, Cc, x.stride(0), ldo, _stream_ptr()))
    return out


def requant_q4k_affine(raw: torch.Tensor, N: int, K: int):
    """Q4_K rows -> (nibbles [K, N / 2] uint8, f16 bit patterns [2 K / 32, N] int16): the runner's affine re-encode."""
    packedT = torch.zeros((K, N // 2), dtype=torch.uint8, device=raw.device)
    scalesT = torch.zeros((2 * (K // 32), N), dtype=torch.int16, device=raw.device)
    L.check(L.lib().cutb_requant_q4k_affine(raw.data_ptr(), raw.numel() * raw.element_size(), packedT.data_ptr(), scalesT.data_ptr(),
                                            N, K, N // 2, N, _stream_ptr()))
    return packedT, scalesT


def quantize_rows_q8_0(x: torch.Tensor):
    """float32 values (multiple of 32) -> (int8 values, f16 scale bit patterns), the runner's Q8_0 requantiser."""
    x = x.contiguous().view(-1)
    vals = torch.empty(x.numel(), dtype=torch.int8, device=x.device)
    scales = torch.empty(x.numel() // 32, dtype=torch.int16, device=x.device)
    L.check(L.lib().cutb_quantize_rows_q8_0(x.data_ptr(), vals.data_ptr(), scales.data_ptr(), x.numel(), _stream_ptr()))
    return vals, scales


# ---- layer operators next to the matmul ----
def rmsnorm(x: torch.Tensor, weight: torch.Tensor, eps: float = 1e-5) -> torch.Tensor:
    """y = x * rsqrt(mean(x^2) + eps) * weight over the last dimension (fp32 or fp16, 1-D or 2-D)."""
    x2 = x if x.dim() == 2 else x.view(1, -1)
    if x2.stride(1) != 1 or weight.dtype != x.dtype:
        raise RuntimeError("rmsnorm: contiguous rows and a weight of the input's dtype")
    y = torch.empty_like(x2)
    dt = L.F16 if x.dtype == torch.float16 else L.F32
    L.check(L.lib().cutb_rmsnorm(dt, x2.data_ptr(), weight.data_ptr(), y.data_ptr(), x2.shape[0], x2.shape[1], x2.stride(0), eps,
                                 _stream_ptr()))
    return y.view_as(x)


def embedding(indices: torch.Tensor, table: torch.Tensor, dim: int | None = None, status: torch.Tensor | None = None) -> torch.Tensor:
    """table [vocab, pad4(dim)] float32, indices int32 -> [n, pad4(dim)]."""
    dim = table.shape[1] if dim is None else dim
    out = torch.empty((indices.numel(), table.shape[1]), dtype=torch.float32, device=table.device)
    L.check(L.lib().cutb_embedding(indices.data_ptr(), table.data_ptr(), out.data_ptr(), indices.numel(), dim, table.shape[0],
                                   status.data_ptr() if status is not None else None, _stream_ptr()))
    return out


def embedding_col(indices: torch.Tensor, matrix: torch.Tensor, scales: torch.Tensor | None = None, vocab: int | None = None,
                  status: torch.Tensor | None = None) -> torch.Tensor:
    """out[i, d] = M[d, indices[i]] for M [dim, vocab_stride] in float16, or int8 with float16 scales [dim / 32, scale_stride]."""
    dim, vstride = matrix.shape
    vocab = vstride if vocab is None else vocab
    fmt = 0 if matrix.dtype == torch.float16 else 1
    ld = (dim + 3) // 4 * 4
    out = torch.zeros((indices.numel(), ld), dtype=torch.float32, device=matrix.device)
    L.check(L.lib().cutb_embedding_col(fmt, indices.data_ptr(), matrix.data_ptr(), scales.data_ptr() if scales is not None else None,
                                       out.data_ptr(), indices.numel(), dim, vocab, vstride,
                                       scales.shape[1] if scales is not None else vstride, ld,
                                       status.data_ptr() if status is not None else None, _stream_ptr()))
    return out


def embedding_blocks(indices: torch.Tensor, raw: torch.Tensor, fmt: int, rows: int, cols: int,
                     status: torch.Tensor | None = None) -> torch.Tensor:
    """out[i, :] = dequant(row indices[i]) of a table kept as raw GGUF blocks (rows x cols weights)."""
    out = torch.empty((indices.numel(), cols), dtype=torch.float32, device=raw.device)
    L.check(L.lib().cutb_embedding_blocks(fmt, indices.data_ptr(), raw.data_ptr(), out.data_ptr(), indices.numel(), rows, cols, cols,
                                          status.data_ptr() if status is not None else None, _stream_ptr()))
    return out


def requant_q8_0_blocks(raw: torch.Tensor, fmt: int, rows: int, cols: int) -> torch.Tensor:
    """Raw blocks of any dequantisable format -> Q8_0 GGUF blocks (uint8, rows * cols / 32 * 34 bytes)."""
    out = torch.empty(rows * (cols // 32) * 34, dtype=torch.uint8, device=raw.device)
    L.check(L.lib().cutb_requant_q8_0_blocks(fmt, raw.data_ptr(), raw.numel() * raw.element_size(), out.data_ptr(), rows, cols,
                                             _stream_ptr()))
    return out


def argreduce(values: torch.Tensor, is_max: bool = True) -> torch.Tensor:
    """Index of the maximum / minimum as a one-element float tensor (the reference's output type and tie rule)."""
    out = torch.empty(1, dtype=torch.float32, device=values.device)
    L.check(L.lib().cutb_argreduce(1 if is_max else 0, values.data_ptr(), out.data_ptr(), values.numel(), _stream_ptr()))
    return out


# ---- decode-step attention ----
def _kv_dtype(cache: torch.Tensor) -> int:
    if cache.dtype == torch.float16:
        return L.F16
    if cache.dtype == torch.float32:
        return L.F32
    raise RuntimeError("KV cache must be float32 or float16")


def rope_kv_write(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, params: torch.Tensor, cos_t: torch.Tensor, sin_t: torch.Tensor,
                  k_cache: torch.Tensor, v_cache: torch.Tensor, head_dim: int, q_out: torch.Tensor | None = None,
                  status: torch.Tensor | None = None) -> torch.Tensor:
    """Half-split RoPE of q and k at params[0]; roped k and v go to row params[0] of the caches
    ([max_seq, ld]); returns the roped q.  params: int32/uint32 device tensor {pos, seqLen}."""
    if q_out is None:
        q_out = torch.empty_like(q)
    L.check(L.lib().cutb_rope_kv_write(_kv_dtype(k_cache), q.data_ptr(), k.data_ptr(), v.data_ptr(), params.data_ptr(),
                                       cos_t.data_ptr(), sin_t.data_ptr(), k_cache.data_ptr(), v_cache.data_ptr(), q_out.data_ptr(),
                                       q.numel(), k.numel(), head_dim, k_cache.stride(0), k_cache.shape[0],
                                       status.data_ptr() if status is not None else None, _stream_ptr()))
    return q_out


def attention_workspace(n_heads: int, n_kv_heads: int, head_dim: int, max_seq: int, device) -> torch.Tensor:
    """Zeroed scratch for attention_decode (its first 256 bytes are arrival counters that every launch leaves zero)."""
    n = int(L.lib().cutb_attention_workspace_bytes(n_heads, n_kv_heads, head_dim, max_seq))
    return torch.zeros(n, dtype=torch.uint8, device=device)


def attention_decode(q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, params: torch.Tensor, n_heads: int,
                     n_kv_heads: int, head_dim: int, workspace: torch.Tensor, out: torch.Tensor | None = None,
                     scale: float | None = None, status: torch.Tensor | None = None) -> torch.Tensor:
    """Grouped-query attention of one roped query [n_heads * head_dim] over rows [0, params[1]) of the caches."""
    if out is None:
        out = torch.empty(n_heads * head_dim, dtype=torch.float32, device=q.device)
    if scale is None:
        scale = 1.0 / float(head_dim) ** 0.5
    L.check(L.lib().cutb_attention_decode(_kv_dtype(k_cache), q.data_ptr(), k_cache.data_ptr(), v_cache.data_ptr(), params.data_ptr(),
                                          out.data_ptr(), n_heads, n_kv_heads, head_dim, k_cache.stride(0), k_cache.shape[0],
                                          scale, workspace.data_ptr(), workspace.numel(),
                                          status.data_ptr() if status is not None else None, _stream_ptr()))
    return out


def rope_attention_decode(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, params: torch.Tensor, cos_t: torch.Tensor,
                          sin_t: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, n_heads: int, n_kv_heads: int,
                          head_dim: int, workspace: torch.Tensor, out: torch.Tensor | None = None, scale: float | None = None,
                          status: torch.Tensor | None = None) -> torch.Tensor:
    """rope_kv_write + attention_decode in one call (one launch where the cluster kernel applies)."""
    if out is None:
        out = torch.empty(n_heads * head_dim, dtype=torch.float32, device=q.device)
    if scale is None:
        scale = 1.0 / float(head_dim) ** 0.5
    L.check(L.lib().cutb_rope_attention_decode(_kv_dtype(k_cache), q.data_ptr(), k.data_ptr(), v.data_ptr(), params.data_ptr(),
                                               cos_t.data_ptr(), sin_t.data_ptr(), k_cache.data_ptr(), v_cache.data_ptr(),
                                               out.data_ptr(), n_heads, n_kv_heads, head_dim, k_cache.stride(0), k_cache.shape[0],
                                               scale, workspace.data_ptr(), workspace.numel(),
                                               status.data_ptr() if status is not None else None, _stream_ptr()))
    return out


# ---- prefill (a batch of prompt tokens) ----
def batched_kv_write(k_in: torch.Tensor, v_in: torch.Tensor, positions: torch.Tensor, cos_t: torch.Tensor, sin_t: torch.Tensor,
                     k_cache: torch.Tensor, v_cache: torch.Tensor, head_dim: int, status: torch.Tensor | None = None) -> None:
    """k_cache[positions[i]] = RoPE(k_in[i]), v_cache[positions[i]] = v_in[i]; k_in / v_in are [T, kv_dim] views (any row stride)."""
    L.check(L.lib().cutb_batched_kv_write(_kv_dtype(k_cache), k_in.data_ptr(), v_in.data_ptr(), k_in.stride(0), v_in.stride(0),
                                          positions.data_ptr(), cos_t.data_ptr(), sin_t.data_ptr(), k_cache.data_ptr(),
                                          v_cache.data_ptr(), k_in.shape[0], k_in.shape[1], head_dim, k_cache.stride(0),
                                          k_cache.shape[0], status.data_ptr() if status is not None else None, _stream_ptr()))


def batched_attention(q_in: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, positions: torch.Tensor, cos_t: torch.Tensor,
                      sin_t: torch.Tensor, n_heads: int, n_kv_heads: int, head_dim: int, out: torch.Tensor | None = None,
                      scale: float | None = None, status: torch.Tensor | None = None) -> torch.Tensor:
    """out[i] = attention of RoPE(q_in[i]) over cache rows [0, positions[i]]; q_in is a [T, n_heads * head_dim] view."""
    T = q_in.shape[0]
    if out is None:
        out = torch.empty((T, n_heads * head_dim), dtype=torch.float32, device=q_in.device)
    if scale is None:
        scale = 1.0 / float(head_dim) ** 0.5
    L.check(L.lib().cutb_batched_attention(_kv_dtype(k_cache), q_in.data_ptr(), q_in.stride(0), k_cache.data_ptr(), v_cache.data_ptr(),
                                           positions.data_ptr(), cos_t.data_ptr(), sin_t.data_ptr(), out.data_ptr(), out.stride(0), T,
                                           n_heads, n_kv_heads, head_dim, k_cache.stride(0), k_cache.shape[0], scale,
                                           status.data_ptr() if status is not None else None, _stream_ptr()))
    return out


def glu_pairs(x: torch.Tensor, unary_op: int = 133, out: torch.Tensor | None = None) -> torch.Tensor:
    """out[r, i] = unary(x[r, 2i]) * x[r, 2i + 1] (SiLU by default)."""
    rows, cols = x.shape
    if out is None:
        out = torch.empty((rows, cols // 2), dtype=torch.float32, device=x.device)
    L.check(L.lib().cutb_glu_pairs(x.data_ptr(), out.data_ptr(), rows, cols // 2, x.stride(0), out.stride(0), unary_op, _stream_ptr()))
    return out



# ---- layer-list models: dense bf16 weights, windowed attention, gated recurrence ----
def _el(t: torch.Tensor) -> int:
    if t.dtype == torch.bfloat16:
        return L.BF16
    if t.dtype == torch.float32:
        return L.F32
    raise RuntimeError("element types here are float32 and bfloat16")


def _ptr(t: torch.Tensor | None):
    return t.data_ptr() if t is not None else None


def dense_desc(A: torch.Tensor | None, W: torch.Tensor, K: int, out: torch.Tensor, *, bias=None, unary: int = 0, variant: int = L.DENSE_AUTO,
               status=None, M: int | None = None, N: int | None = None):
    """cutb_dense_desc of out[M, N] = unary(A[M, K] W[N, :K]^T + bias); W bf16 with rows padded to 8, out a 2-D view.  A may be
    None when the input is staged from the residual stream (ops.stage_input)."""
    d = L.DenseDesc()
    d.M, d.K, d.N = (A.shape[0] if A is not None else 1) if M is None else M, K, W.shape[0] if N is None else N
    d.a_dtype, d.c_dtype = _el(A) if A is not None else L.F32, _el(out)
    if A is not None:
        d.A, d.lda = A.data_ptr(), A.stride(0)
    d.W, d.ldw, d.bias = W.data_ptr(), W.stride(0), _ptr(bias)
    d.unary_op, d.C, d.ldc, d.variant, d.status = unary, out.data_ptr(), out.stride(0), variant, _ptr(status)
    return d


def stage_input(d, x: torch.Tensor, norm_w: torch.Tensor, groups: int, eps: float, y=None, post_w=None, x_out=None, center: bool = False,
                y_scale: float = 1.0, norm_out=None):
    """Makes the mat-vec of `d` read N(x + y_scale P(y); norm_w) instead of A, P = N(.; post_w) or without post_w the identity, N =
    RMS norm or (center) layer norm; x + ... also goes to x_out, the normed row to norm_out."""
    d.res_x, d.norm_w, d.norm_groups, d.norm_eps, d.norm_center, d.res_scale = x.data_ptr(), norm_w.data_ptr(), groups, eps, int(center), y_scale
    d.res_y, d.res_norm_w, d.res_out, d.norm_out = _ptr(y), _ptr(post_w), _ptr(x_out), _ptr(norm_out)
    return d


def batch_desc(A: torch.Tensor, W: torch.Tensor, K: int, out: torch.Tensor, heads: int, a_step: int, c_step: int, *, status=None, low=None,
               scale: float = 1.0):
    """cutb_dense_desc of `heads` products: number b maps columns b * a_step .. + K of A by rows b N .. of W to columns b * c_step .. of out.
    low (one row, bf16 out): the results times scale as the sum of out and low."""
    d = dense_desc(A, W, K, out, status=status, N=W.shape[0] // heads)
    d.batch, d.a_batch, d.c_batch, d.c_low, d.c_scale = heads, a_step, c_step, _ptr(low), scale
    return d


def dense_matmul(d) -> None:
    """Launches a dense matmul, with a workspace of its own if the shape asks for one and the descriptor has none."""
    need = int(L.lib().cutb_dense_workspace_bytes(C.byref(d)))
    ws = None
    if need and not d.workspace:
        ws = torch.empty(need, dtype=torch.uint8, device="cuda")
        d.workspace, d.workspace_bytes = ws.data_ptr(), need
    L.check(L.lib().cutb_dense_matmul(C.byref(d), _stream_ptr()))
    if ws is not None:
        d.workspace, d.workspace_bytes = None, 0


def residual_norm(x: torch.Tensor, norm_w: torch.Tensor, groups: int, eps: float, *, dim: int | None = None, y=None, post_w=None, x_out=None,
                  out: torch.Tensor | None = None, dtype=torch.float32, row_index=None, center: bool = False, y_scale: float = 1.0,
                  parts=None) -> torch.Tensor:
    """h = N(x + y_scale P(y + parts); norm_w) row by row (P = N(.; post_w), or the identity without post_w; N = RMS norm, or layer norm
    with center); the new residual goes to x_out when given (x itself is allowed).  parts: (matrix, rows [., n] int32, weights [., n]):
    row r gains sum_k weights[r, k] * matrix[rows[r, k]]."""
    d = L.ResidualNormDesc()
    dim = x.shape[1] if dim is None else dim
    rows = x.shape[0] if row_index is None else row_index.numel()
    if out is None:
        out = torch.zeros((rows, x.stride(0)), dtype=dtype, device=x.device)
    d.x, d.ldx, d.pre_w, d.x_out = x.data_ptr(), x.stride(0), norm_w.data_ptr(), _ptr(x_out)
    if y is not None:
        d.y, d.ldy = y.data_ptr(), y.stride(0)
    if parts is not None:
        m, part_rows, part_w = parts
        d.parts, d.parts_dtype, d.ld_parts = m.data_ptr(), _el(m), m.stride(0)
        d.part_rows, d.part_w, d.n_parts = part_rows.data_ptr(), part_w.data_ptr(), part_w.shape[1]
    d.post_w, d.center, d.y_scale = _ptr(post_w), int(center), y_scale
    d.h, d.ldh, d.h_dtype, d.row_index = out.data_ptr(), out.stride(0), _el(out), _ptr(row_index)
    d.rows, d.dim, d.groups, d.eps = rows, dim, groups, eps
    L.check(L.lib().cutb_residual_norm(C.byref(d), _stream_ptr()))
    return out


def embedding_bigram(tokens: torch.Tensor, embed: torch.Tensor, *, prev=None, bigram=None, mul_prev: int = 0, mul_cur: int = 0,
                     status=None, scale: float = 1.0) -> torch.Tensor:
    """scale * embed[token] + bigram[hash of (previous token, token)] for int32 tokens; prev: one-element int32 tensor or None."""
    n, dim = tokens.numel(), embed.shape[1]
    out = torch.empty((n, dim), dtype=torch.float32, device=embed.device)
    d = L.EmbedDesc()
    d.tokens, d.prev, d.embed, d.ld_embed, d.out, d.ldo = tokens.data_ptr(), _ptr(prev), embed.data_ptr(), embed.stride(0), out.data_ptr(), dim
    if bigram is not None:
        d.bigram, d.ld_bigram, d.buckets, d.mul_prev, d.mul_cur = bigram.data_ptr(), bigram.stride(0), bigram.shape[0] - 1, mul_prev, mul_cur
    d.n, d.dim, d.vocab, d.status, d.scale = n, dim, embed.shape[0], _ptr(status), scale
    L.check(L.lib().cutb_embedding_bigram(C.byref(d), _stream_ptr()))
    return out


def mingru_scan(zxg: torch.Tensor, width: int, state: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
    """The recurrence over the rows of zxg ([T, >= 3 width] pre-activations); state is continued in place."""
    L.check(L.lib().cutb_mingru_scan(zxg.data_ptr(), zxg.stride(0), width, state.data_ptr(), out.data_ptr(), _el(out), out.stride(0),
                                     zxg.shape[0], _stream_ptr()))
    return out


def window_desc(qkv: torch.Tensor, n_heads: int, n_kv_heads: int, dim: int, vdim: int, k_cache: torch.Tensor, v_cache: torch.Tensor, *,
                window: int, scale: float, out: torch.Tensor, cos_t=None, sin_t=None, rot_dims: int = 0, pairing: int = L.ROT_NEIGHBOURS,
                max_pos: int, sink: bool = False, pos: int = 0, pos_ptr: int | None = None, v_first=None, v_mix: float = 0.0,
                v_first_out=None, status=None):
    """cutb_window_attn_desc over rows [q | k | v] of a stacked projection and ring caches [ring_rows, n_kv_heads * pad8(head)]."""
    d = L.WindowAttnDesc()
    d.kv_dtype, d.out_dtype = _el(k_cache), _el(out)
    d.n_heads, d.n_kv_heads, d.dim, d.vdim = n_heads, n_kv_heads, dim, vdim
    d.k_head, d.v_head, d.ring_rows = k_cache.shape[1] // n_kv_heads, v_cache.shape[1] // n_kv_heads, k_cache.shape[0]
    d.window, d.rot_dims, d.max_pos, d.rot_pairing, d.sink = window, rot_dims, max_pos, pairing, int(sink)
    d.scale, d.v_mix, d.cos_table, d.sin_table = scale, v_mix, _ptr(cos_t), _ptr(sin_t)
    p, q_rows, k_rows = qkv.data_ptr(), n_heads * dim, n_kv_heads * dim
    d.q, d.k, d.v, d.ldqkv = p, p + 4 * q_rows, p + 4 * (q_rows + k_rows), qkv.stride(0)
    d.k_cache, d.v_cache = k_cache.data_ptr(), v_cache.data_ptr()
    d.v_first, d.v_first_out = _ptr(v_first), _ptr(v_first_out)
    first = v_first if v_first is not None else v_first_out
    d.ld_first = first.stride(0) if first is not None else 0
    d.pos_ptr, d.pos, d.n_tokens = pos_ptr, pos, qkv.shape[0]
    d.out, d.ldo, d.status = out.data_ptr(), out.stride(0), _ptr(status)
    return d


def window_kv_write(d) -> None:
    L.check(L.lib().cutb_window_kv_write(C.byref(d), _stream_ptr()))


def window_attention(d) -> None:
    L.check(L.lib().cutb_window_attention(C.byref(d), _stream_ptr()))


def window_attention_decode(d) -> None:
    L.check(L.lib().cutb_window_attention_decode(C.byref(d), _stream_ptr()))


# ---- latent attention, mixtures of experts ----
def latent_desc(cache: torch.Tensor, n_heads: int, dim: int, rot_dim: int, vdim: int, rank: int, *, scale: float, eps: float, max_pos: int,
                n_tokens: int, cos_t=None, sin_t=None, sink=None, pos: int = 0, pos_ptr: int | None = None, lat=None, lat_norm_w=None, cq=None,
                cq_norm_w=None, cq_out=None, q=None, qa=None, qa_split=None, k_exp=None, v_exp=None, out=None, workspace=None, w_uv=None, status=None):
    """cutb_latent_attn_desc over a cache [rows, pad8(rank) + pad8(rot_dim)]; what a call does not use may be missing."""
    d = L.LatentAttnDesc()
    shape = out if out is not None else cq_out
    d.kv_dtype, d.out_dtype = _el(cache), _el(shape) if shape is not None else L.F32
    d.n_heads, d.dim, d.rot_dim, d.vdim, d.rank, d.rot_at, d.max_pos = n_heads, dim, rot_dim, vdim, rank, (rank + 7) // 8 * 8, max_pos
    d.scale, d.eps, d.sink, d.cos_table, d.sin_table = scale, eps, _ptr(sink), _ptr(cos_t), _ptr(sin_t)
    d.cache, d.ld_cache, d.n_tokens, d.pos, d.pos_ptr, d.status = cache.data_ptr(), cache.stride(0), n_tokens, pos, pos_ptr, _ptr(status)
    if lat is not None:
        d.lat, d.ld_lat, d.lat_norm_w = lat.data_ptr(), lat.stride(0), lat_norm_w.data_ptr()
    if cq is not None:
        d.cq, d.ld_cq, d.q_rank, d.cq_norm_w = cq.data_ptr(), cq.stride(0), cq_norm_w.numel(), cq_norm_w.data_ptr()
        d.cq_out, d.ld_cq_out = cq_out.data_ptr(), cq_out.stride(0)
    for name, t in (("q", q), ("qa", qa), ("k_exp", k_exp), ("v_exp", v_exp), ("out", out), ("w_uv", w_uv)):
        if t is not None:
            setattr(d, name, t.data_ptr())
            setattr(d, {"q": "ldq", "qa": "ld_qa", "k_exp": "ld_k", "v_exp": "ld_v", "out": "ldo", "w_uv": "ld_uv"}[name], t.stride(0))
    if qa_split is not None:  # (high, low) [heads, pad8(rank)] bf16
        d.qa_high, d.qa_low, d.ld_qa_split = qa_split[0].data_ptr(), qa_split[1].data_ptr(), qa_split[0].stride(0)
    if workspace is not None:
        d.workspace, d.workspace_bytes = workspace.data_ptr(), workspace.numel() * workspace.element_size()
    return d


def latent_takes_split_queries(d) -> bool:
    return bool(L.lib().cutb_latent_takes_split_queries(C.byref(d)))


def latent_workspace_bytes(d) -> int:
    return int(L.lib().cutb_latent_workspace_bytes(C.byref(d)))


def moe_route_desc(logits: torch.Tensor, experts: int, top: int, weights, ids, slots, offsets):
    """cutb_moe_desc of a batch's routing: logits [T, >= experts]; weights, ids, slots [T, top], offsets [experts + 1] are written."""
    d = L.MoeDesc()
    d.n_tokens, d.experts, d.top = logits.shape[0], experts, top
    d.logits, d.ld_logits = logits.data_ptr(), logits.stride(0)
    d.weights, d.ids, d.slots, d.offsets = weights.data_ptr(), ids.data_ptr(), slots.data_ptr(), offsets.data_ptr()
    return d


def moe_scatter_desc(x: torch.Tensor, K: int, slots: torch.Tensor, experts: int, out: torch.Tensor):
    """out[slots[t, k]] = x[t, :K]."""
    d = L.MoeDesc()
    d.n_tokens, d.top, d.experts, d.K = slots.shape[0], slots.shape[1], experts, K
    d.A, d.lda, d.a_dtype, d.C, d.ldc, d.c_dtype, d.slots = x.data_ptr(), x.stride(0), _el(x), out.data_ptr(), out.stride(0), _el(out), slots.data_ptr()
    return d


def moe_matmul_desc(A: torch.Tensor, W: torch.Tensor, K: int, offsets: torch.Tensor, experts: int, tokens: int, top: int, out: torch.Tensor, *,
                    glu: int = L.GLU_NONE, alpha: float = 0.0, beta: float = 0.0, limit: float = 0.0, variant: int = L.DENSE_SIMT, status=None):
    """The grouped product of expert-sorted rows A [tokens * top, K] with the experts' stacked matrices W [experts * N, ldw]."""
    d = L.MoeDesc()
    d.n_tokens, d.top, d.experts, d.K, d.N = tokens, top, experts, K, W.shape[0] // experts
    d.A, d.lda, d.a_dtype, d.W, d.ldw, d.C, d.ldc, d.c_dtype = A.data_ptr(), A.stride(0), _el(A), W.data_ptr(), W.stride(0), out.data_ptr(), out.stride(0), _el(out)
    d.offsets, d.glu, d.alpha, d.beta, d.limit, d.variant, d.status = offsets.data_ptr(), glu, alpha, beta, limit, variant, _ptr(status)
    return d


def expert_desc(experts: int, top: int, width: int, ff: int, W: torch.Tensor, ids: torch.Tensor, act: torch.Tensor, *, logits=None, x=None,
                alpha: float = 0.0, beta: float = 0.0, limit: float = 0.0, dense=None, dense_K: int = 0, xd=None, xd_norm_w=None, eps: float = 0.0,
                out=None):
    """cutb_expert_desc of one token's expert mat-vecs (logits and x: cutb_expert_up); dense: the companion matrix."""
    d = L.ExpertDesc()
    d.experts, d.top, d.width, d.ff, d.W, d.ldw = experts, top, width, ff, W.data_ptr(), W.stride(0)
    d.ids, d.act, d.logits, d.x, d.alpha, d.beta, d.limit = ids.data_ptr(), act.data_ptr(), _ptr(logits), _ptr(x), alpha, beta, limit
    if dense is not None:
        d.Wd, d.Nd, d.Kd, d.ldwd = dense.data_ptr(), dense.shape[0], dense_K, dense.stride(0)
        d.xd, d.xd_norm_w, d.eps = xd.data_ptr(), _ptr(xd_norm_w), eps
    d.C = _ptr(out)
    return d


def launch_layer_op(name: str, d) -> None:
    """Launches a layer operator (an entry point that takes a descriptor and a stream)."""
    L.check(getattr(L.lib(), name)(C.byref(d), _stream_ptr()))
