"""ctypes view of libcutb.so, laid out exactly as include/cutb.h declares it.

There is no fallback: if the library has not been built, loading raises.
"""
from __future__ import annotations

import ctypes as C
import os

HERE = os.path.dirname(os.path.abspath(__file__))
LIB_PATH = os.path.join(HERE, "libcutb.so")

OK, ERR_INVALID, ERR_UNSUPPORTED, ERR_CUDA, ERR_WORKSPACE, ERR_TIMEOUT, ERR_RANGE = range(7)
Q8_0, Q4_0, Q4_K, Q5_K, Q6_K, BF16, Q4_1, Q5_0 = 0, 1, 2, 3, 4, 5, 6, 7  # from Q5_K on: cutb_dequant only
F32, F16 = 0, 1
UNARY_RELU_SQUARE, NO_TOKEN = 200, 0xFFFFFFFF
GLU_NONE, GLU_CLAMPED = 0, 1
DENSE_AUTO, DENSE_MATVEC, DENSE_TC, DENSE_SIMT = -1, 0, 1, 2
ROT_HALVES, ROT_NEIGHBOURS = 0, 1
LAYOUT_GGUF_BLOCKS, LAYOUT_KN_PLANES = 0, 1
FUSION_NONE, FUSION_UNARY, FUSION_BINARY = 0, 1, 2
VARIANT_AUTO, VARIANT_GENERIC, VARIANT_GEMV_MMA, VARIANT_GEMM_TC, VARIANT_GEMV_PLANES = -1, 0, 1, 2, 3
FLAG_NO_OVERLAP = 1
FLAG_ACT_16BIT = 2
FLAG_A_RMSNORM = 4
FLAG_GLU_PAIRS = 8
FLAG_STAGE_PER_CTA = 16

# every symbol include/cutb.h declares
EXPORTS = [
    "cutb_qmatmul_workspace_bytes", "cutb_qmatmul_select_variant", "cutb_qmatmul", "cutb_qmatmul_decode_noalloc",
    "cutb_qmatmul_scatter", "cutb_peer_exchange", "cutb_copy_batch",
    "cutb_peer_buffer_alloc", "cutb_peer_buffer_open", "cutb_peer_buffer_close", "cutb_peer_buffer_free",
    "cutb_rmsnorm", "cutb_embedding", "cutb_embedding_col", "cutb_embedding_blocks", "cutb_argreduce",
    "cutb_rope_kv_write", "cutb_attention_workspace_bytes", "cutb_attention_decode", "cutb_rope_attention_decode",
    "cutb_batched_kv_write", "cutb_batched_attention", "cutb_glu_pairs",
    "cutb_dequant", "cutb_separate_blocks", "cutb_transpose_2d", "cutb_requant_q4k_affine", "cutb_quantize_rows_q8_0", "cutb_requant_q8_0_blocks",
    "cutb_transpose_q4", "cutb_version", "cutb_status_string", "cutb_last_error", "cutb_device_sm_count",
    "cutb_variant_name",
    "cutb_dense_select_variant", "cutb_dense_workspace_bytes", "cutb_dense_matmul", "cutb_residual_norm", "cutb_embedding_bigram",
    "cutb_mingru_scan", "cutb_sequence_advance", "cutb_window_kv_write", "cutb_window_attention", "cutb_window_attention_decode",
    "cutb_latent_kv_write", "cutb_latent_attention", "cutb_latent_takes_split_queries", "cutb_latent_splits", "cutb_latent_workspace_bytes", "cutb_latent_values",
    "cutb_latent_prefill_supported", "cutb_latent_prefill", "cutb_moe_route", "cutb_moe_scatter", "cutb_moe_matmul", "cutb_expert_up",
    "cutb_expert_down",
]


class QMatmulDesc(C.Structure):
    _fields_ = [
        ("format", C.c_int32), ("layout", C.c_int32), ("affine", C.c_int32), ("a_dtype", C.c_int32),
        ("M", C.c_uint32), ("K", C.c_uint32), ("N", C.c_uint32),
        ("A", C.c_void_p), ("lda", C.c_uint32),
        ("W", C.c_void_p), ("W_bytes", C.c_uint64),
        ("scales", C.c_void_p), ("ldb", C.c_uint32), ("lds", C.c_uint32),
        ("C", C.c_void_p), ("ldc", C.c_uint32),
        ("D", C.c_void_p), ("ldd", C.c_uint32),
        ("fusion_type", C.c_int32), ("fusion_op", C.c_int32), ("variant", C.c_int32),
        ("workspace", C.c_void_p), ("workspace_bytes", C.c_uint64),
        ("status", C.c_void_p),
        ("flags", C.c_uint32),
        ("a_norm_weight", C.c_void_p), ("a_norm_eps", C.c_float),
    ]


class DenseDesc(C.Structure):
    _fields_ = [
        ("a_dtype", C.c_int32), ("c_dtype", C.c_int32),
        ("M", C.c_uint32), ("K", C.c_uint32), ("N", C.c_uint32),
        ("A", C.c_void_p), ("lda", C.c_uint32),
        ("W", C.c_void_p), ("ldw", C.c_uint32),
        ("bias", C.c_void_p), ("unary_op", C.c_int32),
        ("C", C.c_void_p), ("ldc", C.c_uint32),
        ("variant", C.c_int32), ("flags", C.c_uint32),
        ("workspace", C.c_void_p), ("workspace_bytes", C.c_uint64),
        ("status", C.c_void_p),
        ("res_x", C.c_void_p), ("res_y", C.c_void_p), ("res_norm_w", C.c_void_p), ("norm_w", C.c_void_p),
        ("res_out", C.c_void_p),
        ("norm_groups", C.c_uint32), ("norm_eps", C.c_float),
        ("gru_state", C.c_void_p),
        ("norm_center", C.c_int32), ("res_scale", C.c_float), ("norm_out", C.c_void_p),
        ("batch", C.c_uint32), ("a_batch", C.c_uint32), ("c_batch", C.c_uint32),
        ("c_low", C.c_void_p), ("c_scale", C.c_float),
    ]


class ResidualNormDesc(C.Structure):
    _fields_ = [
        ("x", C.c_void_p), ("y", C.c_void_p), ("post_w", C.c_void_p), ("pre_w", C.c_void_p),
        ("x_out", C.c_void_p), ("h", C.c_void_p), ("row_index", C.c_void_p),
        ("ldx", C.c_uint64), ("ldy", C.c_uint64), ("ldh", C.c_uint64),
        ("rows", C.c_uint32), ("dim", C.c_uint32), ("groups", C.c_uint32),
        ("eps", C.c_float), ("h_dtype", C.c_int32),
        ("center", C.c_int32), ("y_scale", C.c_float),
        ("parts", C.c_void_p), ("part_rows", C.c_void_p), ("part_w", C.c_void_p), ("ld_parts", C.c_uint64),
        ("n_parts", C.c_uint32), ("parts_dtype", C.c_int32),
    ]


class EmbedDesc(C.Structure):
    _fields_ = [
        ("tokens", C.c_void_p), ("prev", C.c_void_p), ("embed", C.c_void_p), ("bigram", C.c_void_p), ("out", C.c_void_p),
        ("ld_embed", C.c_uint64), ("ld_bigram", C.c_uint64), ("ldo", C.c_uint64),
        ("n", C.c_uint32), ("dim", C.c_uint32), ("vocab", C.c_uint32), ("buckets", C.c_uint32),
        ("mul_prev", C.c_uint32), ("mul_cur", C.c_uint32),
        ("status", C.c_void_p), ("scale", C.c_float),
    ]


class WindowAttnDesc(C.Structure):
    _fields_ = [
        ("kv_dtype", C.c_int32), ("out_dtype", C.c_int32),
        ("n_heads", C.c_uint32), ("n_kv_heads", C.c_uint32), ("dim", C.c_uint32), ("vdim", C.c_uint32),
        ("k_head", C.c_uint32), ("v_head", C.c_uint32),
        ("ring_rows", C.c_uint32), ("window", C.c_uint32), ("rot_dims", C.c_uint32), ("max_pos", C.c_uint32),
        ("rot_pairing", C.c_int32), ("sink", C.c_int32),
        ("scale", C.c_float), ("v_mix", C.c_float),
        ("cos_table", C.c_void_p), ("sin_table", C.c_void_p),
        ("q", C.c_void_p), ("k", C.c_void_p), ("v", C.c_void_p), ("ldqkv", C.c_uint64),
        ("k_cache", C.c_void_p), ("v_cache", C.c_void_p),
        ("v_first", C.c_void_p), ("v_first_out", C.c_void_p), ("ld_first", C.c_uint64),
        ("pos_ptr", C.c_void_p), ("pos", C.c_uint32), ("n_tokens", C.c_uint32),
        ("out", C.c_void_p), ("ldo", C.c_uint64),
        ("status", C.c_void_p),
    ]


class LatentAttnDesc(C.Structure):
    _fields_ = [
        ("kv_dtype", C.c_int32), ("out_dtype", C.c_int32),
        ("n_heads", C.c_uint32), ("dim", C.c_uint32), ("rot_dim", C.c_uint32), ("vdim", C.c_uint32), ("rank", C.c_uint32),
        ("rot_at", C.c_uint32), ("q_rank", C.c_uint32), ("max_pos", C.c_uint32),
        ("scale", C.c_float), ("eps", C.c_float),
        ("sink", C.c_void_p), ("cos_table", C.c_void_p), ("sin_table", C.c_void_p),
        ("lat", C.c_void_p), ("lat_norm_w", C.c_void_p), ("cq", C.c_void_p), ("cq_norm_w", C.c_void_p),
        ("ld_lat", C.c_uint64), ("ld_cq", C.c_uint64), ("ld_cq_out", C.c_uint64),
        ("cq_out", C.c_void_p),
        ("q", C.c_void_p), ("qa", C.c_void_p), ("ldq", C.c_uint64), ("ld_qa", C.c_uint64),
        ("cache", C.c_void_p), ("ld_cache", C.c_uint64),
        ("k_exp", C.c_void_p), ("v_exp", C.c_void_p), ("ld_k", C.c_uint64), ("ld_v", C.c_uint64),
        ("pos_ptr", C.c_void_p), ("pos", C.c_uint32), ("n_tokens", C.c_uint32),
        ("out", C.c_void_p), ("ldo", C.c_uint64),
        ("workspace", C.c_void_p), ("workspace_bytes", C.c_uint64),
        ("status", C.c_void_p),
        ("w_uv", C.c_void_p), ("ld_uv", C.c_uint64),
        ("qa_high", C.c_void_p), ("qa_low", C.c_void_p), ("ld_qa_split", C.c_uint64),
    ]


class MoeDesc(C.Structure):
    _fields_ = [
        ("n_tokens", C.c_uint32), ("experts", C.c_uint32), ("top", C.c_uint32), ("K", C.c_uint32), ("N", C.c_uint32),
        ("logits", C.c_void_p), ("ld_logits", C.c_uint64),
        ("weights", C.c_void_p), ("ids", C.c_void_p), ("slots", C.c_void_p), ("offsets", C.c_void_p),
        ("a_dtype", C.c_int32), ("c_dtype", C.c_int32),
        ("A", C.c_void_p), ("lda", C.c_uint64), ("W", C.c_void_p), ("ldw", C.c_uint32),
        ("C", C.c_void_p), ("ldc", C.c_uint64),
        ("glu", C.c_int32), ("alpha", C.c_float), ("beta", C.c_float), ("limit", C.c_float),
        ("variant", C.c_int32), ("status", C.c_void_p),
    ]


class ExpertDesc(C.Structure):
    _fields_ = [
        ("experts", C.c_uint32), ("top", C.c_uint32), ("width", C.c_uint32), ("ff", C.c_uint32),
        ("logits", C.c_void_p), ("ids", C.c_void_p), ("W", C.c_void_p), ("ldw", C.c_uint32),
        ("x", C.c_void_p), ("act", C.c_void_p),
        ("alpha", C.c_float), ("beta", C.c_float), ("limit", C.c_float),
        ("Wd", C.c_void_p), ("Nd", C.c_uint32), ("Kd", C.c_uint32), ("ldwd", C.c_uint32),
        ("xd", C.c_void_p), ("xd_norm_w", C.c_void_p), ("eps", C.c_float),
        ("C", C.c_void_p), ("flags", C.c_uint32),
    ]


MAX_PEERS = 8


class PeerScatter(C.Structure):
    _fields_ = [
        ("world", C.c_uint32), ("rank", C.c_uint32), ("ldc_total", C.c_uint32), ("n_offset", C.c_uint32),
        ("C_peers", C.c_void_p * MAX_PEERS), ("flag_peers", C.c_void_p * MAX_PEERS),
    ]


class CutbError(RuntimeError):
    def __init__(self, status: int, message: str):
        super().__init__(f"cutb status {status}: {message}")
        self.status = status


_lib = None


def _bind_layers(l: C.CDLL) -> None:
    l.cutb_copy_batch.restype = C.c_int
    l.cutb_copy_batch.argtypes = [C.c_void_p, C.c_uint32, C.c_uint64, C.c_void_p]
    l.cutb_rmsnorm.restype = C.c_int
    l.cutb_rmsnorm.argtypes = [C.c_int, C.c_void_p, C.c_void_p, C.c_void_p, C.c_uint32, C.c_uint32, C.c_uint64, C.c_float, C.c_void_p]
    l.cutb_embedding.restype = C.c_int
    l.cutb_embedding.argtypes = [C.c_void_p, C.c_void_p, C.c_void_p, C.c_uint64, C.c_uint32, C.c_uint32, C.c_void_p, C.c_void_p]
    l.cutb_embedding_col.restype = C.c_int
    l.cutb_embedding_col.argtypes = [C.c_int, C.c_void_p, C.c_void_p, C.c_void_p, C.c_void_p, C.c_uint32, C.c_uint32, C.c_uint32,
                                     C.c_uint32, C.c_uint32, C.c_uint32, C.c_void_p, C.c_void_p]
    l.cutb_argreduce.restype = C.c_int
    l.cutb_argreduce.argtypes = [C.c_int, C.c_void_p, C.c_void_p, C.c_uint32, C.c_void_p]
    l.cutb_glu_pairs.restype = C.c_int
    l.cutb_glu_pairs.argtypes = [C.c_void_p, C.c_void_p, C.c_uint32, C.c_uint32, C.c_uint64, C.c_uint64, C.c_int, C.c_void_p]
    l.cutb_version.restype = C.c_int
    l.cutb_status_string.restype = C.c_char_p
    l.cutb_status_string.argtypes = [C.c_int]
    l.cutb_last_error.restype = C.c_char_p
    l.cutb_device_sm_count.restype = C.c_int
    for name, desc in (("cutb_dense_matmul", DenseDesc), ("cutb_residual_norm", ResidualNormDesc), ("cutb_embedding_bigram", EmbedDesc),
                       ("cutb_window_kv_write", WindowAttnDesc), ("cutb_window_attention", WindowAttnDesc),
                       ("cutb_window_attention_decode", WindowAttnDesc), ("cutb_latent_kv_write", LatentAttnDesc),
                       ("cutb_latent_attention", LatentAttnDesc), ("cutb_latent_values", LatentAttnDesc), ("cutb_latent_prefill", LatentAttnDesc),
                       ("cutb_moe_route", MoeDesc), ("cutb_moe_scatter", MoeDesc), ("cutb_moe_matmul", MoeDesc), ("cutb_expert_up", ExpertDesc),
                       ("cutb_expert_down", ExpertDesc)):
        getattr(l, name).restype = C.c_int
        getattr(l, name).argtypes = [C.POINTER(desc), C.c_void_p]
    for name, kind in (("cutb_latent_splits", C.c_uint32), ("cutb_latent_workspace_bytes", C.c_uint64), ("cutb_latent_prefill_supported", C.c_int),
                       ("cutb_latent_takes_split_queries", C.c_int)):
        getattr(l, name).restype = kind
        getattr(l, name).argtypes = [C.POINTER(LatentAttnDesc)]
    l.cutb_dense_select_variant.restype = C.c_int
    l.cutb_dense_select_variant.argtypes = [C.POINTER(DenseDesc)]
    l.cutb_dense_workspace_bytes.restype = C.c_uint64
    l.cutb_dense_workspace_bytes.argtypes = [C.POINTER(DenseDesc)]
    l.cutb_mingru_scan.restype = C.c_int
    l.cutb_mingru_scan.argtypes = [C.c_void_p, C.c_uint64, C.c_uint32, C.c_void_p, C.c_void_p, C.c_int, C.c_uint64, C.c_uint32, C.c_void_p]
    l.cutb_sequence_advance.restype = C.c_int
    l.cutb_sequence_advance.argtypes = [C.c_void_p, C.c_void_p, C.c_uint32, C.c_void_p, C.c_void_p]


def _bind_quantized(l: C.CDLL) -> None:
    l.cutb_qmatmul_workspace_bytes.restype = C.c_uint64
    l.cutb_qmatmul_workspace_bytes.argtypes = [C.POINTER(QMatmulDesc)]
    l.cutb_qmatmul_select_variant.restype = C.c_int
    l.cutb_qmatmul_select_variant.argtypes = [C.POINTER(QMatmulDesc)]
    l.cutb_qmatmul.restype = C.c_int
    l.cutb_qmatmul.argtypes = [C.POINTER(QMatmulDesc), C.c_void_p]
    l.cutb_qmatmul_decode_noalloc.restype = C.c_int
    l.cutb_qmatmul_decode_noalloc.argtypes = [C.POINTER(QMatmulDesc), C.c_void_p]
    l.cutb_qmatmul_scatter.restype = C.c_int
    l.cutb_qmatmul_scatter.argtypes = [C.POINTER(QMatmulDesc), C.POINTER(PeerScatter), C.c_void_p]
    l.cutb_peer_exchange.restype = C.c_int
    l.cutb_peer_exchange.argtypes = [C.POINTER(PeerScatter), C.c_void_p, C.c_void_p, C.c_void_p]
    l.cutb_peer_buffer_alloc.restype = C.c_int
    l.cutb_peer_buffer_alloc.argtypes = [C.c_uint64, C.POINTER(C.c_void_p), C.c_char_p]
    l.cutb_peer_buffer_open.restype = C.c_int
    l.cutb_peer_buffer_open.argtypes = [C.c_char_p, C.POINTER(C.c_void_p)]
    l.cutb_peer_buffer_close.restype = C.c_int
    l.cutb_peer_buffer_close.argtypes = [C.c_void_p]
    l.cutb_peer_buffer_free.restype = C.c_int
    l.cutb_peer_buffer_free.argtypes = [C.c_void_p]
    l.cutb_dequant.restype = C.c_int
    l.cutb_dequant.argtypes = [C.c_int, C.c_void_p, C.c_uint64, C.c_void_p, C.c_uint32, C.c_uint32, C.c_uint32,
                               C.c_void_p]
    l.cutb_embedding_blocks.restype = C.c_int
    l.cutb_embedding_blocks.argtypes = [C.c_int, C.c_void_p, C.c_void_p, C.c_void_p, C.c_uint32, C.c_uint32, C.c_uint32, C.c_uint32,
                                        C.c_void_p, C.c_void_p]
    l.cutb_requant_q8_0_blocks.restype = C.c_int
    l.cutb_requant_q8_0_blocks.argtypes = [C.c_int, C.c_void_p, C.c_uint64, C.c_void_p, C.c_uint64, C.c_uint32, C.c_void_p]
    l.cutb_rope_kv_write.restype = C.c_int
    l.cutb_rope_kv_write.argtypes = [C.c_int] + [C.c_void_p] * 9 + [C.c_uint32, C.c_uint32, C.c_uint32, C.c_uint64, C.c_uint32,
                                                                    C.c_void_p, C.c_void_p]
    l.cutb_attention_workspace_bytes.restype = C.c_uint64
    l.cutb_attention_workspace_bytes.argtypes = [C.c_uint32] * 4
    l.cutb_attention_decode.restype = C.c_int
    l.cutb_attention_decode.argtypes = [C.c_int] + [C.c_void_p] * 5 + [C.c_uint32, C.c_uint32, C.c_uint32, C.c_uint64, C.c_uint32,
                                                                       C.c_float, C.c_void_p, C.c_uint64, C.c_void_p, C.c_void_p]
    l.cutb_rope_attention_decode.restype = C.c_int
    l.cutb_rope_attention_decode.argtypes = [C.c_int] + [C.c_void_p] * 9 + [C.c_uint32, C.c_uint32, C.c_uint32, C.c_uint64, C.c_uint32,
                                                                            C.c_float, C.c_void_p, C.c_uint64, C.c_void_p, C.c_void_p]
    l.cutb_batched_kv_write.restype = C.c_int
    l.cutb_batched_kv_write.argtypes = [C.c_int, C.c_void_p, C.c_void_p, C.c_uint32, C.c_uint32] + [C.c_void_p] * 5 + [
        C.c_uint32, C.c_uint32, C.c_uint32, C.c_uint64, C.c_uint32, C.c_void_p, C.c_void_p]
    l.cutb_batched_attention.restype = C.c_int
    l.cutb_batched_attention.argtypes = [C.c_int, C.c_void_p, C.c_uint32] + [C.c_void_p] * 6 + [
        C.c_uint32, C.c_uint32, C.c_uint32, C.c_uint32, C.c_uint32, C.c_uint64, C.c_uint32, C.c_float, C.c_void_p, C.c_void_p]
    l.cutb_separate_blocks.restype = C.c_int
    l.cutb_separate_blocks.argtypes = [C.c_int, C.c_void_p, C.c_uint64, C.c_void_p, C.c_void_p, C.c_uint64, C.c_uint64, C.c_void_p]
    l.cutb_transpose_2d.restype = C.c_int
    l.cutb_transpose_2d.argtypes = [C.c_uint32, C.c_void_p, C.c_void_p, C.c_uint32, C.c_uint32, C.c_uint64, C.c_uint64, C.c_void_p]
    l.cutb_requant_q4k_affine.restype = C.c_int
    l.cutb_requant_q4k_affine.argtypes = [C.c_void_p, C.c_uint64, C.c_void_p, C.c_void_p, C.c_uint32, C.c_uint32, C.c_uint64,
                                          C.c_uint64, C.c_void_p]
    l.cutb_quantize_rows_q8_0.restype = C.c_int
    l.cutb_quantize_rows_q8_0.argtypes = [C.c_void_p, C.c_void_p, C.c_void_p, C.c_uint64, C.c_void_p]
    l.cutb_transpose_q4.restype = C.c_int
    l.cutb_transpose_q4.argtypes = [C.c_void_p, C.c_void_p, C.c_uint32, C.c_uint32, C.c_uint32, C.c_uint32,
                                    C.c_void_p]
    l.cutb_variant_name.restype = C.c_char_p
    l.cutb_variant_name.argtypes = [C.c_int]


def load(path: str) -> C.CDLL:
    """Loads libcutb.so, or the smaller libcutb_layers.so (no quantized matmul), as the library of this process."""
    global _lib
    l = C.CDLL(path)
    _bind_layers(l)
    if os.path.basename(path) == os.path.basename(LIB_PATH):
        _bind_quantized(l)
    _lib = l
    return l


def lib() -> C.CDLL:
    if _lib is None:
        if not os.path.exists(LIB_PATH):
            raise RuntimeError(
                f"{LIB_PATH} is missing: build it with `python -m cut_b200.build` (there is no CPU fallback)")
        load(LIB_PATH)
    return _lib


def check(status: int) -> None:
    if status != OK:
        raise CutbError(status, lib().cutb_last_error().decode() or lib().cutb_status_string(status).decode())
