// extern "C" entry points of the layer operators every model uses and of the layer-list models (dense bf16 weights):
// argument validation and launch.  With the kernels behind them they also make up the smaller library that a model without
// quantized weights needs.
#include "common.cuh"
#include "kernels.h"
#include "moe_common.cuh"

namespace cutb {
const char *last_error();

namespace {

bool dtype_ok(int t) { return t == CUTB_F32 || t == CUTB_BF16; }

int check_dense(const cutb_dense_desc *d) {
  if (!d) {
    set_last_error("dense_matmul: null descriptor");
    return CUTB_ERR_INVALID;
  }
  const bool staged = d->norm_w != nullptr;
  if (!dtype_ok(d->a_dtype) || !dtype_ok(d->c_dtype)) {
    set_last_error("dense_matmul: element types are fp32 or bf16");
    return CUTB_ERR_INVALID;
  }
  if (d->M == 0 || d->K == 0 || d->N == 0 || !d->W || !d->C || (!staged && !d->A)) {
    set_last_error("dense_matmul: empty shape (M=%u K=%u N=%u) or null pointer", d->M, d->K, d->N);
    return CUTB_ERR_INVALID;
  }
  if (d->ldw % 8 || d->ldw < d->K || reinterpret_cast<uintptr_t>(d->W) % 16) {
    set_last_error("dense_matmul: weight rows must be 16-byte aligned and hold K elements (ldw=%u)", d->ldw);
    return CUTB_ERR_INVALID;
  }
  if ((!staged && d->lda < d->K) || (d->M > 1 && d->ldc < d->N)) {
    set_last_error("dense_matmul: lda (%u) < K or ldc (%u) < N", d->lda, d->ldc);
    return CUTB_ERR_INVALID;
  }
  if (!staged && reinterpret_cast<uintptr_t>(d->A) % 16) {
    set_last_error("dense_matmul: A must be 16-byte aligned");
    return CUTB_ERR_INVALID;
  }
  if (d->ldc % 8 == 0 && reinterpret_cast<uintptr_t>(d->C) % 16) {
    set_last_error("dense_matmul: C must be 16-byte aligned");
    return CUTB_ERR_INVALID;
  }
  if (staged) {
    if (d->M != 1 || !d->res_x || d->norm_groups == 0 || d->K % d->norm_groups || d->res_out == d->res_x) {
      set_last_error("dense_matmul: a staged norm needs one row, res_x (not res_out), and groups that divide K");
      return CUTB_ERR_INVALID;
    }
    for (const void *q : {(const void *)d->res_x, (const void *)d->res_y, (const void *)d->res_norm_w, (const void *)d->norm_w, (const void *)d->res_out, (const void *)d->norm_out})
      if (reinterpret_cast<uintptr_t>(q) % 16) {
        set_last_error("dense_matmul: operands of the staged norm must be 16-byte aligned");
        return CUTB_ERR_INVALID;
      }
  }
  if (d->batch > 1 && (staged || d->gru_state || d->bias || d->unary_op || d->lda < (uint64_t)(d->batch - 1) * d->a_batch + d->K ||
                       (d->M > 1 && d->ldc < (uint64_t)(d->batch - 1) * d->c_batch + d->N))) {
    set_last_error("dense_matmul: a batch of products has no bias, no elementwise op and no fused steps, and its columns lie within the rows");
    return CUTB_ERR_INVALID;
  }
  if (d->c_low && (d->M != 1 || d->c_dtype != CUTB_BF16 || d->batch < 2)) {
    set_last_error("dense_matmul: results in two terms are those of a batch for one row, in bf16");
    return CUTB_ERR_INVALID;
  }
  if (d->gru_state && (d->M != 1 || d->N % 3)) {
    set_last_error("dense_matmul: the recurrence step needs one row and three stacked matrices");
    return CUTB_ERR_INVALID;
  }
  if (d->variant < CUTB_DENSE_AUTO || d->variant > CUTB_DENSE_SIMT) {
    set_last_error("dense_matmul: unknown variant %d", d->variant);
    return CUTB_ERR_INVALID;
  }
  return CUTB_OK;
}

int dense_select(const cutb_dense_desc &d) {
  if (d.variant != CUTB_DENSE_AUTO) return d.variant;
  if (d.batch > 1) return d.M == 1 && dense_matvec_supported(d) ? CUTB_DENSE_MATVEC : CUTB_DENSE_SIMT;
  if (d.M == 1) return CUTB_DENSE_MATVEC;
  return dense_gemm_tc_supported(d) ? CUTB_DENSE_TC : CUTB_DENSE_SIMT;
}

int check_window(const cutb_window_attn_desc *d, bool write, bool read) {
  if (!d || !d->k_cache || !d->v_cache || !dtype_ok(d->kv_dtype) || (write && (!d->k || !d->v)) || (read && (!d->q || !d->out || !dtype_ok(d->out_dtype)))) {
    set_last_error("window_attention: null pointer, or an element type that is not fp32 / bf16");
    return CUTB_ERR_INVALID;
  }
  if (d->n_heads == 0 || d->n_kv_heads == 0 || d->n_heads % d->n_kv_heads || d->dim == 0 || d->vdim == 0 || d->dim > 256 || d->vdim > 256) {
    set_last_error("window_attention: n_heads must be a multiple of n_kv_heads, head sizes 1..256");
    return CUTB_ERR_INVALID;
  }
  if (d->k_head % 8 || d->v_head % 8 || d->k_head < d->dim || d->v_head < d->vdim || d->k_head > 256 || d->v_head > 256 ||
      reinterpret_cast<uintptr_t>(d->k_cache) % 32 || reinterpret_cast<uintptr_t>(d->v_cache) % 32) {
    set_last_error("window_attention: cache heads must be multiples of 8 elements that hold a head, caches 32-byte aligned");
    return CUTB_ERR_INVALID;
  }
  if (d->rot_dims % 2 || d->rot_dims > d->dim || (d->rot_dims && (!d->cos_table || !d->sin_table)) || d->max_pos == 0) {
    set_last_error("window_attention: rot_dims must be even and at most dim, with tables");
    return CUTB_ERR_INVALID;
  }
  if (d->n_tokens == 0 || d->window == 0 || d->ring_rows == 0 || d->ring_rows % 64) {
    set_last_error("window_attention: no tokens, an empty window, or ring_rows not a multiple of 64");
    return CUTB_ERR_INVALID;
  }
  // the window cannot reach further back than the positions there are
  const uint64_t need = (uint64_t)(d->window < d->max_pos ? d->window : d->max_pos) + d->n_tokens - 1;
  if (d->ring_rows < need && d->ring_rows < d->max_pos) {
    set_last_error("window_attention: %u ring rows do not hold a window of %u and %u new tokens", d->ring_rows, d->window, d->n_tokens);
    return CUTB_ERR_INVALID;
  }
  return CUTB_OK;
}
int check_latent(const cutb_latent_attn_desc *d, const char *what, bool reads) {
  if (!d || !dtype_ok(d->kv_dtype) || !dtype_ok(d->out_dtype) || d->n_heads == 0 || d->n_tokens == 0 || d->max_pos == 0) {
    set_last_error("%s: null descriptor, no heads, tokens or positions, or an element type that is not fp32 / bf16", what);
    return CUTB_ERR_INVALID;
  }
  if (d->rank == 0 || d->rank > 1024 || d->rot_dim % 2 || d->rot_dim > 1024 || d->rot_at < d->rank || d->rot_at % 8 || d->ld_cache % 8 ||
      d->ld_cache < d->rot_at + (uint64_t)(d->rot_dim + 7) / 8 * 8) {
    set_last_error("%s: rank 1..1024, rot_dim even and at most 1024, rot_at and ld_cache multiples of 8 that hold both parts", what);
    return CUTB_ERR_INVALID;
  }
  if (((reads || d->lat) && (!d->cache || reinterpret_cast<uintptr_t>(d->cache) % 32)) || (d->rot_dim && (!d->cos_table || !d->sin_table)) ||
      (d->lat && (!d->lat_norm_w || d->ld_lat < d->rank + d->rot_dim))) {
    set_last_error("%s: the cache must be 32-byte aligned; tables for the rotation, a norm weight and whole rows for the latents are needed", what);
    return CUTB_ERR_INVALID;
  }
  return CUTB_OK;
}

int check_moe(const cutb_moe_desc *d, const char *what) {
  if (!d || d->n_tokens == 0 || d->top == 0 || d->experts < d->top || d->experts > MOE_MAX_EXPERTS || (uint64_t)d->n_tokens * d->top > 0x7fffffffu) {
    set_last_error("%s: null descriptor, no tokens, or not 1 <= top <= experts <= %u", what, MOE_MAX_EXPERTS);
    return CUTB_ERR_INVALID;
  }
  return CUTB_OK;
}

int check_expert(const cutb_expert_desc *d, bool up) {
  const char *what = up ? "expert_up" : "expert_down";
  if (!d || d->top == 0 || d->experts < d->top || d->experts > MOE_MAX_EXPERTS || d->width == 0 || d->ff == 0 || !d->ids || !d->W || !d->act ||
      (up && (!d->logits || !d->x)) || (!up && !d->C)) {
    set_last_error("%s: null pointer, an empty size, or not 1 <= top <= experts <= %u", what, MOE_MAX_EXPERTS);
    return CUTB_ERR_INVALID;
  }
  if (d->ldw % 8 || d->ldw < (up ? d->width : d->ff) || reinterpret_cast<uintptr_t>(d->W) % 16 ||
      (d->Wd && (d->Nd == 0 || d->Kd == 0 || d->ldwd % 8 || d->ldwd < d->Kd || reinterpret_cast<uintptr_t>(d->Wd) % 16 || !d->xd || !d->C))) {
    set_last_error("%s: weight rows must be 16-byte aligned and hold their elements; the dense matrix needs an input and an output", what);
    return CUTB_ERR_INVALID;
  }
  if ((up && d->Wd && d->xd_norm_w && (reinterpret_cast<uintptr_t>(d->xd) | reinterpret_cast<uintptr_t>(d->xd_norm_w)) % 16) ||
      (!up && d->Wd && d->Nd != d->width)) {
    set_last_error("%s: the normed input must be 16-byte aligned; the dense matrix of expert_down has width rows", what);
    return CUTB_ERR_INVALID;
  }
  if (!expert_matvec_supported(*d, up)) {
    set_last_error("%s: the input does not fit in shared memory, or more than 64 experts per token", what);
    return CUTB_ERR_UNSUPPORTED;
  }
  return CUTB_OK;
}

// the kernels compare positions with the window in 32 bits
cutb_window_attn_desc clamp_window(const cutb_window_attn_desc *d) {
  cutb_window_attn_desc c = *d;
  if (c.window > c.max_pos) c.window = c.max_pos;
  return c;
}

}  // namespace
}  // namespace cutb

using namespace cutb;

extern "C" {

int cutb_version(void) { return CUTB_VERSION; }

const char *cutb_status_string(int status) {
  switch (status) {
    case CUTB_OK: return "ok";
    case CUTB_ERR_INVALID: return "invalid argument";
    case CUTB_ERR_UNSUPPORTED: return "unsupported request";
    case CUTB_ERR_CUDA: return "CUDA error";
    case CUTB_ERR_WORKSPACE: return "workspace missing or too small";
    case CUTB_ERR_TIMEOUT: return "device-side wait timed out";
    case CUTB_ERR_RANGE: return "activation outside the fp16 operand range";
    default: return "unknown status";
  }
}

const char *cutb_last_error(void) { return cutb::last_error(); }

int cutb_device_sm_count(void) {
  DeviceInfo di;
  if (get_device_info(&di) != CUTB_OK) return -1;
  return di.sm_count;
}

int cutb_rmsnorm(int dtype, const void *x, const void *weight, void *y, uint32_t rows, uint32_t dim, uint64_t ldx, float eps,
                 void *stream) {
  if (dtype != CUTB_F32 && dtype != CUTB_F16) {
    set_last_error("rmsnorm: dtype must be fp32 or fp16");
    return CUTB_ERR_INVALID;
  }
  if (rows == 0 || dim == 0) return CUTB_OK;
  if (!x || !weight || !y || ldx < dim) {
    set_last_error("rmsnorm: null pointer or row stride shorter than the row");
    return CUTB_ERR_INVALID;
  }
  return rmsnorm_launch(dtype, x, weight, y, rows, dim, ldx, eps, reinterpret_cast<cudaStream_t>(stream));
}

int cutb_embedding(const uint32_t *indices, const float *table, float *out, uint64_t n, uint32_t dim, uint32_t vocab, int *status,
                   void *stream) {
  if (n == 0 || dim == 0) return CUTB_OK;
  if (!indices || !table || !out || reinterpret_cast<uintptr_t>(table) % 16 || reinterpret_cast<uintptr_t>(out) % 16) {
    set_last_error("embedding: null pointer, or table / output not 16-byte aligned");
    return CUTB_ERR_INVALID;
  }
  return embedding_launch(indices, table, out, n, dim, vocab, status, reinterpret_cast<cudaStream_t>(stream));
}

int cutb_embedding_col(int format, const uint32_t *indices, const void *matrix, const void *scales, float *out, uint32_t n,
                       uint32_t dim, uint32_t vocab, uint32_t vocab_stride, uint32_t scale_stride, uint32_t out_stride, int *status,
                       void *stream) {
  if (n == 0 || dim == 0) return CUTB_OK;
  if (format != 0 && format != 1) {
    set_last_error("embedding_col: format must be 0 (fp16 matrix) or 1 (int8 values + fp16 scales)");
    return CUTB_ERR_INVALID;
  }
  if (!indices || !matrix || !out || (format == 1 && !scales)) {
    set_last_error("embedding_col: null pointer");
    return CUTB_ERR_INVALID;
  }
  if (vocab_stride < vocab || out_stride < dim || (format == 1 && scale_stride < vocab) ||
      (format == 0 && reinterpret_cast<uintptr_t>(matrix) % 2) || (format == 1 && reinterpret_cast<uintptr_t>(scales) % 2)) {
    set_last_error("embedding_col: a stride is shorter than its row, or an fp16 pointer is misaligned");
    return CUTB_ERR_INVALID;
  }
  return embedding_col_launch(format, indices, matrix, scales, out, n, dim, vocab, vocab_stride, scale_stride, out_stride, status,
                              reinterpret_cast<cudaStream_t>(stream));
}

int cutb_argreduce(int is_max, const float *values, float *out, uint32_t n, void *stream) {
  if (!out || (n && !values)) {
    set_last_error("argreduce: null pointer");
    return CUTB_ERR_INVALID;
  }
  return argreduce_launch(is_max, values, out, n, reinterpret_cast<cudaStream_t>(stream));
}

int cutb_glu_pairs(const float *in, float *out, uint32_t rows, uint32_t cols_out, uint64_t ldi, uint64_t ldo, int unary_op, void *stream) {
  if (rows == 0 || cols_out == 0) return CUTB_OK;
  if (!in || !out || ldi % 2 || ldi < 2ull * cols_out || ldo < cols_out || reinterpret_cast<uintptr_t>(in) % 8) {
    set_last_error("glu_pairs: null pointer, odd or short ldi, short ldo, or input not 8-byte aligned");
    return CUTB_ERR_INVALID;
  }
  return glu_pairs_launch(in, out, rows, cols_out, ldi, ldo, unary_op, reinterpret_cast<cudaStream_t>(stream));
}

int cutb_copy_batch(const cutb_copy_range *table, uint32_t n, uint64_t max_bytes, void *stream) {
  if (n == 0) return CUTB_OK;
  if (!table || n > 65535) {
    set_last_error("copy_batch: null table or more than 65535 ranges");
    return CUTB_ERR_INVALID;
  }
  // (the ranges themselves are read on the device: their alignment is the caller's contract)
  uint64_t blocks = (max_bytes / 16 + 2047) / 2048;  // about eight vectors per thread
  if (blocks < 1) blocks = 1;
  if (blocks > 64) blocks = 64;
  return copy_batch_launch(table, n, (uint32_t)blocks, reinterpret_cast<cudaStream_t>(stream));
}

int cutb_dense_select_variant(const cutb_dense_desc *desc) {
  if (check_dense(desc) != CUTB_OK) return -1;
  return dense_select(*desc);
}

uint64_t cutb_dense_workspace_bytes(const cutb_dense_desc *desc) {
  if (check_dense(desc) != CUTB_OK || dense_select(*desc) != CUTB_DENSE_TC) return 0;
  return dense_gemm_tc_workspace(*desc);
}

int cutb_dense_matmul(const cutb_dense_desc *desc, void *stream) {
  if (int rc = check_dense(desc)) return rc;
  const int v = dense_select(*desc);
  if (v != CUTB_DENSE_MATVEC && (desc->norm_w || desc->gru_state)) {
    set_last_error("dense_matmul: the staged norm and the recurrence step exist in the mat-vec only");
    return CUTB_ERR_UNSUPPORTED;
  }
  if ((v == CUTB_DENSE_MATVEC && !dense_matvec_supported(*desc)) || (v == CUTB_DENSE_TC && !dense_gemm_tc_supported(*desc))) {
    set_last_error("dense_matmul: variant %d does not cover this shape", v);
    return CUTB_ERR_UNSUPPORTED;
  }
  cudaStream_t s = reinterpret_cast<cudaStream_t>(stream);
  if (v == CUTB_DENSE_MATVEC) return dense_matvec_launch(*desc, s);
  return v == CUTB_DENSE_TC ? dense_gemm_tc_launch(*desc, s) : dense_gemm_simt_launch(*desc, s);
}

int cutb_residual_norm(const cutb_residual_norm_desc *d, void *stream) {
  if (!d || !d->x || !d->pre_w || !d->h || !dtype_ok(d->h_dtype) ||
      (d->n_parts && (!d->parts || !d->part_rows || !d->part_w || !dtype_ok(d->parts_dtype) || d->ld_parts % 4 || d->ld_parts < d->dim ||
                      reinterpret_cast<uintptr_t>(d->parts) % 16))) {
    set_last_error("residual_norm: null pointer, an element type that is not fp32 / bf16, or parts that are not 16-byte aligned rows");
    return CUTB_ERR_INVALID;
  }
  if (d->rows == 0) return CUTB_OK;
  if (d->dim == 0 || d->groups == 0 || d->dim % d->groups || d->ldx % 4 || d->ldy % 4 || d->ldh % 4 || d->ldx < d->dim || d->ldh < d->dim ||
      (d->y && d->ldy < d->dim)) {
    set_last_error("residual_norm: groups must divide dim, row strides hold dim elements and be multiples of 4");
    return CUTB_ERR_INVALID;
  }
  for (const void *q : {(const void *)d->x, (const void *)d->y, (const void *)d->post_w, (const void *)d->pre_w, (const void *)d->x_out, (const void *)d->h})
    if (reinterpret_cast<uintptr_t>(q) % 16) {
      set_last_error("residual_norm: operands must be 16-byte aligned");
      return CUTB_ERR_INVALID;
    }
  return residual_norm_launch(*d, reinterpret_cast<cudaStream_t>(stream));
}

int cutb_embedding_bigram(const cutb_embed_desc *d, void *stream) {
  if (!d || !d->tokens || !d->embed || !d->out || d->dim == 0 || d->vocab == 0 || d->ld_embed < d->dim || d->ldo < d->dim ||
      (d->bigram && (d->buckets == 0 || d->ld_bigram < d->dim))) {
    set_last_error("embedding_bigram: null pointer, empty table or a row stride shorter than the row");
    return CUTB_ERR_INVALID;
  }
  if (d->n == 0) return CUTB_OK;
  return embedding_bigram_launch(*d, reinterpret_cast<cudaStream_t>(stream));
}

int cutb_mingru_scan(const float *zxg, uint64_t ld, uint32_t width, float *state, void *out, int out_dtype, uint64_t ldo, uint32_t T,
                     void *stream) {
  if (!zxg || !state || !out || !dtype_ok(out_dtype) || ld < 3ull * width || ldo < width) {
    set_last_error("mingru_scan: null pointer, an element type that is not fp32 / bf16, or a short row stride");
    return CUTB_ERR_INVALID;
  }
  if (width == 0 || T == 0) return CUTB_OK;
  return mingru_scan_launch(zxg, ld, width, state, out, out_dtype, ldo, T, reinterpret_cast<cudaStream_t>(stream));
}

int cutb_sequence_advance(cutb_sequence_state *state, const uint32_t *tokens, uint32_t n, const float *next, void *stream) {
  if (!state || (tokens && n == 0)) {
    set_last_error("sequence_advance: null state, or no tokens");
    return CUTB_ERR_INVALID;
  }
  return sequence_advance_launch(state, tokens, n, next, reinterpret_cast<cudaStream_t>(stream));
}

int cutb_window_kv_write(const cutb_window_attn_desc *d, void *stream) {
  if (int rc = check_window(d, true, false)) return rc;
  return window_kv_write_launch(clamp_window(d), reinterpret_cast<cudaStream_t>(stream));
}

int cutb_window_attention(const cutb_window_attn_desc *d, void *stream) {
  if (int rc = check_window(d, false, true)) return rc;
  return window_attention_launch(clamp_window(d), reinterpret_cast<cudaStream_t>(stream));
}

int cutb_window_attention_decode(const cutb_window_attn_desc *d, void *stream) {
  if (int rc = check_window(d, true, true)) return rc;
  if (d->n_tokens != 1) {
    set_last_error("window_attention_decode: one token per call");
    return CUTB_ERR_INVALID;
  }
  return window_attention_decode_launch(clamp_window(d), reinterpret_cast<cudaStream_t>(stream));
}

int cutb_latent_kv_write(const cutb_latent_attn_desc *d, void *stream) {
  if (int rc = check_latent(d, "latent_kv_write", false)) return rc;
  if ((!d->lat && !d->cq) || (d->cq && (!d->cq_norm_w || !d->cq_out || d->q_rank == 0 || d->ld_cq < d->q_rank || d->ld_cq_out < d->q_rank))) {
    set_last_error("latent_kv_write: nothing to do, or no norm weight, output or whole rows for the latent queries");
    return CUTB_ERR_INVALID;
  }
  return latent_kv_write_launch(*d, reinterpret_cast<cudaStream_t>(stream));
}

uint32_t cutb_latent_splits(const cutb_latent_attn_desc *d) { return check_latent(d, "latent_splits", false) == CUTB_OK ? latent_splits(*d) : 0; }

int cutb_latent_takes_split_queries(const cutb_latent_attn_desc *d) {
  return check_latent(d, "latent_takes_split_queries", false) == CUTB_OK && latent_takes_split_queries(*d) ? 1 : 0;
}

uint64_t cutb_latent_workspace_bytes(const cutb_latent_attn_desc *d) {
  if (check_latent(d, "latent_workspace", false) != CUTB_OK || d->n_tokens != 1) return 0;
  const uint64_t n = (uint64_t)d->n_heads * latent_splits(*d);
  return ((2 * n + 3) / 4 * 4 + n * ((d->rank + 3) / 4 * 4)) * sizeof(float);
}

int cutb_latent_attention(const cutb_latent_attn_desc *d, void *stream) {
  if (int rc = check_latent(d, "latent_attention", true)) return rc;
  if (d->qa_high && (!d->qa_low || !latent_takes_split_queries(*d) || d->ld_qa_split % 8 || d->ld_qa_split < d->rank ||
                     (reinterpret_cast<uintptr_t>(d->qa_high) | reinterpret_cast<uintptr_t>(d->qa_low)) % 16)) {
    set_last_error("latent_attention: queries in two terms need one token, a bf16 cache and 16-byte aligned rows");
    return CUTB_ERR_INVALID;
  }
  if (!d->q || (!d->qa && !d->qa_high) || (d->lat && d->n_tokens != 1) || (d->n_tokens != 1 && (!d->out || d->ldo < (uint64_t)d->n_heads * d->rank)) ||
      (d->n_tokens > 1 && (d->ldq < (uint64_t)d->n_heads * (d->dim + d->rot_dim) || d->ld_qa < (uint64_t)d->n_heads * d->rank))) {
    set_last_error("latent_attention: null pointer, short rows, or a cache row to make for more than one token");
    return CUTB_ERR_INVALID;
  }
  if (d->n_tokens > 65535) {
    set_last_error("latent_attention: at most 65535 tokens per call");
    return CUTB_ERR_UNSUPPORTED;
  }
  if (d->n_tokens == 1 && (!d->workspace || d->workspace_bytes < cutb_latent_workspace_bytes(d) || reinterpret_cast<uintptr_t>(d->workspace) % 16)) {
    set_last_error("latent_attention: one token needs a workspace of cutb_latent_workspace_bytes(), 16-byte aligned");
    return CUTB_ERR_WORKSPACE;
  }
  return latent_attention_launch(*d, reinterpret_cast<cudaStream_t>(stream));
}

int cutb_latent_values(const cutb_latent_attn_desc *d, void *stream) {
  if (int rc = check_latent(d, "latent_values", false)) return rc;
  if (d->n_tokens != 1 || d->vdim == 0 || !d->w_uv || d->ld_uv % 8 || d->ld_uv < d->rank || reinterpret_cast<uintptr_t>(d->w_uv) % 16 || !d->out ||
      !d->workspace || d->workspace_bytes < cutb_latent_workspace_bytes(d)) {
    set_last_error("latent_values: one token, its workspace, and 16-byte aligned rows of W_uv are needed");
    return CUTB_ERR_INVALID;
  }
  return latent_values_launch(*d, reinterpret_cast<cudaStream_t>(stream));
}

int cutb_latent_prefill_supported(const cutb_latent_attn_desc *d) { return d && latent_prefill_supported(*d) ? 1 : 0; }

int cutb_latent_prefill(const cutb_latent_attn_desc *d, void *stream) {
  if (int rc = check_latent(d, "latent_prefill", true)) return rc;
  const uint64_t H = d->n_heads;
  if (!d->q || !d->k_exp || !d->v_exp || !d->out || d->ldq < H * (d->dim + d->rot_dim) || d->ld_k < H * d->dim || d->ld_v < H * d->vdim ||
      d->ldo < H * d->vdim || d->ld_k % 8 || d->ld_v % 8 ||
      (reinterpret_cast<uintptr_t>(d->k_exp) | reinterpret_cast<uintptr_t>(d->v_exp)) % 16) {
    set_last_error("latent_prefill: null pointer, short rows, or keys and values that are not 16-byte aligned");
    return CUTB_ERR_INVALID;
  }
  if (!latent_prefill_supported(*d)) {
    set_last_error("latent_prefill: bf16, head parts that are multiples of 8, dim + rot_dim <= 256 and vdim <= 256");
    return CUTB_ERR_UNSUPPORTED;
  }
  return latent_prefill_launch(*d, reinterpret_cast<cudaStream_t>(stream));
}

int cutb_moe_route(const cutb_moe_desc *d, void *stream) {
  if (int rc = check_moe(d, "moe_route")) return rc;
  if (!d->logits || !d->weights || !d->ids || !d->slots || !d->offsets || d->ld_logits < d->experts) {
    set_last_error("moe_route: null pointer, or short rows of logits");
    return CUTB_ERR_INVALID;
  }
  return moe_route_launch(*d, reinterpret_cast<cudaStream_t>(stream));
}

int cutb_moe_scatter(const cutb_moe_desc *d, void *stream) {
  if (int rc = check_moe(d, "moe_scatter")) return rc;
  if (!d->A || !d->C || !d->slots || !dtype_ok(d->a_dtype) || d->c_dtype != d->a_dtype || d->K == 0 || d->lda < d->K || d->ldc < d->K) {
    set_last_error("moe_scatter: null pointer, short rows, or different element types");
    return CUTB_ERR_INVALID;
  }
  return moe_scatter_launch(*d, reinterpret_cast<cudaStream_t>(stream));
}

int cutb_moe_matmul(const cutb_moe_desc *d, void *stream) {
  if (int rc = check_moe(d, "moe_matmul")) return rc;
  const uint32_t cols = d->glu ? d->N / 2 : d->N;
  if (!d->A || !d->W || !d->C || !d->offsets || !dtype_ok(d->a_dtype) || !dtype_ok(d->c_dtype) || d->K == 0 || d->N == 0 || d->lda < d->K ||
      d->ldc < cols || (d->glu && d->N % 2) || d->glu < CUTB_GLU_NONE || d->glu > CUTB_GLU_CLAMPED) {
    set_last_error("moe_matmul: null pointer, short rows, an unknown element type or gated unit, or an odd number of paired rows");
    return CUTB_ERR_INVALID;
  }
  if (d->ldw % 8 || d->ldw < d->K || reinterpret_cast<uintptr_t>(d->W) % 16 || reinterpret_cast<uintptr_t>(d->A) % 16 ||
      (d->ldc % 8 == 0 && reinterpret_cast<uintptr_t>(d->C) % 16)) {
    set_last_error("moe_matmul: A, C and the weight rows must be 16-byte aligned and hold K elements (ldw=%u)", d->ldw);
    return CUTB_ERR_INVALID;
  }
  if (d->variant == CUTB_DENSE_TC) {
    if (d->a_dtype != CUTB_BF16 || d->lda % 8) {
      set_last_error("moe_matmul: the tensor cores read bf16 rows, 16-byte aligned");
      return CUTB_ERR_UNSUPPORTED;
    }
    return moe_gemm_tc_launch(*d, reinterpret_cast<cudaStream_t>(stream));
  }
  if (d->variant != CUTB_DENSE_SIMT) {
    set_last_error("moe_matmul: unknown variant %d", d->variant);
    return CUTB_ERR_INVALID;
  }
  return moe_gemm_simt_launch(*d, reinterpret_cast<cudaStream_t>(stream));
}

int cutb_expert_up(const cutb_expert_desc *d, void *stream) {
  if (int rc = check_expert(d, true)) return rc;
  return expert_up_launch(*d, reinterpret_cast<cudaStream_t>(stream));
}

int cutb_expert_down(const cutb_expert_desc *d, void *stream) {
  if (int rc = check_expert(d, false)) return rc;
  return expert_down_launch(*d, reinterpret_cast<cudaStream_t>(stream));
}

}  // extern "C"
