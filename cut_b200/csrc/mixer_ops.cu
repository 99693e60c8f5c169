// Bandwidth-bound operators of the layer-list models: embedding with a hashed bigram table, the norm / residual step between
// two sublayers for a batch of tokens, the minGRU scan, and the hand-over of a sequence's {token, previous token, position}.
#include <cuda_bf16.h>

#include "common.cuh"
#include "dense_common.cuh"
#include "kernels.h"
#include "norm_stage.cuh"

namespace cutb {
namespace {

// out[i, :] = scale embed[token_i] + bigram[(prev_i * mul_prev + token_i * mul_cur) mod buckets]; a sequence's first token has no
// previous one and takes row `buckets`.  One block per token.
__global__ void __launch_bounds__(256) embedding_bigram_kernel(const cutb_embed_desc d, int vec) {
  pdl_enter();
  const uint32_t i = blockIdx.x;
  uint32_t tok = __ldg(d.tokens + i);
  uint32_t prev = i ? __ldg(d.tokens + i - 1) : (d.prev ? *d.prev : CUTB_NO_TOKEN);
  const bool bad = tok >= d.vocab || (prev != CUTB_NO_TOKEN && prev >= d.vocab);
  float *out = d.out + (size_t)i * d.ldo;
  if (bad) {  // never read outside the tables
    if (d.status && threadIdx.x == 0) atomicExch(d.status, (int)CUTB_ERR_INVALID);
    for (uint32_t c = threadIdx.x; c < d.dim; c += 256) out[c] = 0.f;
    return;
  }
  const __nv_bfloat16 *e = reinterpret_cast<const __nv_bfloat16 *>(d.embed) + (size_t)tok * d.ld_embed;
  const __nv_bfloat16 *b = nullptr;
  if (d.bigram) {
    const uint64_t row = prev == CUTB_NO_TOKEN ? d.buckets : ((uint64_t)prev * d.mul_prev + (uint64_t)tok * d.mul_cur) % d.buckets;
    b = reinterpret_cast<const __nv_bfloat16 *>(d.bigram) + row * d.ld_bigram;
  }
  if (vec) {  // eight elements at a time
    for (uint32_t c = threadIdx.x; c < d.dim / 8; c += 256) {
      const uint4 x = __ldg(reinterpret_cast<const uint4 *>(e) + c), y = b ? __ldg(reinterpret_cast<const uint4 *>(b) + c) : make_uint4(0, 0, 0, 0);
      float4 *o = reinterpret_cast<float4 *>(out) + 2 * c;
      o[0] = make_float4(fmaf(d.scale, bf16_lo(x.x), bf16_lo(y.x)), fmaf(d.scale, bf16_hi(x.x), bf16_hi(y.x)),
                         fmaf(d.scale, bf16_lo(x.y), bf16_lo(y.y)), fmaf(d.scale, bf16_hi(x.y), bf16_hi(y.y)));
      o[1] = make_float4(fmaf(d.scale, bf16_lo(x.z), bf16_lo(y.z)), fmaf(d.scale, bf16_hi(x.z), bf16_hi(y.z)),
                         fmaf(d.scale, bf16_lo(x.w), bf16_lo(y.w)), fmaf(d.scale, bf16_hi(x.w), bf16_hi(y.w)));
    }
    return;
  }
  for (uint32_t c = threadIdx.x; c < d.dim; c += 256) out[c] = fmaf(d.scale, __bfloat162float(e[c]), b ? __bfloat162float(b[c]) : 0.f);
}

// One block per row: x' = x + y_scale P(y + gathered parts), h = N(x') (norm_stage.cuh), h in bf16 or fp32.
template <int IT, bool PLAIN>  // 16-byte pieces per thread of the register path; 0: any row
__global__ void __launch_bounds__(512) residual_norm_kernel(NormStage n, uint64_t ldx, uint64_t ldy, const uint32_t *row_index, void *h,
                                                            uint64_t ldh, int h_bf16) {
  extern __shared__ __align__(16) float rn_smem[];
  pdl_enter();
  const uint32_t row = blockIdx.x, src = row_index ? __ldg(row_index + row) : row;
  n.x += src * ldx;
  if (n.y) n.y += src * ldy;
  n.part_rows += src * n.n_parts, n.part_w += src * n.n_parts;
  if (n.x_out) n.x_out += src * ldx;
  const size_t base = (size_t)row * ldh;
  auto put4 = [&](uint32_t i, float4 v) {
    if (h_bf16) *reinterpret_cast<uint2 *>(reinterpret_cast<__nv_bfloat16 *>(h) + base + i) = make_uint2(pack_bf16(v.x, v.y), pack_bf16(v.z, v.w));
    else *reinterpret_cast<float4 *>(reinterpret_cast<float *>(h) + base + i) = v;
  };
  auto put1 = [&](uint32_t i, float v) { store_out(h, h_bf16, base + i, v); };
  if constexpr (IT > 0) stage_norm_regs<IT, PLAIN>(n, rn_smem, nullptr, n.x_out != nullptr, put4);
  else stage_norm(n, rn_smem, n.x_out != nullptr, put4, put1);
}

// The recurrence over T tokens.  A block owns SC_CH channels; SC_SEG groups of threads take consecutive segments of SC_L
// tokens each, so a turn covers SC_SEG * SC_L tokens.  A segment is first reduced to the affine map s -> A s + B it applies,
// the maps meet in shared memory, and every segment is then run from its true start state.  All in fp32.
constexpr int SC_CH = 16, SC_SEG = 32, SC_L = 4, SC_THREADS = SC_CH * SC_SEG;

__global__ void __launch_bounds__(SC_THREADS, 2) mingru_scan_kernel(const float *__restrict__ zxg, uint64_t ld, uint32_t width, float *state,
                                                                    void *out, uint64_t ldo, int out_bf16, uint32_t T) {
  __shared__ float As[SC_CH][SC_SEG + 1], Bs[SC_CH][SC_SEG + 1];  // the segments' maps, then (in Bs) their start states
  pdl_enter();
  const uint32_t c = threadIdx.x % SC_CH, seg = threadIdx.x / SC_CH, ch = blockIdx.x * SC_CH + c;
  const bool live = ch < width;
  // (warp w carries the state of channel w from turn to turn)
  const uint32_t lane = threadIdx.x & 31, warp = threadIdx.x >> 5, wch = blockIdx.x * SC_CH + warp;
  static_assert(SC_SEG == 32 && SC_THREADS / 32 == SC_CH, "one warp per channel, one lane per segment");
  float carry = wch < width ? state[wch] : 0.f;
  float z1[SC_L], u1[SC_L], g1[SC_L];  // the next turn's pre-activations, in flight
  auto load = [&](uint32_t t0) {
#pragma unroll
    for (int i = 0; i < SC_L; ++i) {
      const uint32_t t = t0 + seg * SC_L + i;
      const bool in = live && t < T;
      const float *row = zxg + (size_t)t * ld + ch;
      z1[i] = in ? __ldg(row) : 0.f;
      u1[i] = in ? __ldg(row + width) : 0.f;
      g1[i] = in ? __ldg(row + 2 * (size_t)width) : 0.f;
    }
  };
  load(0);
  for (uint32_t t0 = 0; t0 < T; t0 += SC_SEG * SC_L) {
    float a[SC_L], b[SC_L], g[SC_L];
    float A = 1.f, B = 0.f;
#pragma unroll
    for (int i = 0; i < SC_L; ++i) a[i] = z1[i], b[i] = u1[i], g[i] = g1[i];
    load(t0 + SC_SEG * SC_L);
#pragma unroll
    for (int i = 0; i < SC_L; ++i) {
      const bool in = t0 + seg * SC_L + i < T;
      const float z = in ? sigmoid(a[i]) : 0.f;
      b[i] = z * mingru_candidate(b[i]);
      a[i] = 1.0f - z;
      A *= a[i];
      B = fmaf(a[i], B, b[i]);
    }
    As[c][seg] = A, Bs[c][seg] = B;
    __syncthreads();
    {  // warp w composes the maps of channel w, lane = segment
      float pa = As[warp][lane], pb = Bs[warp][lane];
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float qa = __shfl_up_sync(0xffffffffu, pa, o), qb = __shfl_up_sync(0xffffffffu, pb, o);
        if (lane >= (uint32_t)o) pb = fmaf(pa, qb, pb), pa *= qa;
      }
      const float after = fmaf(pa, carry, pb);  // state behind this lane's segment
      const float start = __shfl_up_sync(0xffffffffu, after, 1);
      Bs[warp][lane] = lane ? start : carry;
      carry = __shfl_sync(0xffffffffu, after, 31);
    }
    __syncthreads();
    float mine = Bs[c][seg];
#pragma unroll
    for (int i = 0; i < SC_L; ++i) {
      const uint32_t t = t0 + seg * SC_L + i;
      mine = fmaf(a[i], mine, b[i]);
      if (live && t < T) store_out(out, out_bf16, (size_t)t * ldo + ch, mine * silu(g[i]));
    }
  }
  if (wch < width && lane == 0) state[wch] = carry;
}

__global__ void sequence_advance_kernel(cutb_sequence_state *s, const uint32_t *tokens, uint32_t n, const float *next) {
  pdl_enter();
  s->prev = tokens ? tokens[n - 1] : s->token;
  if (next) s->token = (uint32_t)*next;
  s->pos += tokens ? n : 1;
}

}  // namespace

int embedding_bigram_launch(const cutb_embed_desc &d, cudaStream_t stream) {
  const uintptr_t bases = reinterpret_cast<uintptr_t>(d.embed) | reinterpret_cast<uintptr_t>(d.bigram) | reinterpret_cast<uintptr_t>(d.out);
  const int vec = (d.dim | d.ld_embed | d.ld_bigram | d.ldo) % 8 == 0 && bases % 16 == 0;
  CUTB_CUDA_TRY(launch_pdl(embedding_bigram_kernel, dim3(d.n), dim3(256), 0, stream, d, vec));
  return CUTB_OK;
}

int residual_norm_launch(const cutb_residual_norm_desc &d, cudaStream_t stream) {
  const NormStage n{d.x, d.y, d.post_w, d.pre_w, d.y || d.n_parts ? d.x_out : nullptr, d.dim, d.groups, d.eps, d.center, d.y_scale,
                    d.parts, d.part_rows, d.part_w, d.ld_parts, d.n_parts, d.parts_dtype == CUTB_BF16};
  const int bf16 = d.h_dtype == CUTB_BF16;
  if (norm_stage_fits(d.dim, d.groups, 512, 4)) {  // the row stays in registers
    const uint32_t small = 4 * (d.dim / 32);
    auto go = [&](auto kernel, uint32_t threads) -> cudaError_t {
      return launch_pdl(kernel, dim3(d.rows), dim3(threads), small, stream, n, d.ldx, d.ldy, d.row_index, d.h, d.ldh, bf16);
    };
    const bool plain = norm_stage_plain(n);
    const uint32_t threads = d.dim <= 1024 ? 128 : d.dim <= 2048 ? 256 : 512;
    if (d.dim <= 4096) CUTB_CUDA_TRY(plain ? go(residual_norm_kernel<2, true>, threads) : go(residual_norm_kernel<2, false>, threads));
    else CUTB_CUDA_TRY(plain ? go(residual_norm_kernel<4, true>, threads) : go(residual_norm_kernel<4, false>, threads));
    return CUTB_OK;
  }
  const uint32_t smem = 4 * norm_stage_floats(d.dim, d.groups);
  if (smem > 48 * 1024) {
    DeviceInfo di;
    if (int rc = get_device_info(&di)) return rc;
    if (smem > di.smem_optin) {
      set_last_error("residual_norm: rows of %u elements do not fit in shared memory", d.dim);
      return CUTB_ERR_UNSUPPORTED;
    }
    CUTB_CUDA_TRY(cudaFuncSetAttribute(residual_norm_kernel<0, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  }
  CUTB_CUDA_TRY(launch_pdl(residual_norm_kernel<0, false>, dim3(d.rows), dim3(256), smem, stream, n, d.ldx, d.ldy, d.row_index, d.h, d.ldh, bf16));
  return CUTB_OK;
}

int mingru_scan_launch(const float *zxg, uint64_t ld, uint32_t width, float *state, void *out, int out_dtype, uint64_t ldo, uint32_t T,
                       cudaStream_t stream) {
  CUTB_CUDA_TRY(launch_pdl(mingru_scan_kernel, dim3((width + SC_CH - 1) / SC_CH), dim3(SC_THREADS), 0, stream, zxg, ld, width, state, out,
                           ldo, (int)(out_dtype == CUTB_BF16), T));
  return CUTB_OK;
}

int sequence_advance_launch(cutb_sequence_state *s, const uint32_t *tokens, uint32_t n, const float *next, cudaStream_t stream) {
  CUTB_CUDA_TRY(launch_pdl(sequence_advance_kernel, dim3(1), dim3(1), 0, stream, s, tokens, n, next));
  return CUTB_OK;
}

}  // namespace cutb
