// Decode mat-vec over dense bf16 weights: C[N] = act(W[N, K] x + bias) for one activation row, fp32 throughout besides the
// weights themselves (a bf16 weight times an fp32 activation, fp32 accumulation).
//
// HBM-bound: every weight is read once.  One block per SM, up to 28 warps; a tile is R rows (one or two, or the three rows
// z / x / g of one recurrence channel) and belongs to one warp, tiles are dealt round-robin over the SMs first and the warps of
// an SM second, so all SMs stream the same number of rows.  A lane takes every 32nd 16-byte piece of a row; the pieces of the
// next step (also of the next tile) are in flight while the current ones are used.  The first two steps' loads are issued
// before the wait for the previous kernel (weights are constants of the model), so under programmatic launch the stream starts
// while the predecessor still finishes.  The activation row lies in two planes of shared memory (elements 8 i .. 8 i + 3 and
// 8 i + 4 .. 8 i + 7), so the 16-byte reads of a warp fall on distinct banks.
//
// Fused steps:
//  * input: the row is either given (fp32 or bf16), or made here from the residual stream and the previous sublayer's output
//    (post-norm, residual add, pre-norm: norm_stage.cuh); block 0 writes the new residual row.  The norm weights are
//    prefetched before the wait;
//  * output: bias and one elementwise op, or the gated recurrence  s = (1 - z) s + z c  of one token with its state update
//    and output gate (rows z, x, g of channel j are rows j, width + j, 2 width + j of the stacked weight).
//
// head_matvec_kernel: the same for a batch of small products, a matrix and a slice of the row per head (latent attention's
// W_uk^T q and W_uv o).  4 .. 32 lanes share a row by its length, a block takes consecutive rows and stages the slices of their
// heads only.  A slice may be made here from the partial sums that the blocks of an attention left (each with its maximum and
// weight sum).
#include <cuda_bf16.h>

#include "common.cuh"
#include "dense_common.cuh"
#include "kernels.h"
#include "norm_stage.cuh"

namespace cutb {
namespace {

constexpr int MV_MIN_WARPS = 16, MV_MAX_WARPS = 28, MV_MAX_THREADS = 32 * MV_MAX_WARPS;

struct MvParams {
  const void *A;
  const __nv_bfloat16 *W;
  const float *bias;
  void *C;
  float *state;  // recurrence
  uint32_t K, K8, N, ldw8;
  uint32_t ntiles;   // row tiles
  uint32_t row_step; // distance of a tile's rows (1, or width for the recurrence)
  int a_bf16, c_bf16, unary;
  NormStage norm;  // norm.pre_w != null: the input is staged from the residual stream
  float *norm_out;
};

__device__ __forceinline__ void cp_async16(uint32_t dst, const void *src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
template <int R, int UNR, bool GRU, bool PLAIN>
__global__ void __launch_bounds__(MV_MAX_THREADS, 1) dense_matvec_kernel(const MvParams p) {
  extern __shared__ __align__(16) float mv_smem[];
  float4 *lo = reinterpret_cast<float4 *>(mv_smem), *hi = lo + p.K8;  // activation planes
  float *stage = mv_smem + 8 * p.K8;                                  // norm staging rows
  const uint32_t tid = threadIdx.x, nt = blockDim.x, lane = tid & 31, warp = tid >> 5;
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");

  const uint4 *W4 = reinterpret_cast<const uint4 *>(p.W);
  const uint32_t tstep = gridDim.x * (nt >> 5), first = warp * gridDim.x + blockIdx.x;
  // step = UNR pieces of every row of a tile; the load cursor runs ahead of the compute cursor
  uint32_t l_tile = first, l_k = lane;
  auto load = [&](uint4 (&w)[UNR][R]) {
#pragma unroll
    for (int u = 0; u < UNR; ++u)
#pragma unroll
      for (int r = 0; r < R; ++r) {
        const uint32_t row = GRU ? l_tile + (uint32_t)r * p.row_step : l_tile * R + (uint32_t)r, k = l_k + 32 * u;
        w[u][r] = l_tile < p.ntiles && row < p.N && k < p.K8 ? ld_stream(W4 + (size_t)row * p.ldw8 + k) : make_uint4(0, 0, 0, 0);
      }
    l_k += 32 * UNR;
    if (l_k >= p.K8 + lane) l_k = lane, l_tile += tstep;  // (the same step in every lane)
  };
  uint4 wa[UNR][R], wb[UNR][R];
  load(wa);
  load(wb);
  if (R == 2 && lane < R) {
    // many rows: the rest of the first tile starts towards L2, so that the stream does not pause while the input is staged
    // (32000 x 4096: 43.4 -> 39.9 us; with fewer rows or long ones it only gets in the way of the loads)
    const uint32_t row = first * R + lane;
    if (first < p.ntiles && row < p.N)
      asm volatile("cp.async.bulk.prefetch.L2.global [%0], %1;" ::"l"(W4 + (size_t)row * p.ldw8), "r"(p.K8 * 16u) : "memory");
  }
  const bool fast_norm = p.norm.pre_w && norm_stage_fits(p.K, p.norm.groups, nt, 2);
  if (fast_norm) {  // the norm weights are constants too: on their way to shared memory before the wait
    for (uint32_t i = tid; i < p.K / 4; i += nt) {
      if (p.norm.post_w) cp_async16(smem_u32(stage + 4 * i), p.norm.post_w + 4 * i);
      cp_async16(smem_u32(stage + p.K + 4 * i), p.norm.pre_w + 4 * i);
    }
  }
  asm volatile("griddepcontrol.wait;" ::: "memory");

  // ---- the activation row -> two planes, zero past K ----
  auto put1 = [&](uint32_t i, float v) { mv_smem[(i & 4 ? 4 * p.K8 : 0) + (i >> 3) * 4 + (i & 3)] = v; };
  auto put4 = [&](uint32_t i, float4 v) { (i & 4 ? hi : lo)[i >> 3] = v; };
  float *keep = !GRU && blockIdx.x == 0 ? p.norm_out : nullptr;
  auto norm1 = [&](uint32_t i, float v) {
    put1(i, v);
    if (!GRU && keep) keep[i] = v;
  };
  auto norm4 = [&](uint32_t i, float4 v) {
    put4(i, v);
    if (!GRU && keep) *reinterpret_cast<float4 *>(keep + i) = v;
  };
  for (uint32_t i = p.K + tid; i < 8 * p.K8; i += nt) put1(i, 0.f);
  if (fast_norm) {
    stage_norm_regs<2, PLAIN>(p.norm, stage + 2 * p.K, stage, blockIdx.x == 0 && p.norm.x_out != nullptr, norm4);
  } else if (p.norm.pre_w) {
    stage_norm(p.norm, stage, blockIdx.x == 0 && p.norm.x_out != nullptr, norm4, norm1);
  } else if (p.a_bf16) {
    const __nv_bfloat16 *a = reinterpret_cast<const __nv_bfloat16 *>(p.A);
    for (uint32_t i = tid; i < p.K; i += nt) put1(i, __bfloat162float(a[i]));
  } else {
    const float *a = reinterpret_cast<const float *>(p.A);
    const uint32_t k4 = p.K / 4;
#pragma unroll 4
    for (uint32_t i = tid; i < k4; i += nt) put4(4 * i, reinterpret_cast<const float4 *>(a)[i]);
    for (uint32_t i = 4 * k4 + tid; i < p.K; i += nt) put1(i, a[i]);
  }
  __syncthreads();

  uint32_t tile = first, k = lane;
  float acc[R];
#pragma unroll
  for (int r = 0; r < R; ++r) acc[r] = 0.f;
  // bias and state of the tile in work, on their way while it streams
  float bias = 0.f, state = 0.f;
  auto constants = [&]() {
    const uint32_t row = GRU ? tile + lane * p.row_step : tile * R + lane;
    if (lane < R && tile < p.ntiles && row < p.N) {
      if (p.bias) bias = __ldg(p.bias + row);
      if (GRU && lane == 0) state = p.state[tile];
    }
  };
  constants();
  auto use = [&](const uint4 (&w)[UNR][R]) {
#pragma unroll
    for (int u = 0; u < UNR; ++u)
      if (k + 32 * u < p.K8) {
        const float4 a = lo[k + 32 * u], b = hi[k + 32 * u];
#pragma unroll
        for (int r = 0; r < R; ++r) fma8(acc[r], w[u][r], a, b);
      }
    k += 32 * UNR;
    if (k < p.K8 + lane) return;
    // the tile's last piece
    float sum = 0.f;
#pragma unroll
    for (int r = 0; r < R; ++r) {
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) acc[r] += __shfl_xor_sync(0xffffffffu, acc[r], o);
      if (lane == (uint32_t)r) sum = acc[r];
      acc[r] = 0.f;
    }
    sum += bias;
    if constexpr (GRU) {
      const float z = __shfl_sync(0xffffffffu, sum, 0), u = __shfl_sync(0xffffffffu, sum, 1), g = __shfl_sync(0xffffffffu, sum, 2);
      if (lane == 0) {
        const float s = mingru_update(state, z, u);
        p.state[tile] = s;
        store_out(p.C, p.c_bf16, tile, s * silu(g));
      }
    } else {
      const uint32_t row = tile * R + lane;
      if (lane < R && row < p.N) store_out(p.C, p.c_bf16, row, dense_unary(sum, p.unary));
    }
    k = lane, tile += tstep;
    constants();
  };
  while (tile < p.ntiles) {
    use(wa);
    load(wa);
    if (tile >= p.ntiles) break;
    use(wb);
    load(wb);
  }
}

template <int R, int UNR, bool GRU, bool PLAIN> int mv_launch(MvParams &p, uint32_t smem, uint32_t sms, bool overlap, cudaStream_t stream) {
  static bool configured[64] = {};
  int dev = 0;
  CUTB_CUDA_TRY(cudaGetDevice(&dev));
  if (dev < 0 || dev >= 64 || !configured[dev]) {
    DeviceInfo di;
    if (int rc = get_device_info(&di)) return rc;
    CUTB_CUDA_TRY(cudaFuncSetAttribute(dense_matvec_kernel<R, UNR, GRU, PLAIN>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)di.smem_optin - 2048));
    if (dev >= 0 && dev < 64) configured[dev] = true;
  }
  const uint32_t per_sm = (p.ntiles + sms - 1) / sms, turns = (per_sm + MV_MAX_WARPS - 1) / MV_MAX_WARPS;
  uint32_t warps = (per_sm + turns - 1) / turns;
  if (warps < MV_MIN_WARPS) warps = MV_MIN_WARPS;  // (the staging of the input wants threads too)
  const dim3 grid(p.ntiles < sms ? p.ntiles : sms), block(32 * warps);
  if (overlap) {
    CUTB_CUDA_TRY(launch_pdl(dense_matvec_kernel<R, UNR, GRU, PLAIN>, grid, block, smem, stream, p));
  } else {
    dense_matvec_kernel<R, UNR, GRU, PLAIN><<<grid, block, smem, stream>>>(p);
    CUTB_CUDA_TRY(cudaGetLastError());
  }
  return CUTB_OK;
}

// ---- a product per head ------------------------------------------------------------------------------------------------
constexpr int HV_THREADS = 256;

template <int LPR> __global__ void __launch_bounds__(HV_THREADS) head_matvec_kernel(const HeadMvParams p, uint32_t rows_per_block) {
  extern __shared__ __align__(16) float hv_smem[];
  __shared__ float share[64];
  constexpr uint32_t RPW = 32 / LPR, PASS = HV_THREADS / 32 * RPW;  // rows of a warp and of the block at a time
  constexpr int U = 4;
  const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, sub = lane % LPR;
  const uint32_t total = p.batch * p.N, r0 = blockIdx.x * rows_per_block, r1 = min(r0 + rows_per_block, total);
  const uint32_t h0 = r0 / p.N, nh = (r1 - 1) / p.N - h0 + 1, K8 = p.K8, plane = nh * K8;
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  float4 *lo = reinterpret_cast<float4 *>(hv_smem), *hi = lo + plane;
  const uint4 *W4 = reinterpret_cast<const uint4 *>(p.W);
  // the first row's weights are on their way before the wait for the previous kernel
  uint4 w[U];
  auto load = [&](uint32_t row, uint32_t k) {
#pragma unroll
    for (int u = 0; u < U; ++u) w[u] = row < r1 && k + LPR * u < K8 ? ld_stream(W4 + (size_t)row * p.ldw8 + k + LPR * u) : make_uint4(0, 0, 0, 0);
  };
  const uint32_t first = r0 + warp * RPW + lane / LPR;
  load(first, sub);
  pdl_enter();
  auto put = [&](uint32_t h, uint32_t k, float v) { hv_smem[(k & 4 ? 4 * plane : 0) + (h * K8 + (k >> 3)) * 4 + (k & 3)] = v; };
  for (uint32_t h = 0; h < nh; ++h) {
    if (p.splits) {
      const float2 *ml = p.ml + (size_t)(h0 + h) * p.splits;
      const float *part = p.part + (size_t)(h0 + h) * p.splits * p.ld_part;
      float a[2][16];  // the first ones are on their way while their shares are worked out
#pragma unroll
      for (uint32_t i = 0; i < 2; ++i)
#pragma unroll
        for (uint32_t s = 0; s < 16; ++s) {
          const uint32_t k = tid + i * HV_THREADS;
          a[i][s] = k < p.K && s < p.splits ? part[(size_t)s * p.ld_part + k] : 0.f;
        }
      if (warp == 0) {  // a partial sum's share: exp2(its maximum - the largest) / the whole weight sum
        const float2 a = lane < p.splits ? ml[lane] : make_float2(-1e30f, 0.f), b = lane + 32 < p.splits ? ml[lane + 32] : make_float2(-1e30f, 0.f);
        float m = fmaxf(a.x, b.x);
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
        const float wa = exp2f(a.x - m), wb = exp2f(b.x - m);
        const float inv = 1.0f / warp_sum(wa * a.y + wb * b.y);
        share[lane] = wa * inv, share[lane + 32] = wb * inv;
      }
      __syncthreads();
#pragma unroll
      for (uint32_t i = 0; i < 2; ++i) {
        const uint32_t k = tid + i * HV_THREADS;
        float v = 0.f;
#pragma unroll
        for (uint32_t s = 0; s < 16; ++s) v = fmaf(share[s], a[i][s], v);
        for (uint32_t s = 16; s < p.splits && k < p.K; ++s) v = fmaf(share[s], part[(size_t)s * p.ld_part + k], v);
        if (k < 8 * K8) put(h, k, v);
      }
      for (uint32_t k = tid + 2 * HV_THREADS; k < 8 * K8; k += HV_THREADS) {
        float v = 0.f;
        for (uint32_t s = 0; s < p.splits && k < p.K; ++s) v = fmaf(share[s], part[(size_t)s * p.ld_part + k], v);
        put(h, k, v);
      }
      __syncthreads();
    } else {
      const float *x = p.x + (size_t)(h0 + h) * p.x_batch;
      for (uint32_t k = tid; k < 8 * K8; k += HV_THREADS) put(h, k, k < p.K ? x[k] : 0.f);
    }
  }
  __syncthreads();
  for (uint32_t row = first; row - lane / LPR < r1; row += PASS) {  // (the same number of turns in every lane)
    const uint32_t h = min(row, r1 - 1) / p.N - h0;
    const float4 *xl = lo + h * K8, *xh = hi + h * K8;
    float acc = 0.f;
    for (uint32_t k = sub; k < K8 + sub; k += LPR * U) {
      if (!(row == first && k == sub)) load(row, k);
#pragma unroll
      for (int u = 0; u < U; ++u)
        if (k + LPR * u < K8) fma8(acc, w[u], xl[k + LPR * u], xh[k + LPR * u]);
    }
#pragma unroll
    for (int o = LPR / 2; o > 0; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
    if (sub == 0 && row < r1) {
      const size_t at = (size_t)(row / p.N) * p.c_batch + row % p.N;
      if (p.c_low) {
        acc *= p.scale;
        const __nv_bfloat16 high = __float2bfloat16_rn(acc);
        reinterpret_cast<__nv_bfloat16 *>(p.C)[at] = high;
        reinterpret_cast<__nv_bfloat16 *>(p.c_low)[at] = __float2bfloat16_rn(acc - __bfloat162float(high));
      } else {
        store_out(p.C, p.c_bf16, at, acc);
      }
    }
  }
}

template <int LPR> int hv_launch(const HeadMvParams &p, uint32_t sms, cudaStream_t stream) {
  constexpr uint32_t PASS = HV_THREADS / 32 * (32 / LPR);
  const uint32_t total = p.batch * p.N;
  uint32_t rows = (total + 2 * sms - 1) / (2 * sms);
  rows = (rows + PASS - 1) / PASS * PASS;
  auto smem_of = [&](uint32_t r) { return 32 * p.K8 * (r / p.N + 2 < p.batch ? r / p.N + 2 : p.batch); };
  while (rows > PASS && smem_of(rows) > 96 * 1024) rows -= PASS;
  const uint32_t smem = smem_of(rows);
  if (smem > 200 * 1024) {
    set_last_error("head mat-vec: the slices of %u rows of %u elements do not fit in shared memory", rows, p.K);
    return CUTB_ERR_UNSUPPORTED;
  }
  if (smem > 48 * 1024) CUTB_CUDA_TRY(cudaFuncSetAttribute(head_matvec_kernel<LPR>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  CUTB_CUDA_TRY(launch_pdl(head_matvec_kernel<LPR>, dim3((total + rows - 1) / rows), dim3(HV_THREADS), smem, stream, p, rows));
  return CUTB_OK;
}

uint32_t mv_smem_bytes(const cutb_dense_desc &d) {
  const uint32_t K8 = (d.K + 7) / 8;
  return 4 * (8 * K8 + (d.norm_w ? norm_stage_floats(d.K, d.norm_groups) : 0));
}

}  // namespace

bool dense_matvec_supported(const cutb_dense_desc &d) {
  if (d.batch > 1) return d.M == 1 && d.a_dtype == CUTB_F32 && !d.bias && !d.unary_op;
  return d.M == 1 && mv_smem_bytes(d) <= 220 * 1024;
}

int head_matvec_launch(const HeadMvParams &p, cudaStream_t stream) {
  DeviceInfo di;
  if (int rc = get_device_info(&di)) return rc;
  const uint32_t sms = (uint32_t)di.sm_count;
  // about four 16-byte pieces per lane
  if (p.K8 <= 16) return hv_launch<4>(p, sms, stream);
  if (p.K8 <= 32) return hv_launch<8>(p, sms, stream);
  if (p.K8 <= 64) return hv_launch<16>(p, sms, stream);
  return hv_launch<32>(p, sms, stream);
}

int dense_matvec_launch(const cutb_dense_desc &d, cudaStream_t stream) {
  DeviceInfo di;
  if (int rc = get_device_info(&di)) return rc;
  if (d.batch > 1) {
    HeadMvParams h{};
    h.x = reinterpret_cast<const float *>(d.A), h.x_batch = d.a_batch, h.W = d.W, h.C = d.C, h.c_bf16 = d.c_dtype == CUTB_BF16;
    h.c_low = d.c_low, h.scale = d.c_scale;
    h.batch = d.batch, h.K = d.K, h.K8 = (d.K + 7) / 8, h.N = d.N, h.ldw8 = d.ldw / 8, h.c_batch = d.c_batch;
    return head_matvec_launch(h, stream);
  }
  MvParams p{};
  p.A = d.A, p.W = reinterpret_cast<const __nv_bfloat16 *>(d.W), p.bias = d.bias, p.C = d.C, p.state = d.gru_state;
  p.K = d.K, p.K8 = (d.K + 7) / 8, p.N = d.N, p.ldw8 = d.ldw / 8;
  p.a_bf16 = d.a_dtype == CUTB_BF16, p.c_bf16 = d.c_dtype == CUTB_BF16, p.unary = d.unary_op;
  p.norm = NormStage{d.res_x, d.res_y, d.res_norm_w, d.norm_w, d.res_out, d.K, d.norm_groups ? d.norm_groups : 1, d.norm_eps, d.norm_center, d.res_scale};
  p.norm_out = d.norm_out;
  const bool gru = d.gru_state != nullptr;
  const uint32_t sms = (uint32_t)di.sm_count;
  const uint32_t sms_all = sms * MV_MAX_WARPS;
  const bool two = !gru && d.N >= 2 * sms_all;  // enough rows: two per warp share the activation reads
  p.row_step = gru ? d.N / 3 : 1;
  p.ntiles = gru ? d.N / 3 : (two ? (d.N + 1) / 2 : d.N);
  const uint32_t smem = mv_smem_bytes(d);
  const bool overlap = !(d.flags & CUTB_FLAG_NO_OVERLAP);
  if (gru && (!norm_stage_plain(p.norm) || p.norm_out)) {
    set_last_error("dense_matvec: the recurrence step behind a layer norm or a plain residual, or with the normed row kept, is not built");
    return CUTB_ERR_UNSUPPORTED;
  }
  if (!norm_stage_plain(p.norm))
    return two ? mv_launch<2, 2, false, false>(p, smem, sms, overlap, stream) : mv_launch<1, 4, false, false>(p, smem, sms, overlap, stream);
  if (gru) return mv_launch<3, 1, true, true>(p, smem, sms, overlap, stream);
  return two ? mv_launch<2, 2, false, true>(p, smem, sms, overlap, stream) : mv_launch<1, 4, false, true>(p, smem, sms, overlap, stream);
}

}  // namespace cutb
