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
};

__device__ __forceinline__ void cp_async16(uint32_t dst, const void *src) {
  asm volatile("cp.async.ca.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
__device__ __forceinline__ void fma8(float &acc, const uint4 w, const float4 a, const float4 b) {
  acc = fmaf(bf16_lo(w.x), a.x, acc);
  acc = fmaf(bf16_hi(w.x), a.y, acc);
  acc = fmaf(bf16_lo(w.y), a.z, acc);
  acc = fmaf(bf16_hi(w.y), a.w, acc);
  acc = fmaf(bf16_lo(w.z), b.x, acc);
  acc = fmaf(bf16_hi(w.z), b.y, acc);
  acc = fmaf(bf16_lo(w.w), b.z, acc);
  acc = fmaf(bf16_hi(w.w), b.w, acc);
}

template <int R, int UNR, bool GRU>
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
  for (uint32_t i = p.K + tid; i < 8 * p.K8; i += nt) put1(i, 0.f);
  if (fast_norm) {
    stage_norm_regs<2>(p.norm, stage + 2 * p.K, stage, blockIdx.x == 0 && p.norm.x_out != nullptr, put4);
  } else if (p.norm.pre_w) {
    stage_norm(p.norm, stage, blockIdx.x == 0 && p.norm.x_out != nullptr, put4, put1);
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

template <int R, int UNR, bool GRU> int mv_launch(MvParams &p, uint32_t smem, uint32_t sms, bool overlap, cudaStream_t stream) {
  static bool configured[64] = {};
  int dev = 0;
  CUTB_CUDA_TRY(cudaGetDevice(&dev));
  if (dev < 0 || dev >= 64 || !configured[dev]) {
    DeviceInfo di;
    if (int rc = get_device_info(&di)) return rc;
    CUTB_CUDA_TRY(cudaFuncSetAttribute(dense_matvec_kernel<R, UNR, GRU>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)di.smem_optin - 2048));
    if (dev >= 0 && dev < 64) configured[dev] = true;
  }
  const uint32_t per_sm = (p.ntiles + sms - 1) / sms, turns = (per_sm + MV_MAX_WARPS - 1) / MV_MAX_WARPS;
  uint32_t warps = (per_sm + turns - 1) / turns;
  if (warps < MV_MIN_WARPS) warps = MV_MIN_WARPS;  // (the staging of the input wants threads too)
  const dim3 grid(p.ntiles < sms ? p.ntiles : sms), block(32 * warps);
  if (overlap) {
    CUTB_CUDA_TRY(launch_pdl(dense_matvec_kernel<R, UNR, GRU>, grid, block, smem, stream, p));
  } else {
    dense_matvec_kernel<R, UNR, GRU><<<grid, block, smem, stream>>>(p);
    CUTB_CUDA_TRY(cudaGetLastError());
  }
  return CUTB_OK;
}

uint32_t mv_smem_bytes(const cutb_dense_desc &d) {
  const uint32_t K8 = (d.K + 7) / 8;
  return 4 * (8 * K8 + (d.norm_w ? norm_stage_floats(d.K, d.norm_groups) : 0));
}

}  // namespace

bool dense_matvec_supported(const cutb_dense_desc &d) { return d.M == 1 && mv_smem_bytes(d) <= 220 * 1024; }

int dense_matvec_launch(const cutb_dense_desc &d, cudaStream_t stream) {
  DeviceInfo di;
  if (int rc = get_device_info(&di)) return rc;
  MvParams p{};
  p.A = d.A, p.W = reinterpret_cast<const __nv_bfloat16 *>(d.W), p.bias = d.bias, p.C = d.C, p.state = d.gru_state;
  p.K = d.K, p.K8 = (d.K + 7) / 8, p.N = d.N, p.ldw8 = d.ldw / 8;
  p.a_bf16 = d.a_dtype == CUTB_BF16, p.c_bf16 = d.c_dtype == CUTB_BF16, p.unary = d.unary_op;
  p.norm = NormStage{d.res_x, d.res_y, d.res_norm_w, d.norm_w, d.res_out, d.K, d.norm_groups ? d.norm_groups : 1, d.norm_eps};
  const bool gru = d.gru_state != nullptr;
  const uint32_t sms = (uint32_t)di.sm_count;
  const uint32_t sms_all = sms * MV_MAX_WARPS;
  const bool two = !gru && d.N >= 2 * sms_all;  // enough rows: two per warp share the activation reads
  p.row_step = gru ? d.N / 3 : 1;
  p.ntiles = gru ? d.N / 3 : (two ? (d.N + 1) / 2 : d.N);
  const uint32_t smem = mv_smem_bytes(d);
  const bool overlap = !(d.flags & CUTB_FLAG_NO_OVERLAP);
  if (gru) return mv_launch<3, 1, true>(p, smem, sms, overlap, stream);
  return two ? mv_launch<2, 2, false>(p, smem, sms, overlap, stream) : mv_launch<1, 4, false>(p, smem, sms, overlap, stream);
}

}  // namespace cutb
