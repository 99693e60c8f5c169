// Decode mat-vec over dense bf16 weights: C[N] = act(W[N, K] x + bias) for one activation row, fp32 throughout besides the
// weights themselves (a bf16 weight times an fp32 activation, fp32 accumulation).
//
// HBM-bound: every weight is read once.  A block of 16 warps keeps the activation row in shared memory; a warp owns R weight
// rows (R = 1, 2, or the three rows z / x / g of one recurrence channel) and, for narrow weights, a 1 / WK share of K, and
// keeps UNR x R 16-byte loads in flight.  The grid covers the SMs once or twice and walks the rows.  The first batch of
// weight loads is issued before the wait for the previous kernel (weights are constants of the model), so under programmatic
// launch the stream starts while the predecessor still finishes.  The activation row lies in two planes (elements 8 i .. 8 i + 3
// and 8 i + 4 .. 8 i + 7), so the 16-byte reads of a warp fall on distinct banks.
//
// Fused steps:
//  * input: the row is either given (fp32 or bf16), or made here from the residual stream and the previous sublayer's output
//    (post-norm, residual add, pre-norm: norm_stage.cuh); block 0 writes the new residual row;
//  * output: bias and one elementwise op, or the gated recurrence  s = (1 - z) s + z c  of one token with its state update
//    and output gate (rows z, x, g of channel j are rows j, width + j, 2 width + j of the stacked weight).
#include <cuda_bf16.h>

#include "common.cuh"
#include "dense_common.cuh"
#include "kernels.h"
#include "norm_stage.cuh"

namespace cutb {
namespace {

constexpr int MV_THREADS = 512, MV_WARPS = MV_THREADS / 32;

struct MvParams {
  const void *A;
  const __nv_bfloat16 *W;
  const float *bias;
  void *C;
  float *state;  // recurrence
  uint32_t K, K8, N, ldw8;
  uint32_t wk;       // warps that share a row (power of two, <= MV_WARPS)
  uint32_t ntiles;   // row tiles
  uint32_t row_step; // distance of a tile's rows (1, or width for the recurrence)
  int a_bf16, c_bf16, unary;
  NormStage norm;  // norm.pre_w != null: the input is staged from the residual stream
};

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
__global__ void __launch_bounds__(MV_THREADS, 2) dense_matvec_kernel(const MvParams p) {
  extern __shared__ __align__(16) float mv_smem[];
  float4 *lo = reinterpret_cast<float4 *>(mv_smem), *hi = lo + p.K8;  // activation planes
  float *stage = mv_smem + 8 * p.K8;                                  // norm staging rows
  __shared__ float part[MV_WARPS][R];
  const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  const uint32_t WK = p.wk, groups = MV_WARPS / WK, grp = warp / WK, wk = warp % WK;
  const uint32_t step = 32 * WK, k0 = wk * 32 + lane;
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");

  const uint4 *W4 = reinterpret_cast<const uint4 *>(p.W);
  uint32_t tile = blockIdx.x * groups + grp;
  auto row_of = [&](uint32_t t, int r) -> uint32_t { return GRU ? t + (uint32_t)r * p.row_step : t * R + (uint32_t)r; };
  uint4 w[UNR][R];
  auto load_batch = [&](uint32_t t, uint32_t kb) {
#pragma unroll
    for (int u = 0; u < UNR; ++u) {
      const uint32_t k = kb + u * step;
#pragma unroll
      for (int r = 0; r < R; ++r) {
        const uint32_t row = row_of(t, r);
        w[u][r] = (t < p.ntiles && row < p.N && k < p.K8) ? ld_stream(W4 + (size_t)row * p.ldw8 + k) : make_uint4(0, 0, 0, 0);
      }
    }
  };
  load_batch(tile, k0);
  asm volatile("griddepcontrol.wait;" ::: "memory");

  // ---- the activation row -> two planes, zero past K ----
  auto put1 = [&](uint32_t i, float v) { mv_smem[(i & 4 ? 4 * p.K8 : 0) + (i >> 3) * 4 + (i & 3)] = v; };
  auto put4 = [&](uint32_t i, float4 v) { (i & 4 ? hi : lo)[i >> 3] = v; };
  for (uint32_t i = p.K + tid; i < 8 * p.K8; i += MV_THREADS) put1(i, 0.f);
  if (p.norm.pre_w) {
    stage_norm(p.norm, stage, blockIdx.x == 0 && p.norm.x_out != nullptr, put4, put1);
  } else if (p.a_bf16) {
    const __nv_bfloat16 *a = reinterpret_cast<const __nv_bfloat16 *>(p.A);
    for (uint32_t i = tid; i < p.K; i += MV_THREADS) put1(i, __bfloat162float(a[i]));
  } else {
    const float *a = reinterpret_cast<const float *>(p.A);
    const uint32_t k4 = p.K / 4;
#pragma unroll 4
    for (uint32_t i = tid; i < k4; i += MV_THREADS) put4(4 * i, reinterpret_cast<const float4 *>(a)[i]);
    for (uint32_t i = 4 * k4 + tid; i < p.K; i += MV_THREADS) put1(i, a[i]);
  }
  __syncthreads();

  const uint32_t turns = (p.ntiles + gridDim.x * groups - 1) / (gridDim.x * groups);
  for (uint32_t turn = 0; turn < turns; ++turn) {
    float acc[R];
#pragma unroll
    for (int r = 0; r < R; ++r) acc[r] = 0.f;
    const uint32_t next = tile + gridDim.x * groups;
    for (uint32_t kb = k0; kb < p.K8 + k0; kb += UNR * step) {  // (the same trip count in every lane)
#pragma unroll
      for (int u = 0; u < UNR; ++u) {
        const uint32_t k = kb + u * step;
        if (k < p.K8) {
          const float4 a = lo[k], b = hi[k];
#pragma unroll
          for (int r = 0; r < R; ++r) fma8(acc[r], w[u][r], a, b);
        }
      }
      if (kb + UNR * step < p.K8 + k0) load_batch(tile, kb + UNR * step);
    }
    if (turn + 1 < turns) load_batch(next, k0);  // in flight during the reduction below
#pragma unroll
    for (int r = 0; r < R; ++r)
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) acc[r] += __shfl_xor_sync(0xffffffffu, acc[r], o);
    bool writer = lane == 0;
    if (WK > 1) {
      if (turn) __syncthreads();  // the previous turn's sums have been read
      if (lane == 0) {
#pragma unroll
        for (int r = 0; r < R; ++r) part[warp][r] = acc[r];
      }
      __syncthreads();
      writer = lane == 0 && wk == 0;
      if (writer) {
#pragma unroll
        for (int r = 0; r < R; ++r) {
          acc[r] = 0.f;
          for (uint32_t i = 0; i < WK; ++i) acc[r] += part[warp + i][r];
        }
      }
    }
    if (writer && tile < p.ntiles) {
      if constexpr (GRU) {
        const uint32_t j = tile, width = p.row_step;
        float z = acc[0], u = acc[1], g = acc[2];
        if (p.bias) z += __ldg(p.bias + j), u += __ldg(p.bias + width + j), g += __ldg(p.bias + 2 * width + j);
        const float s = mingru_update(p.state[j], z, u);
        p.state[j] = s;
        store_out(p.C, p.c_bf16, j, s * silu(g));
      } else {
#pragma unroll
        for (int r = 0; r < R; ++r) {
          const uint32_t row = tile * R + r;
          if (row < p.N) store_out(p.C, p.c_bf16, row, dense_unary(acc[r] + (p.bias ? __ldg(p.bias + row) : 0.f), p.unary));
        }
      }
    }
    tile = next;
  }
}

template <int R, int UNR, bool GRU> int mv_launch(MvParams &p, uint32_t smem, uint32_t sms, bool overlap, cudaStream_t stream) {
  static bool configured[64] = {};
  int dev = 0;
  CUTB_CUDA_TRY(cudaGetDevice(&dev));
  if (dev < 0 || dev >= 64 || !configured[dev]) {
    DeviceInfo di;
    if (int rc = get_device_info(&di)) return rc;
    CUTB_CUDA_TRY(cudaFuncSetAttribute(dense_matvec_kernel<R, UNR, GRU>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                       (int)di.smem_optin - 2048));
    if (dev >= 0 && dev < 64) configured[dev] = true;
  }
  const uint32_t per_block = MV_WARPS / p.wk, want = (p.ntiles + per_block - 1) / per_block;
  const uint32_t per_sm = smem + 2048 <= 113 * 1024 ? 2u : 1u;
  // as many blocks as fit at once, but the rows dealt evenly: ceil(want / turns) blocks take `turns` tiles each
  const uint32_t turns = (want + sms * per_sm - 1) / (sms * per_sm);
  const uint32_t grid = (want + turns - 1) / turns;
  if (overlap) {
    CUTB_CUDA_TRY(launch_pdl(dense_matvec_kernel<R, UNR, GRU>, dim3(grid), dim3(MV_THREADS), smem, stream, p));
  } else {
    dense_matvec_kernel<R, UNR, GRU><<<grid, MV_THREADS, smem, stream>>>(p);
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
  const uint32_t sms = (uint32_t)di.sm_count, warps = sms * 2 * MV_WARPS;
  // two rows per warp share the activation reads; one where two would leave warps idle
  const bool one = !gru && d.N < warps;
  p.row_step = gru ? d.N / 3 : 1;
  p.ntiles = gru ? d.N / 3 : (one ? d.N : (d.N + 1) / 2);
  // share a row between warps while there are warps to spare and a share still is a full batch of loads
  const uint32_t batch = 32 * (gru ? 2 : 4);
  p.wk = 1;
  while (p.wk < MV_WARPS && p.ntiles * p.wk * 2 <= warps && p.K8 >= batch * p.wk * 2) p.wk *= 2;
  const uint32_t smem = mv_smem_bytes(d);
  const bool overlap = !(d.flags & CUTB_FLAG_NO_OVERLAP);
  if (gru) return mv_launch<3, 2, true>(p, smem, sms, overlap, stream);
  if (one) return mv_launch<1, 4, false>(p, smem, sms, overlap, stream);
  return mv_launch<2, 4, false>(p, smem, sms, overlap, stream);
}

}  // namespace cutb
