// Routing of a batch of tokens to experts: the choice and its weights per token, and the expert-sorted order of all (token,
// choice) pairs, by expert and then token, so that the grouped GEMMs (dense_gemm.cu) read each expert's rows in one piece.
//  * moe_route_kernel: a warp per token;
//  * moe_sort_kernel: a block per expert counts the choices of lower experts (where its rows begin) and ranks its own;
//  * moe_scatter_kernel: copies the tokens' rows to their places.
#include <cuda_bf16.h>

#include "common.cuh"
#include "dense_common.cuh"
#include "kernels.h"
#include "moe_common.cuh"

namespace cutb {
namespace {

constexpr int MR_WARPS = 4;

__global__ void __launch_bounds__(32 * MR_WARPS) moe_route_kernel(const cutb_moe_desc d, uint32_t epad) {
  extern __shared__ __align__(16) float mr_smem[];  // per warp: logits [epad], choices [top]
  pdl_enter();
  const uint32_t lane = threadIdx.x & 31, warp = threadIdx.x >> 5, t = blockIdx.x * MR_WARPS + warp;
  if (t >= d.n_tokens) return;
  float *z = mr_smem + warp * (epad + (d.top + 3) / 4 * 4);
  uint32_t *ids = reinterpret_cast<uint32_t *>(z + epad);
  for (uint32_t e = lane; e < epad; e += 32) z[e] = e < d.experts ? __ldg(d.logits + t * d.ld_logits + e) : -INFINITY;
  for (uint32_t k = lane; k < d.top; k += 32) ids[k] = 0;
  __syncwarp();
  choose_experts(z, d.experts, d.top, lane, 32, ids);
  __syncwarp();
  for (uint32_t k = lane; k < d.top; k += 32) {
    d.ids[t * d.top + k] = ids[k];
    d.weights[t * d.top + k] = choice_weight(z, ids, d.top, k);
  }
}

constexpr int MS_THREADS = 1024;

// Thread i owns the i-th stretch of the choices; two passes over it: count, then number.
__global__ void __launch_bounds__(MS_THREADS) moe_sort_kernel(const uint32_t *ids, uint32_t n, uint32_t experts, uint32_t *slots, uint32_t *offsets) {
  __shared__ uint32_t less_w[MS_THREADS / 32], same_w[MS_THREADS / 32];
  pdl_enter();
  const uint32_t e = blockIdx.x, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, per = (n + MS_THREADS - 1) / MS_THREADS;
  const uint32_t lo = min(tid * per, n), hi = min(lo + per, n);
  uint32_t less = 0, same = 0;
  for (uint32_t i = lo; i < hi; ++i) {
    const uint32_t v = __ldg(ids + i);
    less += v < e, same += v == e;
  }
  uint32_t before = same;  // choices of this expert up to and including this thread's
#pragma unroll
  for (int o = 1; o < 32; o <<= 1) {
    const uint32_t v = __shfl_up_sync(0xffffffffu, before, o);
    if (lane >= (uint32_t)o) before += v;
  }
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) less += __shfl_xor_sync(0xffffffffu, less, o);
  if (lane == 31) same_w[warp] = before;
  if (lane == 0) less_w[warp] = less;
  __syncthreads();
  uint32_t start = 0;
  for (uint32_t w = 0; w < MS_THREADS / 32; ++w) start += less_w[w];
  uint32_t at = start + before - same;
  for (uint32_t w = 0; w < warp; ++w) at += same_w[w];
  if (tid == 0) offsets[e] = start;
  if (e == 0 && tid == 0) offsets[experts] = n;
  for (uint32_t i = lo; i < hi && same; ++i)
    if (__ldg(ids + i) == e) slots[i] = at++;
}

// one block per (token, choice)
template <typename T> __global__ void __launch_bounds__(128) moe_scatter_kernel(const cutb_moe_desc d, int vec) {
  pdl_enter();
  const uint32_t i = blockIdx.x, t = i / d.top, to = __ldg(d.slots + i);
  if (to >= d.n_tokens * d.top) return;
  const T *src = reinterpret_cast<const T *>(d.A) + t * d.lda;
  T *dst = reinterpret_cast<T *>(d.C) + to * d.ldc;
  if (vec) {
    constexpr uint32_t V = 16 / sizeof(T);
    for (uint32_t c = threadIdx.x; c < (d.K + V - 1) / V; c += 128) reinterpret_cast<uint4 *>(dst)[c] = __ldg(reinterpret_cast<const uint4 *>(src) + c);
  } else {
    for (uint32_t c = threadIdx.x; c < d.K; c += 128) dst[c] = src[c];
  }
}

}  // namespace

int moe_route_launch(const cutb_moe_desc &d, cudaStream_t stream) {
  const uint32_t epad = (d.experts + 3) / 4 * 4, smem = MR_WARPS * 4 * (epad + (d.top + 3) / 4 * 4);
  CUTB_CUDA_TRY(launch_pdl(moe_route_kernel, dim3((d.n_tokens + MR_WARPS - 1) / MR_WARPS), dim3(32 * MR_WARPS), smem, stream, d, epad));
  CUTB_CUDA_TRY(launch_pdl(moe_sort_kernel, dim3(d.experts), dim3(MS_THREADS), 0, stream, d.ids, d.n_tokens * d.top, d.experts, d.slots, d.offsets));
  return CUTB_OK;
}

int moe_scatter_launch(const cutb_moe_desc &d, cudaStream_t stream) {
  const uint32_t size = d.a_dtype == CUTB_BF16 ? 2 : 4, V = 16 / size, whole = (d.K + V - 1) / V * V;
  // (16 bytes at a time: rows may be copied up to the next multiple when both strides hold it)
  const int vec = d.lda % V == 0 && d.ldc % V == 0 && d.lda >= whole && d.ldc >= whole &&
                  (reinterpret_cast<uintptr_t>(d.A) | reinterpret_cast<uintptr_t>(d.C)) % 16 == 0;
  const dim3 grid(d.n_tokens * d.top);
  if (d.a_dtype == CUTB_BF16) CUTB_CUDA_TRY(launch_pdl(moe_scatter_kernel<uint16_t>, grid, dim3(128), 0, stream, d, vec));
  else CUTB_CUDA_TRY(launch_pdl(moe_scatter_kernel<float>, grid, dim3(128), 0, stream, d, vec));
  return CUTB_OK;
}

}  // namespace cutb
