// The router's choice, shared by the batch kernel (moe.cu) and the decode mat-vec (expert_matvec.cu).
#pragma once
#include "common.cuh"

namespace cutb {
namespace {

constexpr uint32_t MOE_MAX_EXPERTS = 1024;

// Called by `nt` threads numbered t: ids[r] = expert with the r-th largest logit (ties: the lower index first), r < top.  z holds E
// logits and -inf up to a multiple of 4.  ids must hold valid indices before (an entry stays as it is when a logit is NaN).
__device__ __forceinline__ void choose_experts(const float *z, uint32_t E, uint32_t top, uint32_t t, uint32_t nt, uint32_t *ids) {
  for (uint32_t e = t; e < E; e += nt) {
    const float mine = z[e];
    uint32_t rank = 0;
    for (uint32_t i = 0; i < E; i += 4) {
      const float4 o = *reinterpret_cast<const float4 *>(z + i);
      rank += (o.x > mine || (o.x == mine && i < e)) + (o.y > mine || (o.y == mine && i + 1 < e)) + (o.z > mine || (o.z == mine && i + 2 < e)) +
              (o.w > mine || (o.w == mine && i + 3 < e));
    }
    if (rank < top) ids[rank] = e;
  }
}
// weight of choice r: the softmax over the chosen logits
__device__ __forceinline__ float choice_weight(const float *z, const uint32_t *ids, uint32_t top, uint32_t r) {
  const float m = z[ids[0]];
  float sum = 0.f;
  for (uint32_t k = 0; k < top; ++k) sum += expf(z[ids[k]] - m);
  return expf(z[ids[r]] - m) / sum;
}

}  // namespace
}  // namespace cutb
