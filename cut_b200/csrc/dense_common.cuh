// Elementwise pieces shared by the kernels of the layer-list models (dense bf16 weights).
#pragma once
#include <cuda_bf16.h>

#include "common.cuh"

namespace cutb {
namespace {

__device__ __forceinline__ float bf16_lo(uint32_t x) { return __uint_as_float(x << 16); }
__device__ __forceinline__ float bf16_hi(uint32_t x) { return __uint_as_float(x & 0xffff0000u); }
__device__ __forceinline__ uint32_t pack_bf16(float a, float b) {
  const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
  return *reinterpret_cast<const uint32_t *>(&h);
}
// 16 bytes that are read once: keep them out of L1
__device__ __forceinline__ uint4 ld_stream(const uint4 *p) {
  uint4 v;
  asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0, %1, %2, %3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
  return v;
}
// eight bf16 weights times eight activations
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
__device__ __forceinline__ void store_out(void *C, int bf16, size_t i, float v) {
  if (bf16) reinterpret_cast<__nv_bfloat16 *>(C)[i] = __float2bfloat16_rn(v);
  else reinterpret_cast<float *>(C)[i] = v;
}
// (__fdividef: within 2 ulp; a denominator past 2^126, x below -87, gives 0 like the exact quotient to fp32's last digits)
__device__ __forceinline__ float sigmoid(float x) { return __fdividef(1.0f, 1.0f + expf(-x)); }
__device__ __forceinline__ float silu(float x) { return __fdividef(x, 1.0f + expf(-x)); }

// Elementwise epilogue: 0 none, CUTB_UNARY_RELU_SQUARE, or one of the unary codes of the quantized matmul.
__device__ __forceinline__ float dense_unary(float x, int op) {
  if (op == 0) return x;
  if (op == CUTB_UNARY_RELU_SQUARE) {
    const float r = fmaxf(x, 0.f);
    return r * r;
  }
  return apply_epilogue(x, CUTB_FUSION_UNARY, op, 0.f);
}

// The gated unit of a feed-forward's element: the gate clamped from above, the up value from both sides.
struct GluParams {
  int kind;  // CUTB_GLU_*
  float alpha, beta, limit;
};
__device__ __forceinline__ float glu(const GluParams &p, float g, float u) {
  g = fminf(g, p.limit), u = fminf(fmaxf(u, -p.limit), p.limit);
  return __fdividef(g, 1.0f + expf(-p.alpha * g)) * (u + p.beta);
}

// The gated recurrence of one channel: gate z and candidate c from this token's pre-activations.
__device__ __forceinline__ float mingru_candidate(float u) { return u >= 0.f ? u + 0.5f : sigmoid(u); }
__device__ __forceinline__ float mingru_update(float s, float z_pre, float u) {
  const float z = sigmoid(z_pre);
  return fmaf(1.0f - z, s, z * mingru_candidate(u));
}

}  // namespace
}  // namespace cutb
