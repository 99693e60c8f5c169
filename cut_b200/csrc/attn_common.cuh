// Cache element access, asynchronous copies and warp MMA wrappers shared by the attention kernels of the layer-list models.
#pragma once
#include <cuda_bf16.h>

#include "common.cuh"
#include "dense_common.cuh"

namespace cutb {
namespace {

__device__ __forceinline__ float kvf(float v) { return v; }
__device__ __forceinline__ float kvf(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void kv_put(float *p, float v) { *p = v; }
__device__ __forceinline__ void kv_put(__nv_bfloat16 *p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ float kv_round(float v, const float *) { return v; }
__device__ __forceinline__ float kv_round(float v, const __nv_bfloat16 *) { return __bfloat162float(__float2bfloat16_rn(v)); }
// eight consecutive cache elements
struct Raw8f { float4 a, b; };
__device__ __forceinline__ Raw8f kv_raw8(const float *p) {
  return Raw8f{__ldg(reinterpret_cast<const float4 *>(p)), __ldg(reinterpret_cast<const float4 *>(p) + 1)};
}
__device__ __forceinline__ uint4 kv_raw8(const __nv_bfloat16 *p) { return __ldg(reinterpret_cast<const uint4 *>(p)); }
__device__ __forceinline__ void kv_zero8(Raw8f &r) { r.a = r.b = make_float4(0.f, 0.f, 0.f, 0.f); }
__device__ __forceinline__ void kv_zero8(uint4 &r) { r = make_uint4(0, 0, 0, 0); }
__device__ __forceinline__ void kv_unpack8(const Raw8f &r, float (&v)[8]) {
  v[0] = r.a.x, v[1] = r.a.y, v[2] = r.a.z, v[3] = r.a.w, v[4] = r.b.x, v[5] = r.b.y, v[6] = r.b.z, v[7] = r.b.w;
}
__device__ __forceinline__ void kv_unpack8(const uint4 &r, float (&v)[8]) {
  v[0] = bf16_lo(r.x), v[1] = bf16_hi(r.x), v[2] = bf16_lo(r.y), v[3] = bf16_hi(r.y);
  v[4] = bf16_lo(r.z), v[5] = bf16_hi(r.z), v[6] = bf16_lo(r.w), v[7] = bf16_hi(r.w);
}
template <typename KV> struct RawOf { using type = uint4; };
template <> struct RawOf<float> { using type = Raw8f; };

__device__ __forceinline__ void cp_async16(uint32_t dst, const void *src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ void ldsm_x4(uint32_t addr, uint32_t &r0, uint32_t &r1, uint32_t &r2, uint32_t &r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void ldsm_x4_trans(uint32_t addr, uint32_t &r0, uint32_t &r1, uint32_t &r2, uint32_t &r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
               : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3)
               : "r"(addr));
}
__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
  // (not volatile: a pure function of its registers, free to move between the loads of the next fragments)
  asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// two weights as bf16 high parts, and what the rounding left as bf16 low parts
__device__ __forceinline__ void split_bf16(float a, float b, uint32_t &hi, uint32_t &lo) {
  hi = pack_bf16(a, b);
  lo = pack_bf16(a - bf16_lo(hi), b - bf16_hi(hi));
}

}  // namespace
}  // namespace cutb
