// One block turns a row of the residual stream into the next sublayer's normalised input: the step between two
// sublayers of a model whose norms sit before and after each of them,
//   x' = x + N(y; post_w)      N(v; w)[i] = v[i] / sqrt(mean(part(i)^2) + eps) * w[i]
//   h  = N(x'; pre_w)
// with `groups` equal consecutive parts, each normalised by its own mean square.  y may be null (the first sublayer:
// x' = x).  Used by the row kernel of the prefill (mixer_ops.cu) and by the decode mat-vec's activation staging
// (dense_matvec.cu).
#pragma once
#include "common.cuh"

namespace cutb {
namespace {

struct NormStage {
  const float *x, *y, *post_w, *pre_w;
  float *x_out;  // x' goes here when not null (must not alias x when several blocks stage the same row)
  uint32_t dim, groups;
  float eps;
};

// floats of shared memory a stage may need: two rows, a partial sum per warp, a factor per group, two sums per 128 elements
__host__ __device__ inline uint32_t norm_stage_floats(uint32_t dim, uint32_t groups) { return 2 * ((dim + 3) / 4 * 4) + 32 + (groups + 3) / 4 * 4 + dim / 64; }

// inv[g] = 1 / sqrt(mean of row[part g]^2 + eps); part = 32 floats of scratch.  Fixed summation order.
__device__ __forceinline__ void group_factors(const float *row, uint32_t dim, uint32_t groups, float eps, float *part, float *inv) {
  const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, nwarps = blockDim.x >> 5, gs = dim / groups;
  if (groups <= nwarps) {  // several warps per group
    const uint32_t wpg = nwarps / groups, g = warp / wpg, sub = warp % wpg;
    float s = 0.f;
    if (g < groups) {
      const float *r = row + g * gs;
      for (uint32_t i = sub * 32 + lane; i < gs; i += wpg * 32) s = fmaf(r[i], r[i], s);
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
    if (lane == 0) part[warp] = s;
    __syncthreads();
    if (tid < groups) {
      float t = 0.f;
      for (uint32_t w = 0; w < wpg; ++w) t += part[tid * wpg + w];
      inv[tid] = 1.0f / sqrtf(t / (float)gs + eps);
    }
  } else {
    for (uint32_t g = warp; g < groups; g += nwarps) {
      const float *r = row + g * gs;
      float s = 0.f;
      for (uint32_t i = lane; i < gs; i += 32) s = fmaf(r[i], r[i], s);
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
      if (lane == 0) inv[g] = 1.0f / sqrtf(s / (float)gs + eps);
    }
  }
  __syncthreads();
}

// Fast path for rows whose groups are whole multiples of 128 elements and which the block holds in registers (IT 16-byte pieces
// per thread): a warp's piece of 128 elements lies in one group, its sum of squares is one entry of `part`, and every warp adds
// up its own group's entries.  Two barriers in all.  `norms` (optional): post_w then pre_w in shared
// memory, copied there by this block's own cp.async.
template <int IT, class Store4>
__device__ __forceinline__ void stage_norm_regs(const NormStage &n, float *part, const float *norms, bool write_x, Store4 store4) {
  const uint32_t tid = threadIdx.x, lane = tid & 31, nt = blockDim.x, d4 = n.dim / 4, chunks = n.dim / 128, per = chunks / n.groups;
  const float inv_gs = 1.0f / (float)(n.dim / n.groups);
  float4 x[IT], y[IT];
#pragma unroll
  for (int it = 0; it < IT; ++it) {
    const uint32_t i = tid + it * nt;
    x[it] = i < d4 ? reinterpret_cast<const float4 *>(n.x)[i] : make_float4(0.f, 0.f, 0.f, 0.f);
    y[it] = n.y && i < d4 ? reinterpret_cast<const float4 *>(n.y)[i] : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  if (norms) asm volatile("cp.async.wait_all;" ::: "memory");  // (this thread's pieces; a barrier lies before their use)
  auto factors = [&](const float4 (&v)[IT], float *buf, float (&f)[IT]) {
#pragma unroll
    for (int it = 0; it < IT; ++it) {
      float s = fmaf(v[it].x, v[it].x, fmaf(v[it].y, v[it].y, fmaf(v[it].z, v[it].z, v[it].w * v[it].w)));
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
      const uint32_t c = (tid + it * nt) / 32;
      if (lane == 0 && c < chunks) buf[c] = s;
    }
    __syncthreads();
#pragma unroll
    for (int it = 0; it < IT; ++it) {
      const uint32_t c = (tid + it * nt) / 32, g0 = c / per * per;
      float s = 0.f;
      if (c < chunks)
        for (uint32_t k = lane; k < per; k += 32) s += buf[g0 + k];
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
      f[it] = 1.0f / sqrtf(s * inv_gs + n.eps);
    }
  };
  float f[IT];
  if (n.y) {
    factors(y, part, f);
    const float4 *w4 = reinterpret_cast<const float4 *>(norms ? norms : n.post_w);
#pragma unroll
    for (int it = 0; it < IT; ++it) {
      const uint32_t i = tid + it * nt;
      if (i < d4) {
        const float4 w = w4[i];
        x[it].x = fmaf(y[it].x * f[it], w.x, x[it].x), x[it].y = fmaf(y[it].y * f[it], w.y, x[it].y);
        x[it].z = fmaf(y[it].z * f[it], w.z, x[it].z), x[it].w = fmaf(y[it].w * f[it], w.w, x[it].w);
        if (write_x) reinterpret_cast<float4 *>(n.x_out)[i] = x[it];
      }
    }
  }
  factors(x, part + chunks, f);
  const float4 *w4 = reinterpret_cast<const float4 *>(norms ? norms + n.dim : n.pre_w);
#pragma unroll
  for (int it = 0; it < IT; ++it) {
    const uint32_t i = tid + it * nt;
    if (i < d4) {
      const float4 w = w4[i];
      store4(4 * i, make_float4(x[it].x * f[it] * w.x, x[it].y * f[it] * w.y, x[it].z * f[it] * w.z, x[it].w * f[it] * w.w));
    }
  }
}
__host__ __device__ inline bool norm_stage_fits(uint32_t dim, uint32_t groups, uint32_t threads, int it) {
  return dim % groups == 0 && dim / groups % 128 == 0 && dim <= threads * 4 * (uint32_t)it;
}

// Runs on all threads of the block; `smem` holds norm_stage_floats() floats.  store4(i, h[i .. i+3]) is called for every i
// that is a multiple of 4 when the group size allows it (VEC), else store1(i, h[i]) for every i.  Both rows are loaded at
// once, so the stage costs one memory round trip and two block reductions.
template <class Store4, class Store1>
__device__ __forceinline__ void stage_norm(const NormStage &n, float *smem, bool write_x, Store4 store4, Store1 store1) {
  const uint32_t tid = threadIdx.x, nt = blockDim.x, dim = n.dim, gs = dim / n.groups, pad = (dim + 3) / 4 * 4;
  float *rx = smem, *ry = smem + pad, *part = ry + pad, *inv = part + 32;
  if (gs % 4 == 0) {
    float4 *rx4 = reinterpret_cast<float4 *>(rx), *ry4 = reinterpret_cast<float4 *>(ry);
    const float4 *x4 = reinterpret_cast<const float4 *>(n.x), *y4 = reinterpret_cast<const float4 *>(n.y);
    const uint32_t d4 = dim / 4, gs4 = gs / 4;
#pragma unroll 4
    for (uint32_t i = tid; i < d4; i += nt) {
      rx4[i] = x4[i];
      if (n.y) ry4[i] = y4[i];
    }
    __syncthreads();
    if (n.y) {
      group_factors(ry, dim, n.groups, n.eps, part, inv);
      const float4 *w4 = reinterpret_cast<const float4 *>(n.post_w);
      float4 *o4 = reinterpret_cast<float4 *>(n.x_out);
#pragma unroll 4
      for (uint32_t i = tid; i < d4; i += nt) {
        const float f = inv[i / gs4];
        const float4 w = __ldg(w4 + i), y = ry4[i];
        float4 x = rx4[i];
        x.x = fmaf(y.x * f, w.x, x.x), x.y = fmaf(y.y * f, w.y, x.y), x.z = fmaf(y.z * f, w.z, x.z), x.w = fmaf(y.w * f, w.w, x.w);
        rx4[i] = x;
        if (write_x) o4[i] = x;
      }
      __syncthreads();
    }
    group_factors(rx, dim, n.groups, n.eps, part, inv);
    const float4 *w4 = reinterpret_cast<const float4 *>(n.pre_w);
#pragma unroll 4
    for (uint32_t i = tid; i < d4; i += nt) {
      const float f = inv[i / gs4];
      const float4 w = __ldg(w4 + i), x = rx4[i];
      store4(4 * i, make_float4(x.x * f * w.x, x.y * f * w.y, x.z * f * w.z, x.w * f * w.w));
    }
  } else {
    for (uint32_t i = tid; i < dim; i += nt) {
      rx[i] = n.x[i];
      if (n.y) ry[i] = n.y[i];
    }
    __syncthreads();
    if (n.y) {
      group_factors(ry, dim, n.groups, n.eps, part, inv);
      for (uint32_t i = tid; i < dim; i += nt) {
        rx[i] = fmaf(ry[i] * inv[i / gs], __ldg(n.post_w + i), rx[i]);
        if (write_x) n.x_out[i] = rx[i];
      }
      __syncthreads();
    }
    group_factors(rx, dim, n.groups, n.eps, part, inv);
    for (uint32_t i = tid; i < dim; i += nt) store1(i, rx[i] * inv[i / gs] * __ldg(n.pre_w + i));
  }
}

}  // namespace
}  // namespace cutb
