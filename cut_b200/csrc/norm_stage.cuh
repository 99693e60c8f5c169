// One block turns a row of the residual stream into the next sublayer's normalised input: the step between two sublayers,
//   x' = x + y_scale * P(y + sum_k part_w[k] * parts[part_rows[k]])       P = N(.; post_w), or the identity without post_w
//   h  = N(x'; pre_w)
//   N(v; w)[i] = (v[i] - c) / sqrt(mean((v - c)^2) + eps) * w[i]          c = mean(v) when centred (layer norm), else 0
// with `groups` equal consecutive parts of a row, each normalised by its own moments.  y and the gathered parts (the experts'
// outputs of a mixture) may be missing; without both x' = x.  Used by the row kernel of the prefill (mixer_ops.cu) and by the
// activation staging of the decode mat-vecs (dense_matvec.cu, expert_matvec.cu).
//
// Centred moments are merged from pieces (mean and sum of squared deviations of each), never as a difference of large sums.
#pragma once
#include "common.cuh"
#include "dense_common.cuh"

namespace cutb {
namespace {

struct NormStage {
  const float *x, *y, *post_w, *pre_w;
  float *x_out;  // x' goes here when not null (must not alias x when several blocks stage the same row)
  uint32_t dim, groups;
  float eps;
  int center;
  float y_scale;
  const void *parts;  // rows of ld_parts elements, fp32 or bf16
  const uint32_t *part_rows;
  const float *part_w;
  uint64_t ld_parts;
  uint32_t n_parts;
  int parts_bf16;
};

// floats of shared memory a stage may need: two rows, a partial sum per warp, two moments per group, four sums per 128 elements
__host__ __device__ inline uint32_t norm_stage_floats(uint32_t dim, uint32_t groups) {
  return 2 * ((dim + 3) / 4 * 4) + 32 + 2 * ((groups + 3) / 4 * 4) + dim / 32;
}

__device__ __forceinline__ bool stage_has_y(const NormStage &n) { return n.y != nullptr || n.n_parts != 0; }
__device__ __forceinline__ float4 stage_y4(const NormStage &n, uint32_t i4) {
  float4 v = n.y ? reinterpret_cast<const float4 *>(n.y)[i4] : make_float4(0.f, 0.f, 0.f, 0.f);
  for (uint32_t k = 0; k < n.n_parts; ++k) {
    const float w = n.part_w[k];
    const size_t at = n.part_rows[k] * n.ld_parts + 4 * (size_t)i4;
    float4 a;
    if (n.parts_bf16) {
      const uint2 r = *reinterpret_cast<const uint2 *>(reinterpret_cast<const __nv_bfloat16 *>(n.parts) + at);
      a = make_float4(bf16_lo(r.x), bf16_hi(r.x), bf16_lo(r.y), bf16_hi(r.y));
    } else {
      a = *reinterpret_cast<const float4 *>(reinterpret_cast<const float *>(n.parts) + at);
    }
    v.x = fmaf(w, a.x, v.x), v.y = fmaf(w, a.y, v.y), v.z = fmaf(w, a.z, v.z), v.w = fmaf(w, a.w, v.w);
  }
  return v;
}
__device__ __forceinline__ float stage_y1(const NormStage &n, uint32_t i) {
  float v = n.y ? n.y[i] : 0.f;
  for (uint32_t k = 0; k < n.n_parts; ++k) {
    const size_t at = n.part_rows[k] * n.ld_parts + i;
    v = fmaf(n.part_w[k], n.parts_bf16 ? __bfloat162float(reinterpret_cast<const __nv_bfloat16 *>(n.parts)[at]) : reinterpret_cast<const float *>(n.parts)[at], v);
  }
  return v;
}
__device__ __forceinline__ float warp_sum(float s) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
  return s;
}

// out[g] = sum of f(row[i]) over part g; part = 32 floats of scratch.  Fixed summation order; ends with a barrier.
template <class F, class G>
__device__ __forceinline__ void group_reduce(uint32_t dim, uint32_t groups, float *part, F f, G put) {
  const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, nwarps = blockDim.x >> 5, gs = dim / groups;
  if (groups <= nwarps) {  // several warps per group
    const uint32_t wpg = nwarps / groups, g = warp / wpg, sub = warp % wpg;
    float s = 0.f;
    if (g < groups)
      for (uint32_t i = sub * 32 + lane; i < gs; i += wpg * 32) s += f(g, g * gs + i);
    s = warp_sum(s);
    if (lane == 0) part[warp] = s;
    __syncthreads();
    if (tid < groups) {
      float t = 0.f;
      for (uint32_t w = 0; w < wpg; ++w) t += part[tid * wpg + w];
      put(tid, t / (float)gs);
    }
  } else {
    for (uint32_t g = warp; g < groups; g += nwarps) {
      float s = 0.f;
      for (uint32_t i = lane; i < gs; i += 32) s += f(g, g * gs + i);
      s = warp_sum(s);
      if (lane == 0) put(g, s / (float)gs);
    }
  }
  __syncthreads();
}
// mu[g] (0 unless centred) and inv[g] = 1 / sqrt(mean of (row[part g] - mu)^2 + eps)
__device__ __forceinline__ void group_factors(const float *row, const NormStage &n, float *part, float *inv, float *mu) {
  if (n.center) group_reduce(n.dim, n.groups, part, [&](uint32_t, uint32_t i) { return row[i]; }, [&](uint32_t g, float m) { mu[g] = m; });
  group_reduce(
      n.dim, n.groups, part,
      [&](uint32_t g, uint32_t i) {
        const float d = n.center ? row[i] - mu[g] : row[i];
        return d * d;
      },
      [&](uint32_t g, float m) {
        inv[g] = 1.0f / sqrtf(m + n.eps);
        if (!n.center) mu[g] = 0.f;
      });
}

// Fast path for rows whose groups are whole multiples of 128 elements and which the block holds in registers (IT 16-byte pieces
// per thread): a warp's piece of 128 elements lies in one group, its moments are entries of `part`, and every warp merges its
// own group's entries.  Two barriers in all.  `norms` (optional): post_w then pre_w in shared memory, copied there by this
// block's own cp.async.  PLAIN: RMS norms before and after, nothing gathered, y_scale 1 (norm_stage_plain), known at compile time.
template <int IT, bool PLAIN, class Store4>
__device__ __forceinline__ void stage_norm_regs(const NormStage &n, float *part, const float *norms, bool write_x, Store4 store4) {
  const uint32_t tid = threadIdx.x, lane = tid & 31, nt = blockDim.x, d4 = n.dim / 4, chunks = n.dim / 128, per = chunks / n.groups;
  const float inv_gs = 1.0f / (float)(n.dim / n.groups);
  float4 x[IT], y[IT];
#pragma unroll
  for (int it = 0; it < IT; ++it) {
    const uint32_t i = tid + it * nt;
    x[it] = i < d4 ? reinterpret_cast<const float4 *>(n.x)[i] : make_float4(0.f, 0.f, 0.f, 0.f);
    if constexpr (PLAIN) y[it] = n.y && i < d4 ? reinterpret_cast<const float4 *>(n.y)[i] : make_float4(0.f, 0.f, 0.f, 0.f);
    else y[it] = i < d4 ? stage_y4(n, i) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  const bool center = !PLAIN && n.center;
  if (norms) asm volatile("cp.async.wait_all;" ::: "memory");  // (this thread's pieces; a barrier lies before their use)
  auto factors = [&](float4 (&v)[IT], float *buf, float (&f)[IT]) {  // centred: v loses its mean here
    float *dev = buf + chunks;
#pragma unroll
    for (int it = 0; it < IT; ++it) {
      const uint32_t c = (tid + it * nt) / 32;
      if (center) {
        const float m = warp_sum((v[it].x + v[it].y) + (v[it].z + v[it].w)) * (1.0f / 128.0f);
        const float a = v[it].x - m, b = v[it].y - m, e = v[it].z - m, g = v[it].w - m;
        const float s = warp_sum(fmaf(a, a, fmaf(b, b, fmaf(e, e, g * g))));
        if (lane == 0 && c < chunks) buf[c] = m, dev[c] = s;
      } else {
        const float s = warp_sum(fmaf(v[it].x, v[it].x, fmaf(v[it].y, v[it].y, fmaf(v[it].z, v[it].z, v[it].w * v[it].w))));
        if (lane == 0 && c < chunks) buf[c] = s;
      }
    }
    __syncthreads();
#pragma unroll
    for (int it = 0; it < IT; ++it) {
      const uint32_t c = (tid + it * nt) / 32, g0 = c / per * per;
      float s = 0.f;
      if (c < chunks)
        for (uint32_t k = lane; k < per; k += 32) s += buf[g0 + k];
      s = warp_sum(s);
      if (center) {
        const float m = s / (float)per;
        s = 0.f;
        if (c < chunks)
          for (uint32_t k = lane; k < per; k += 32) {
            const float d = buf[g0 + k] - m;
            s += fmaf(128.0f * d, d, dev[g0 + k]);
          }
        s = warp_sum(s);
        v[it].x -= m, v[it].y -= m, v[it].z -= m, v[it].w -= m;
      }
      f[it] = 1.0f / sqrtf(s * inv_gs + n.eps);
    }
  };
  float f[IT];
  if (PLAIN && n.y) {
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
  if (!PLAIN && stage_has_y(n)) {
    if (n.post_w) {
      factors(y, part, f);
      const float4 *w4 = reinterpret_cast<const float4 *>(norms ? norms : n.post_w);
#pragma unroll
      for (int it = 0; it < IT; ++it) {
        const uint32_t i = tid + it * nt;
        if (i < d4) {
          const float4 w = w4[i];
          y[it].x *= f[it] * w.x, y[it].y *= f[it] * w.y, y[it].z *= f[it] * w.z, y[it].w *= f[it] * w.w;
        }
      }
    }
#pragma unroll
    for (int it = 0; it < IT; ++it) {
      const uint32_t i = tid + it * nt;
      x[it].x = fmaf(n.y_scale, y[it].x, x[it].x), x[it].y = fmaf(n.y_scale, y[it].y, x[it].y);
      x[it].z = fmaf(n.y_scale, y[it].z, x[it].z), x[it].w = fmaf(n.y_scale, y[it].w, x[it].w);
      if (write_x && i < d4) reinterpret_cast<float4 *>(n.x_out)[i] = x[it];
    }
  }
  factors(x, part + 2 * chunks, f);
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
__host__ __device__ inline bool norm_stage_plain(const NormStage &n) {
  return !n.center && n.n_parts == 0 && (!n.y || (n.post_w && n.y_scale == 1.0f));
}
__host__ __device__ inline bool norm_stage_fits(uint32_t dim, uint32_t groups, uint32_t threads, int it) {
  return dim % groups == 0 && dim / groups % 128 == 0 && dim <= threads * 4 * (uint32_t)it;
}

// Runs on all threads of the block; `smem` holds norm_stage_floats() floats.  store4(i, h[i .. i+3]) is called for every i
// that is a multiple of 4 when the group size allows it (VEC), else store1(i, h[i]) for every i.  Both rows are loaded at
// once, so the stage costs one memory round trip and two block reductions (three when centred).
template <class Store4, class Store1>
__device__ __forceinline__ void stage_norm(const NormStage &n, float *smem, bool write_x, Store4 store4, Store1 store1) {
  const uint32_t tid = threadIdx.x, nt = blockDim.x, dim = n.dim, gs = dim / n.groups, pad = (dim + 3) / 4 * 4, gpad = (n.groups + 3) / 4 * 4;
  float *rx = smem, *ry = smem + pad, *part = ry + pad, *inv = part + 32, *mu = inv + gpad;
  const bool has_y = stage_has_y(n);
  if (gs % 4 == 0) {
    float4 *rx4 = reinterpret_cast<float4 *>(rx), *ry4 = reinterpret_cast<float4 *>(ry);
    const float4 *x4 = reinterpret_cast<const float4 *>(n.x);
    const uint32_t d4 = dim / 4, gs4 = gs / 4;
#pragma unroll 4
    for (uint32_t i = tid; i < d4; i += nt) {
      rx4[i] = x4[i];
      if (has_y) ry4[i] = stage_y4(n, i);
    }
    __syncthreads();
    if (has_y) {
      if (n.post_w) group_factors(ry, n, part, inv, mu);
      const float4 *w4 = reinterpret_cast<const float4 *>(n.post_w);
      float4 *o4 = reinterpret_cast<float4 *>(n.x_out);
#pragma unroll 4
      for (uint32_t i = tid; i < d4; i += nt) {
        float4 y = ry4[i], x = rx4[i];
        if (n.post_w) {
          const float f = inv[i / gs4], m = mu[i / gs4];
          const float4 w = __ldg(w4 + i);
          y.x = (y.x - m) * f * w.x, y.y = (y.y - m) * f * w.y, y.z = (y.z - m) * f * w.z, y.w = (y.w - m) * f * w.w;
        }
        x.x = fmaf(n.y_scale, y.x, x.x), x.y = fmaf(n.y_scale, y.y, x.y), x.z = fmaf(n.y_scale, y.z, x.z), x.w = fmaf(n.y_scale, y.w, x.w);
        rx4[i] = x;
        if (write_x) o4[i] = x;
      }
      __syncthreads();
    }
    group_factors(rx, n, part, inv, mu);
    const float4 *w4 = reinterpret_cast<const float4 *>(n.pre_w);
#pragma unroll 4
    for (uint32_t i = tid; i < d4; i += nt) {
      const float f = inv[i / gs4], m = mu[i / gs4];
      const float4 w = __ldg(w4 + i), x = rx4[i];
      store4(4 * i, make_float4((x.x - m) * f * w.x, (x.y - m) * f * w.y, (x.z - m) * f * w.z, (x.w - m) * f * w.w));
    }
  } else {
    for (uint32_t i = tid; i < dim; i += nt) {
      rx[i] = n.x[i];
      if (has_y) ry[i] = stage_y1(n, i);
    }
    __syncthreads();
    if (has_y) {
      if (n.post_w) group_factors(ry, n, part, inv, mu);
      for (uint32_t i = tid; i < dim; i += nt) {
        const float y = n.post_w ? (ry[i] - mu[i / gs]) * inv[i / gs] * __ldg(n.post_w + i) : ry[i];
        rx[i] = fmaf(n.y_scale, y, rx[i]);
        if (write_x) n.x_out[i] = rx[i];
      }
      __syncthreads();
    }
    group_factors(rx, n, part, inv, mu);
    for (uint32_t i = tid; i < dim; i += nt) store1(i, (rx[i] - mu[i / gs]) * inv[i / gs] * __ldg(n.pre_w + i));
  }
}

}  // namespace
}  // namespace cutb
