// Latent attention over whole-context caches: row p of a cache holds position p's normed latent c and, from column rot_at on, the
// rotated key part that all heads share.  Beside window_attention.cu, whose caches hold keys and values per head.
//
//  * latent_kv_write_kernel: a batch of tokens into the cache, and the norm of the latent queries;
//  * latent_attention_simt_kernel: the absorbed form (every head's query against the cache row itself) in fp32 arithmetic, for
//    any size, either cache type, and any number of tokens.  For one token the keys are shared out over blocks, which leave
//    partial sums; the values' mat-vec behind it merges them while it stages its input (head_matvec_kernel).
#include <cuda_bf16.h>

#include "attn_common.cuh"
#include "common.cuh"
#include "dense_common.cuh"
#include "kernels.h"

namespace cutb {
namespace {

constexpr float LA_NEG = -1e30f, LA_LOG2E = 1.4426950408889634f;
constexpr int LA_THREADS = 256, LA_WARPS = LA_THREADS / 32;

// sum over the block, the same in every thread; `part` holds a float per warp
__device__ __forceinline__ float block_sum(float s, float *part) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
  if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = s;
  __syncthreads();
  s = 0.f;
  for (uint32_t w = 0; w < blockDim.x / 32; ++w) s += part[w];
  __syncthreads();
  return s;
}

// The cache row of one token: put(column, value) for every column of the latent and of the turned key part.  The whole block.
template <class Put> __device__ __forceinline__ void make_cache_row(const cutb_latent_attn_desc &d, uint32_t tok, uint32_t pos, float *part, Put put) {
  const float *row = d.lat + tok * d.ld_lat;
  float s = 0.f;
  for (uint32_t i = threadIdx.x; i < d.rank; i += blockDim.x) s = fmaf(row[i], row[i], s);
  const float inv = 1.0f / sqrtf(block_sum(s, part) / (float)d.rank + d.eps);
  for (uint32_t i = threadIdx.x; i < d.rank; i += blockDim.x) put(i, row[i] * inv * __ldg(d.lat_norm_w + i));
  const uint32_t half = d.rot_dim / 2;
  for (uint32_t i = threadIdx.x; i < half; i += blockDim.x) {
    const float c = __ldg(d.cos_table + (size_t)pos * half + i), sn = __ldg(d.sin_table + (size_t)pos * half + i);
    const float u = row[d.rank + 2 * i], v = row[d.rank + 2 * i + 1];
    put(d.rot_at + 2 * i, u * c - v * sn);
    put(d.rot_at + 2 * i + 1, v * c + u * sn);
  }
}

template <typename KV> __global__ void __launch_bounds__(128) latent_kv_write_kernel(const cutb_latent_attn_desc d) {
  __shared__ float part[4];
  pdl_enter();
  const uint32_t tok = blockIdx.x, pos = (d.pos_ptr ? *d.pos_ptr : d.pos) + tok;
  if (pos >= d.max_pos) {  // no row: record it and write nothing
    if (d.status && threadIdx.x == 0) atomicExch(d.status, (int)CUTB_ERR_INVALID);
    return;
  }
  if (d.lat && blockIdx.y == 0) {
    KV *row = reinterpret_cast<KV *>(d.cache) + pos * d.ld_cache;
    make_cache_row(d, tok, pos, part, [&](uint32_t i, float v) { kv_put(row + i, v); });
  } else {
    const float *row = d.cq + tok * d.ld_cq;
    float s = 0.f;
    for (uint32_t i = threadIdx.x; i < d.q_rank; i += blockDim.x) s = fmaf(row[i], row[i], s);
    const float inv = 1.0f / sqrtf(block_sum(s, part) / (float)d.q_rank + d.eps);
    for (uint32_t i = threadIdx.x; i < d.q_rank; i += blockDim.x)
      store_out(d.cq_out, d.out_dtype == CUTB_BF16, tok * d.ld_cq_out + i, row[i] * inv * __ldg(d.cq_norm_w + i));
  }
}

// ---- absorbed form, fp32 arithmetic ------------------------------------------------------------------------------------
constexpr int LS_HEADS = 4, LS_KEYS = 64, LS_COLS = 4;  // heads of a block, keys of a turn, columns per thread

struct LatentSplit {
  float2 *ml;   // [H][splits]: maximum in log2 units, weight sum
  float *part;  // [H][splits][ld]: weighted sums of latents
  uint32_t splits, ld;
};

template <typename KV> __global__ void __launch_bounds__(LA_THREADS) latent_attention_simt_kernel(const cutb_latent_attn_desc d, const LatentSplit sp,
                                                                                                 uint32_t row_len) {
  extern __shared__ __align__(16) float ls_smem[];  // queries [LS_HEADS][row_len], the new row [row_len]
  __shared__ float sc[LS_HEADS][LS_KEYS], fac[LS_HEADS], head_m[LS_HEADS], head_l[LS_HEADS], part[LA_WARPS];
  const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h0 = blockIdx.x * LS_HEADS, split = blockIdx.y, tok = blockIdx.z;
  const uint32_t nh = min((uint32_t)LS_HEADS, d.n_heads - h0), width = d.dim + d.rot_dim;
  float *qs = ls_smem, *fresh = ls_smem + LS_HEADS * row_len;
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  pdl_enter();
  const uint32_t pos = (d.pos_ptr ? *d.pos_ptr : d.pos) + tok;
  if (pos >= d.max_pos) {
    if (d.status && tid == 0) atomicExch(d.status, (int)CUTB_ERR_INVALID);
    return;
  }
  const uint32_t n = pos + 1, per = (n + sp.splits - 1) / sp.splits, k_lo = min(split * per, n), k_hi = min(k_lo + per, n);
  const KV *cache = reinterpret_cast<const KV *>(d.cache);
  const bool make = d.lat && k_hi == n && k_lo < n;  // this block's keys end with the token's own

  // queries laid out as a cache row, scaled to log2 units, zeros in its gaps
  for (uint32_t i = tid; i < LS_HEADS * row_len; i += LA_THREADS) qs[i] = 0.f;
  for (uint32_t i = tid; i < row_len; i += LA_THREADS) fresh[i] = 0.f;
  __syncthreads();
  const float scale = d.scale * LA_LOG2E;
  for (uint32_t r = 0; r < nh; ++r) {
    const float *qa = d.qa + tok * d.ld_qa + (size_t)(h0 + r) * d.rank, *q = d.q + tok * d.ldq + (size_t)(h0 + r) * width + d.dim;
    for (uint32_t i = tid; i < d.rank; i += LA_THREADS) qs[r * row_len + i] = qa[i] * scale;
    for (uint32_t i = tid; i < d.rot_dim / 2; i += LA_THREADS) {
      const float c = __ldg(d.cos_table + (size_t)pos * (d.rot_dim / 2) + i), s = __ldg(d.sin_table + (size_t)pos * (d.rot_dim / 2) + i);
      const float u = q[2 * i], v = q[2 * i + 1];
      qs[r * row_len + d.rot_at + 2 * i] = (u * c - v * s) * scale;
      qs[r * row_len + d.rot_at + 2 * i + 1] = (v * c + u * s) * scale;
    }
  }
  if (make) {
    KV *row = reinterpret_cast<KV *>(d.cache) + pos * d.ld_cache;
    make_cache_row(d, tok, pos, part, [&](uint32_t i, float v) {
      fresh[i] = kv_round(v, (const KV *)nullptr);
      if (blockIdx.x == 0) kv_put(row + i, v);
    });
  }
  if (tid < LS_HEADS) {
    const bool sink = d.sink && split == 0 && tid < nh;
    head_m[tid] = sink ? d.sink[h0 + tid] * LA_LOG2E : LA_NEG, head_l[tid] = sink ? 1.f : 0.f;
  }
  float acc[LS_HEADS][LS_COLS];
#pragma unroll
  for (int r = 0; r < LS_HEADS; ++r)
#pragma unroll
    for (int c = 0; c < LS_COLS; ++c) acc[r][c] = 0.f;
  __syncthreads();

  for (uint32_t k0 = k_lo; k0 < k_hi; k0 += LS_KEYS) {
    const uint32_t cnt = min((uint32_t)LS_KEYS, k_hi - k0);
    for (uint32_t j = warp; j < cnt; j += LA_WARPS) {
      const KV *row = cache + (size_t)(k0 + j) * d.ld_cache;
      const bool own = make && k0 + j == pos;
      float dot[LS_HEADS] = {};
      for (uint32_t i = lane * 8; i < row_len; i += 256) {
        float kv[8];
        if (own) {
#pragma unroll
          for (int e = 0; e < 8; ++e) kv[e] = fresh[i + e];
        } else {
          kv_unpack8(kv_raw8(row + i), kv);
        }
#pragma unroll
        for (int r = 0; r < LS_HEADS; ++r) {
          const float4 a = *reinterpret_cast<const float4 *>(qs + r * row_len + i), b = *reinterpret_cast<const float4 *>(qs + r * row_len + i + 4);
          dot[r] = fmaf(a.x, kv[0], fmaf(a.y, kv[1], fmaf(a.z, kv[2], fmaf(a.w, kv[3], dot[r]))));
          dot[r] = fmaf(b.x, kv[4], fmaf(b.y, kv[5], fmaf(b.z, kv[6], fmaf(b.w, kv[7], dot[r]))));
        }
      }
#pragma unroll
      for (int r = 0; r < LS_HEADS; ++r) {
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) dot[r] += __shfl_xor_sync(0xffffffffu, dot[r], o);
        if (lane == 0) sc[r][j] = dot[r];
      }
    }
    __syncthreads();
    if (warp < LS_HEADS) {
      const uint32_t r = warp;
      float m = head_m[r];
      for (uint32_t j = lane; j < cnt; j += 32) m = fmaxf(m, sc[r][j]);
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
      float l = 0.f;
      for (uint32_t j = lane; j < cnt; j += 32) {
        const float e = exp2f(sc[r][j] - m);
        sc[r][j] = e;
        l += e;
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) l += __shfl_xor_sync(0xffffffffu, l, o);
      __syncwarp();
      if (lane == 0) {
        const float f = exp2f(head_m[r] - m);
        head_l[r] = fmaf(head_l[r], f, l), head_m[r] = m, fac[r] = f;
      }
    }
    __syncthreads();
#pragma unroll
    for (int c = 0; c < LS_COLS; ++c) {
      const uint32_t col = tid + c * LA_THREADS;
      if (col >= d.rank) break;
#pragma unroll
      for (int r = 0; r < LS_HEADS; ++r) acc[r][c] *= fac[r];
      const KV *p = cache + (size_t)k0 * d.ld_cache + col;
      for (uint32_t j = 0; j < cnt; ++j, p += d.ld_cache) {
        const float v = make && k0 + j == pos ? fresh[col] : kvf(*p);
#pragma unroll
        for (int r = 0; r < LS_HEADS; ++r) acc[r][c] = fmaf(sc[r][j], v, acc[r][c]);
      }
    }
    __syncthreads();  // the next turn overwrites the scores
  }
#pragma unroll
  for (int c = 0; c < LS_COLS; ++c) {
    const uint32_t col = tid + c * LA_THREADS;
    if (col >= d.rank) break;
    for (uint32_t r = 0; r < nh; ++r) {
      const float v = r == 0 ? acc[0][c] : r == 1 ? acc[1][c] : r == 2 ? acc[2][c] : acc[3][c];
      if (sp.part) sp.part[((size_t)(h0 + r) * sp.splits + split) * sp.ld + col] = v;
      else store_out(d.out, d.out_dtype == CUTB_BF16, tok * d.ldo + (size_t)(h0 + r) * d.rank + col, v / head_l[r]);
    }
  }
  if (sp.part && tid < nh) sp.ml[(size_t)(h0 + tid) * sp.splits + split] = make_float2(head_m[tid], head_l[tid]);
}

LatentSplit split_of(const cutb_latent_attn_desc &d) {
  LatentSplit s{};
  s.splits = latent_splits(d), s.ld = (d.rank + 3) / 4 * 4;
  if (d.n_tokens == 1) {
    s.ml = reinterpret_cast<float2 *>(d.workspace);
    s.part = reinterpret_cast<float *>(d.workspace) + ((size_t)2 * d.n_heads * s.splits + 3) / 4 * 4;
  }
  return s;
}

}  // namespace

uint32_t latent_splits(const cutb_latent_attn_desc &d) {
  if (d.n_tokens != 1) return 1;
  DeviceInfo di;
  const uint32_t sms = get_device_info(&di) == CUTB_OK ? (uint32_t)di.sm_count : 148u, groups = (d.n_heads + LS_HEADS - 1) / LS_HEADS;
  uint32_t s = 2 * sms / groups, most = (d.max_pos + 31) / 32;
  if (s > most) s = most;
  if (s > 64) s = 64;
  return s < 1 ? 1 : s;
}

int latent_kv_write_launch(const cutb_latent_attn_desc &d, cudaStream_t stream) {
  const dim3 grid(d.n_tokens, d.lat && d.cq ? 2 : 1);
  if (d.kv_dtype == CUTB_BF16) CUTB_CUDA_TRY(launch_pdl(latent_kv_write_kernel<__nv_bfloat16>, grid, dim3(128), 0, stream, d));
  else CUTB_CUDA_TRY(launch_pdl(latent_kv_write_kernel<float>, grid, dim3(128), 0, stream, d));
  return CUTB_OK;
}

int latent_attention_launch(const cutb_latent_attn_desc &d, cudaStream_t stream) {
  const LatentSplit sp = split_of(d);
  const uint32_t row_len = d.rot_at + (d.rot_dim + 7) / 8 * 8, smem = 4 * row_len * (LS_HEADS + 1);
  const dim3 grid((d.n_heads + LS_HEADS - 1) / LS_HEADS, sp.splits, d.n_tokens);
  auto go = [&](auto kernel) -> int {
    if (smem > 48 * 1024) CUTB_CUDA_TRY(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    CUTB_CUDA_TRY(launch_pdl(kernel, grid, dim3(LA_THREADS), smem, stream, d, sp, row_len));
    return CUTB_OK;
  };
  return d.kv_dtype == CUTB_BF16 ? go(latent_attention_simt_kernel<__nv_bfloat16>) : go(latent_attention_simt_kernel<float>);
}

int latent_values_launch(const cutb_latent_attn_desc &d, cudaStream_t stream) {
  const LatentSplit sp = split_of(d);
  HeadMvParams h{};
  h.W = d.w_uv, h.C = d.out, h.c_bf16 = d.out_dtype == CUTB_BF16;
  h.batch = d.n_heads, h.K = d.rank, h.K8 = (d.rank + 7) / 8, h.N = d.vdim, h.ldw8 = (uint32_t)d.ld_uv / 8, h.c_batch = d.vdim;
  h.ml = sp.ml, h.part = sp.part, h.splits = sp.splits, h.ld_part = sp.ld;
  return head_matvec_launch(h, stream);
}

bool latent_prefill_supported(const cutb_latent_attn_desc &) { return false; }
int latent_prefill_launch(const cutb_latent_attn_desc &, cudaStream_t) { return CUTB_ERR_UNSUPPORTED; }

}  // namespace cutb
