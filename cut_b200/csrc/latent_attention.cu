// Latent attention over whole-context caches: row p of a cache holds position p's normed latent c and, from column rot_at on, the
// rotated key part that all heads share.  Beside window_attention.cu, whose caches hold keys and values per head.
//
//  * latent_kv_write_kernel: a batch of tokens into the cache, and the norm of the latent queries;
//  * latent_decode_tc_kernel: the absorbed form (every head's query against the cache row itself) over a bf16 cache: one token
//    or a few.  A block takes 16 heads of a token and a share of its keys; the eight blocks of a cluster take neighbouring
//    shares and merge their sums through distributed shared memory.  Products are m16n8k16 warp MMAs; queries and weights enter
//    as the sum of two bf16 terms, so they keep 16 significant bits;
//  * latent_attention_simt_kernel: the same in fp32 arithmetic, for any size and either cache type.
//    For one token the partial sums of the clusters (or blocks) go to memory; the values' mat-vec behind them merges them
//    while it stages its input (head_matvec_kernel);
//  * latent_prefill_tc_kernel: many tokens over expanded keys and values (a GEMM over the cache makes them), bf16.  A block of
//    eight warps owns 128 consecutive tokens of one head; tiles of 64 keys -- the head's own part, and the shared rotated part
//    straight from the cache -- stream through a two-deep cp.async ring, products are m16n8k16 warp MMAs with fp32
//    accumulators, the softmax runs online.  The weights enter the value product as the sum of two bf16 terms.
#include <cooperative_groups.h>
#include <cuda_bf16.h>

#include "attn_common.cuh"
#include "common.cuh"
#include "dense_common.cuh"
#include "kernels.h"

namespace cg = cooperative_groups;

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

// ---- absorbed form on the tensor cores ---------------------------------------------------------------------------------
constexpr int LD_THREADS = 256, LD_WARPS = 8, LD_HEADS = 16, LD_KEYS = 16, LD_STAGES = 3, LD_CLUSTER = 8, LD_PAD = 8;

// shared memory: queries (high and low parts), a ring of key tiles (afterwards the block's sums), the new row.  Below 112 KB two
// blocks share an SM, so that 32 clusters run at once.
__host__ __device__ inline uint32_t ld_stride(uint32_t row_len) { return (row_len + 15) / 16 * 16 + LD_PAD; }
__host__ __device__ inline uint32_t ld_sums_stride(uint32_t rank) { return (rank + 31) / 32 * 32 + 8; }  // (rows eight banks apart)
uint32_t ld_smem_bytes(const cutb_latent_attn_desc &d) {
  const uint32_t st = ld_stride(d.rot_at + (d.rot_dim + 7) / 8 * 8), tiles = LD_STAGES * LD_KEYS * st * 2, sums = LD_HEADS * ld_sums_stride(d.rank) * 4;
  return 2 * LD_HEADS * st * 2 + (tiles > sums ? tiles : sums) + st * 2;
}
bool ld_applies(const cutb_latent_attn_desc &d) { return d.kv_dtype == CUTB_BF16 && d.rank <= 1024 && ld_smem_bytes(d) <= 220 * 1024; }

// NC: 16-column pieces of the latent per warp.  grid = (head groups, shares, tokens), cluster (1, 8, 1).
template <int NC> __global__ void __launch_bounds__(LD_THREADS) latent_decode_tc_kernel(const cutb_latent_attn_desc d, const LatentSplit sp, uint32_t row_len) {
  extern __shared__ __align__(16) uint8_t ld_smem[];
  __shared__ float sc[4][LD_HEADS][LD_KEYS + 1];                        // scores, a quarter of the row each
  __shared__ __align__(16) __nv_bfloat16 ps[2][LD_HEADS][LD_KEYS + 8];  // weights, high and low parts
  __shared__ float head_m[LD_HEADS], head_l[LD_HEADS], fac[LD_HEADS], part[LD_WARPS];
  __shared__ float2 all_ml[LD_CLUSTER][LD_HEADS];  // every block's maxima and weight sums
  cg::cluster_group cluster = cg::this_cluster();
  const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h0 = blockIdx.x * LD_HEADS, split = blockIdx.y, shares = gridDim.y, tok = blockIdx.z;
  const uint32_t nh = min((uint32_t)LD_HEADS, d.n_heads - h0), width = d.dim + d.rot_dim, st = ld_stride(row_len), steps = (st - LD_PAD) / 16;
  __nv_bfloat16 *qh = reinterpret_cast<__nv_bfloat16 *>(ld_smem), *ql = qh + LD_HEADS * st, *tiles = ql + LD_HEADS * st;
  float *sums = reinterpret_cast<float *>(tiles);
  const uint32_t tile_bytes = LD_KEYS * st * 2, tiles_len = LD_STAGES * tile_bytes, sums_ld = ld_sums_stride(d.rank), sums_len = LD_HEADS * sums_ld * 4;
  __nv_bfloat16 *fresh = reinterpret_cast<__nv_bfloat16 *>(reinterpret_cast<uint8_t *>(tiles) + (tiles_len > sums_len ? tiles_len : sums_len));
  const uint32_t qh_u = smem_u32(qh), ql_u = smem_u32(ql), tile_u = smem_u32(tiles), ps_u = smem_u32(ps);
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");
  asm volatile("barrier.cluster.arrive.aligned;" ::: "memory");  // (waited for before the first access to another block)
  pdl_enter();
  const bool split_q = d.qa_high != nullptr;
  if (split_q) {  // the latent parts as they are, asynchronously
    const __nv_bfloat16 *gh = reinterpret_cast<const __nv_bfloat16 *>(d.qa_high) + h0 * d.ld_qa_split, *gl = reinterpret_cast<const __nv_bfloat16 *>(d.qa_low) + h0 * d.ld_qa_split;
    for (uint32_t r = warp; r < LD_HEADS; r += LD_WARPS)
      for (uint32_t c = lane * 8; c < st - LD_PAD; c += 256) {
        const uint32_t at = r * st + c;
        if (r < nh && c < d.rot_at) {
          cp_async16(qh_u + at * 2, gh + r * d.ld_qa_split + c);
          cp_async16(ql_u + at * 2, gl + r * d.ld_qa_split + c);
        } else {
          *reinterpret_cast<uint4 *>(qh + at) = *reinterpret_cast<uint4 *>(ql + at) = make_uint4(0, 0, 0, 0);
        }
      }
  }
  // the first latent parts of the queries (a warp per two heads, eight pairs per lane) are on their way before anything else
  const float *qa0 = d.qa + tok * d.ld_qa + (size_t)h0 * d.rank, *q0 = d.q + tok * d.ldq + (size_t)h0 * width + d.dim;
  constexpr uint32_t QH = LD_HEADS / LD_WARPS;
  float u[QH][4], v[QH][4];
  auto load_q = [&](uint32_t e0) {
#pragma unroll
    for (uint32_t i = 0; i < QH; ++i)
#pragma unroll
      for (uint32_t j = 0; j < 4; ++j) {
        const uint32_t r = warp + i * LD_WARPS, e = e0 + j * 64 + lane * 2;
        const float *qa = qa0 + (size_t)r * d.rank + e;
        u[i][j] = r < nh && e < d.rank ? qa[0] : 0.f, v[i][j] = r < nh && e + 1 < d.rank ? qa[1] : 0.f;
      }
  };
  if (!split_q) load_q(0);
  const uint32_t pos = (d.pos_ptr ? *d.pos_ptr : d.pos) + tok;
  if (pos >= d.max_pos) {  // (the same in every block of the cluster)
    if (d.status && tid == 0) atomicExch(d.status, (int)CUTB_ERR_INVALID);
    cp_async_wait<0>();
    asm volatile("barrier.cluster.wait.aligned;" ::: "memory");
    return;
  }
  const uint32_t n = pos + 1, per = (n + shares - 1) / shares, k_lo = min(split * per, n), k_hi = min(k_lo + per, n);
  const __nv_bfloat16 *cache = reinterpret_cast<const __nv_bfloat16 *>(d.cache);
  const bool make = d.lat && k_hi == n && k_lo < n;  // this block's keys end with the token's own
  const uint32_t pieces = (st - LD_PAD) / 8;
  auto load_tile = [&](uint32_t k0, uint32_t buf) {
    for (uint32_t r = warp; r < LD_KEYS; r += LD_WARPS) {
      const uint32_t key = k0 + r;
      const bool in = key < k_hi && !(make && key == pos);
      const __nv_bfloat16 *src = cache + (size_t)key * d.ld_cache;
      const uint32_t dst = tile_u + buf * tile_bytes + r * st * 2;
      for (uint32_t c = lane; c < pieces; c += 32) {
        if (in && c * 8 < row_len) cp_async16(dst + c * 16, src + c * 8);
        else *reinterpret_cast<uint4 *>(reinterpret_cast<uint8_t *>(tiles) + buf * tile_bytes + r * st * 2 + c * 16) = make_uint4(0, 0, 0, 0);
      }
    }
  };
#pragma unroll
  for (uint32_t i = 0; i + 1 < LD_STAGES; ++i) {
    if (k_lo + i * LD_KEYS < k_hi) load_tile(k_lo + i * LD_KEYS, i);
    cp_async_commit();
  }

  // queries laid out as a cache row, scaled to log2 units, zeros in its gaps and past the last head
  const float scale = d.scale * LA_LOG2E;
  const uint32_t half = d.rot_dim / 2;
  auto put_q = [&](uint32_t r, uint32_t e, float u, float v) {
    uint32_t hi, lo;
    split_bf16(u, v, hi, lo);
    *reinterpret_cast<uint32_t *>(qh + r * st + e) = hi;
    *reinterpret_cast<uint32_t *>(ql + r * st + e) = lo;
  };
  constexpr int RU = 2;
  float ra[RU], rb[RU], rc[RU], rs[RU];
#pragma unroll
  for (int u = 0; u < RU; ++u) {
    const uint32_t i = tid + u * LD_THREADS, r = half ? i / half : 0, e = half ? i - r * half : 0;
    const bool in = half && r < nh;
    ra[u] = in ? q0[(size_t)r * width + 2 * e] : 0.f, rb[u] = in ? q0[(size_t)r * width + 2 * e + 1] : 0.f;
    rc[u] = in ? __ldg(d.cos_table + (size_t)pos * half + e) : 0.f, rs[u] = in ? __ldg(d.sin_table + (size_t)pos * half + e) : 0.f;
  }
  for (uint32_t e0 = 0; e0 < st - LD_PAD && !split_q; e0 += 256) {
    if (e0) load_q(e0);
#pragma unroll
    for (uint32_t i = 0; i < QH; ++i)
#pragma unroll
      for (uint32_t j = 0; j < 4; ++j) {
        const uint32_t e = e0 + j * 64 + lane * 2;
        if (e < st - LD_PAD) put_q(warp + i * LD_WARPS, e, u[i][j] * scale, v[i][j] * scale);
      }
  }
  __syncthreads();  // (the turned part overwrites zeros)
#pragma unroll
  for (int u = 0; u < RU; ++u) {
    const uint32_t i = tid + u * LD_THREADS, r = half ? i / half : 0, e = half ? i - r * half : 0;
    if (half && r < nh) put_q(r, d.rot_at + 2 * e, (ra[u] * rc[u] - rb[u] * rs[u]) * scale, (rb[u] * rc[u] + ra[u] * rs[u]) * scale);
  }
  for (uint32_t i = tid + RU * LD_THREADS; i < nh * half; i += LD_THREADS) {
    const uint32_t r = i / half, e = i - r * half;
    const float c = __ldg(d.cos_table + (size_t)pos * half + e), s = __ldg(d.sin_table + (size_t)pos * half + e);
    const float a = q0[(size_t)r * width + 2 * e], b = q0[(size_t)r * width + 2 * e + 1];
    put_q(r, d.rot_at + 2 * e, (a * c - b * s) * scale, (b * c + a * s) * scale);
  }
  if (make) {
    __nv_bfloat16 *row = reinterpret_cast<__nv_bfloat16 *>(d.cache) + pos * d.ld_cache;
    for (uint32_t i = tid; i < st; i += LD_THREADS) fresh[i] = __float2bfloat16_rn(0.f);
    __syncthreads();
    make_cache_row(d, tok, pos, part, [&](uint32_t i, float v) {
      fresh[i] = __float2bfloat16_rn(v);
      if (blockIdx.x == 0) row[i] = fresh[i];
    });
  }
  if (tid < LD_HEADS) {
    const bool sink = d.sink && split == 0 && tid < nh;
    head_m[tid] = sink ? d.sink[h0 + tid] * LA_LOG2E : LA_NEG, head_l[tid] = sink ? 1.f : 0.f;
  }
  const uint32_t g = lane >> 2, tg = lane & 3, mat = lane >> 3, mr = lane & 7;
  float o[2 * NC][4];
#pragma unroll
  for (int j = 0; j < 2 * NC; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
  const uint32_t col0 = warp * NC * 16;  // this warp's columns of the latent
  const uint32_t s_part = warp >> 1, s_n = warp & 1;  // and its part of the scores: a quarter of the row, eight keys
  const uint32_t s_first = steps * s_part / 4, s_last = steps * (s_part + 1) / 4;

  for (uint32_t k0 = k_lo, turn = 0; k0 < k_hi; k0 += LD_KEYS, ++turn) {
    const uint32_t buf = turn % LD_STAGES, cnt = min((uint32_t)LD_KEYS, k_hi - k0);
    if (k0 + (LD_STAGES - 1) * LD_KEYS < k_hi) load_tile(k0 + (LD_STAGES - 1) * LD_KEYS, (turn + LD_STAGES - 1) % LD_STAGES);
    cp_async_commit();
    cp_async_wait<LD_STAGES - 1>();
    __syncthreads();
    if (make && pos - k0 < cnt) {  // the row made here
      for (uint32_t c = tid; c < pieces; c += LD_THREADS)
        *reinterpret_cast<uint4 *>(reinterpret_cast<uint8_t *>(tiles) + buf * tile_bytes + (pos - k0) * st * 2 + c * 16) = reinterpret_cast<const uint4 *>(fresh)[c];
      __syncthreads();
    }
    const uint32_t t_u = tile_u + buf * tile_bytes;
    {  // scores of 16 heads x 8 keys over a quarter of the row; high and low query parts in sums of their own
      float s0[4] = {}, s1[4] = {};
      const uint32_t a_off = ((mat & 1) * 8 + mr) * st + (mat >> 1) * 8, b_off = (s_n * 8 + mr) * st + mat * 8;
      uint32_t k = s_first;
      for (; k + 1 < s_last; k += 2) {
        uint32_t ah[4], al[4], b0, b1, b2, b3;
        ldsm_x4(t_u + (b_off + k * 16) * 2, b0, b1, b2, b3);
        ldsm_x4(qh_u + (a_off + k * 16) * 2, ah[0], ah[1], ah[2], ah[3]);
        ldsm_x4(ql_u + (a_off + k * 16) * 2, al[0], al[1], al[2], al[3]);
        mma_bf16(s0, ah, b0, b1);
        mma_bf16(s1, al, b0, b1);
        ldsm_x4(qh_u + (a_off + k * 16 + 16) * 2, ah[0], ah[1], ah[2], ah[3]);
        ldsm_x4(ql_u + (a_off + k * 16 + 16) * 2, al[0], al[1], al[2], al[3]);
        mma_bf16(s0, ah, b2, b3);
        mma_bf16(s1, al, b2, b3);
      }
      if (k < s_last) {
        uint32_t ah[4], al[4], b0, b1, b2, b3;
        // (lanes 16 and up would address past the last step: they repeat the first half's rows)
        ldsm_x4(t_u + ((s_n * 8 + mr) * st + (mat & 1) * 8 + k * 16) * 2, b0, b1, b2, b3);
        ldsm_x4(qh_u + (a_off + k * 16) * 2, ah[0], ah[1], ah[2], ah[3]);
        ldsm_x4(ql_u + (a_off + k * 16) * 2, al[0], al[1], al[2], al[3]);
        mma_bf16(s0, ah, b0, b1);
        mma_bf16(s1, al, b0, b1);
      }
      const uint32_t c = s_n * 8 + 2 * tg;
      sc[s_part][g][c] = s0[0] + s1[0], sc[s_part][g][c + 1] = s0[1] + s1[1];
      sc[s_part][g + 8][c] = s0[2] + s1[2], sc[s_part][g + 8][c + 1] = s0[3] + s1[3];
    }
    __syncthreads();
    {  // softmax: half a warp per head, a lane per key
      static_assert(LD_KEYS == 16 && LD_HEADS == 2 * LD_WARPS, "a head per 16 lanes");
      const uint32_t r = warp * 2 + (lane >> 4), key = lane & 15;
      const float x = key < cnt ? (sc[0][r][key] + sc[1][r][key]) + (sc[2][r][key] + sc[3][r][key]) : -INFINITY, before = head_m[r];
      float m = fmaxf(x, before);
#pragma unroll
      for (int w = 8; w > 0; w >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, w));
      const float e = exp2f(x - m);
      float l = e;
#pragma unroll
      for (int w = 8; w > 0; w >>= 1) l += __shfl_xor_sync(0xffffffffu, l, w);
      const __nv_bfloat16 hi = __float2bfloat16_rn(e);
      ps[0][r][key] = hi;
      ps[1][r][key] = __float2bfloat16_rn(e - __bfloat162float(hi));
      __syncwarp();
      if (key == 0) {
        const float f = exp2f(before - m);
        head_l[r] = fmaf(head_l[r], f, l), head_m[r] = m, fac[r] = f;
      }
    }
    __syncthreads();
    if (col0 < d.rank) {
      const float f_lo = fac[g], f_hi = fac[g + 8];
#pragma unroll
      for (int j = 0; j < 2 * NC; ++j) o[j][0] *= f_lo, o[j][1] *= f_lo, o[j][2] *= f_hi, o[j][3] *= f_hi;
#pragma unroll
      for (int kk = 0; kk < LD_KEYS / 16; ++kk) {
        uint32_t ph[4], pl[4];
        const uint32_t a_off = ((mat & 1) * 8 + mr) * (LD_KEYS + 8) + kk * 16 + (mat >> 1) * 8;
        ldsm_x4(ps_u + a_off * 2, ph[0], ph[1], ph[2], ph[3]);
        ldsm_x4(ps_u + (LD_HEADS * (LD_KEYS + 8) + a_off) * 2, pl[0], pl[1], pl[2], pl[3]);
#pragma unroll
        for (int j2 = 0; j2 < NC; ++j2) {
          const uint32_t row = kk * 16 + (mat & 1) * 8 + mr, col = col0 + j2 * 16 + (mat >> 1) * 8;
          if (col0 + j2 * 16 < d.rank) {
            uint32_t b0, b1, b2, b3;
            ldsm_x4_trans(t_u + (row * st + col) * 2, b0, b1, b2, b3);
            mma_bf16(o[2 * j2], ph, b0, b1);
            mma_bf16(o[2 * j2 + 1], ph, b2, b3);
            mma_bf16(o[2 * j2], pl, b0, b1);
            mma_bf16(o[2 * j2 + 1], pl, b2, b3);
          }
        }
      }
    }
    __syncthreads();  // the tile is free for the copy issued next turn
  }

  // the block's sums, then the cluster's; maxima and weight sums go to every block
  cp_async_wait<0>();
  __syncthreads();
#pragma unroll
  for (int j = 0; j < 2 * NC; ++j) {
    const uint32_t c = col0 + j * 8 + 2 * tg;
    if (c < d.rank) {
      *reinterpret_cast<float2 *>(sums + g * sums_ld + c) = make_float2(o[j][0], o[j][1]);
      *reinterpret_cast<float2 *>(sums + (g + 8) * sums_ld + c) = make_float2(o[j][2], o[j][3]);
    }
  }
  asm volatile("barrier.cluster.wait.aligned;" ::: "memory");
  if (tid < LD_CLUSTER * LD_HEADS) {
    const uint32_t r = tid % LD_HEADS;
    *cluster.map_shared_rank(&all_ml[cluster.block_rank()][r], tid / LD_HEADS) = make_float2(head_m[r], head_l[r]);
  }
  cluster.sync();
  const uint32_t me = cluster.block_rank(), out_split = split / LD_CLUSTER, out_splits = shares / LD_CLUSTER;
  const uint32_t quads = (d.rank + 3) / 4;
  for (uint32_t i = me * LD_THREADS + tid; i < nh * quads; i += LD_CLUSTER * LD_THREADS) {
    const uint32_t r = i / quads, c = i % quads * 4;
    float m = LA_NEG, l = 0.f;
    float4 ak[LD_CLUSTER], s = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (uint32_t k = 0; k < LD_CLUSTER; ++k)  // every remote read in flight at once
      ak[k] = *reinterpret_cast<const float4 *>(cluster.map_shared_rank(&sums[r * sums_ld + c], k));
#pragma unroll
    for (uint32_t k = 0; k < LD_CLUSTER; ++k) m = fmaxf(m, all_ml[k][r].x);
#pragma unroll
    for (uint32_t k = 0; k < LD_CLUSTER; ++k) {
      const float w = exp2f(all_ml[k][r].x - m);
      l = fmaf(w, all_ml[k][r].y, l);
      s.x = fmaf(w, ak[k].x, s.x), s.y = fmaf(w, ak[k].y, s.y), s.z = fmaf(w, ak[k].z, s.z), s.w = fmaf(w, ak[k].w, s.w);
    }
    if (sp.part) {
      *reinterpret_cast<float4 *>(sp.part + ((size_t)(h0 + r) * out_splits + out_split) * sp.ld + c) = s;
      if (c == 0) sp.ml[(size_t)(h0 + r) * out_splits + out_split] = make_float2(m, l);
    } else {
      const float inv = 1.0f / l, v[4] = {s.x * inv, s.y * inv, s.z * inv, s.w * inv};
#pragma unroll
      for (int e = 0; e < 4; ++e)
        if (c + e < d.rank) store_out(d.out, d.out_dtype == CUTB_BF16, tok * d.ldo + (size_t)(h0 + r) * d.rank + c + e, v[e]);
    }
  }
  cluster.sync();  // nobody leaves while its shared memory may still be read
}

// ---- expanded form on the tensor cores ---------------------------------------------------------------------------------
constexpr int LP_BM = 128, LP_BN = 64, LP_THREADS = 256, LP_PAD = 8;

template <int DK, int DV> __global__ void __launch_bounds__(LP_THREADS, 1) latent_prefill_tc_kernel(const cutb_latent_attn_desc d) {
  constexpr int LK = DK + LP_PAD, LV = DV + LP_PAD, KS = DK / 16, KC = DK / 8, VC = DV / 8;
  constexpr uint32_t KT = LP_BN * LK * 2, VT = LP_BN * LV * 2;
  constexpr bool Q_IN_REGS = DK <= 128;
  extern __shared__ __align__(16) uint8_t lp_smem[];
  __nv_bfloat16 *Qs = reinterpret_cast<__nv_bfloat16 *>(lp_smem);
  const uint32_t qs_u = smem_u32(lp_smem), k_u = qs_u + LP_BM * LK * 2, v_u = k_u + 2 * KT;

  const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  // later tokens (which see more keys) first
  const uint32_t tok0 = (gridDim.y - 1 - blockIdx.y) * LP_BM, h = blockIdx.x;
  pdl_enter();
  const uint32_t p0 = (d.pos_ptr ? *d.pos_ptr : d.pos) + tok0, ntok = min((uint32_t)LP_BM, d.n_tokens - tok0);
  if (p0 + ntok > d.max_pos) {  // no table rows: the cache write has done nothing for them either
    if (d.status && tid == 0 && h == 0) atomicExch(d.status, (int)CUTB_ERR_INVALID);
    return;
  }
  const uint32_t p_last = p0 + ntok - 1, t_end = p_last / LP_BN + 1, width = d.dim + d.rot_dim;
  const __nv_bfloat16 *kbase = reinterpret_cast<const __nv_bfloat16 *>(d.k_exp) + (size_t)h * d.dim;
  const __nv_bfloat16 *vbase = reinterpret_cast<const __nv_bfloat16 *>(d.v_exp) + (size_t)h * d.vdim;
  const __nv_bfloat16 *rbase = reinterpret_cast<const __nv_bfloat16 *>(d.cache) + d.rot_at;
  // Keys past the block's last token are zero (a weight of zero times a stray NaN would not be); so are columns past the head's.
  auto load_tile = [&](uint32_t t, uint32_t buf) {
    const uint32_t key0 = t * LP_BN;
#pragma unroll
    for (uint32_t i = tid; i < LP_BN * KC; i += LP_THREADS) {
      const uint32_t r = i / KC, c = i % KC * 8, key = key0 + r;
      const __nv_bfloat16 *src = c < d.dim ? kbase + key * d.ld_k + c : rbase + key * d.ld_cache + (c - d.dim);
      const uint32_t off = buf * KT + (r * LK + c) * 2;
      if (key <= p_last && c < width) cp_async16(k_u + off, src);
      else *reinterpret_cast<uint4 *>(lp_smem + (k_u - qs_u) + off) = make_uint4(0, 0, 0, 0);
    }
#pragma unroll
    for (uint32_t i = tid; i < LP_BN * VC; i += LP_THREADS) {
      const uint32_t r = i / VC, c = i % VC * 8, key = key0 + r;
      const uint32_t off = buf * VT + (r * LV + c) * 2;
      if (key <= p_last && c < d.vdim) cp_async16(v_u + off, vbase + key * d.ld_v + c);
      else *reinterpret_cast<uint4 *>(lp_smem + (v_u - qs_u) + off) = make_uint4(0, 0, 0, 0);
    }
    cp_async_commit();
  };
  load_tile(0, 0);

  // queries: the rotated part turned at their own positions, rounded to bf16; pairs of neighbours
  {
    constexpr uint32_t PP = DK / 2;
    const float *q0 = d.q + (size_t)tok0 * d.ldq + (size_t)h * width;
    const uint32_t half = d.rot_dim / 2;
#pragma unroll 4
    for (uint32_t i = tid; i < LP_BM * PP; i += LP_THREADS) {
      const uint32_t r = i / PP, e = i % PP * 2, rc = min(r, ntok - 1);  // (rows past the last token repeat it)
      float u = 0.f, v = 0.f;
      if (e < width) {
        u = __ldg(q0 + rc * d.ldq + e), v = __ldg(q0 + rc * d.ldq + e + 1);
        if (e >= d.dim) {
          const size_t at = (size_t)(p0 + rc) * half + (e - d.dim) / 2;
          const float c = __ldg(d.cos_table + at), s = __ldg(d.sin_table + at), u0 = u;
          u = u0 * c - v * s, v = v * c + u0 * s;
        }
      }
      *reinterpret_cast<uint32_t *>(Qs + r * LK + e) = pack_bf16(u, v);
    }
  }
  __syncthreads();

  const uint32_t g = lane >> 2, tg = lane & 3, mat = lane >> 3, mr = lane & 7;
  const uint32_t q_row = warp * 16 + (mat & 1) * 8 + mr;
  uint32_t qa[Q_IN_REGS ? KS : 1][4];
  if constexpr (Q_IN_REGS) {
#pragma unroll
    for (int ks = 0; ks < KS; ++ks) ldsm_x4(qs_u + (q_row * LK + ks * 16 + (mat >> 1) * 8) * 2, qa[ks][0], qa[ks][1], qa[ks][2], qa[ks][3]);
  }
  const uint32_t row_lo = warp * 16 + g, row_hi = row_lo + 8;
  const uint32_t pos_lo = p0 + row_lo, pos_hi = p0 + row_hi;          // (rows past ntok compute and are not stored)
  const uint32_t wp_first = p0 + warp * 16, wp_last = wp_first + 15;  // this warp's positions
  const float scale_log2 = d.scale * LA_LOG2E;

  float o[DV / 8][4];
#pragma unroll
  for (int j = 0; j < DV / 8; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
  // running maxima (log2 units) and sums; a sink is a key without a value seen before all others
  const float sink = d.sink ? __ldg(d.sink + h) * LA_LOG2E : LA_NEG;
  float m_lo = sink, m_hi = sink, l_lo = 0.f, l_hi = 0.f;

  for (uint32_t t = 0; t < t_end; ++t) {
    const uint32_t buf = t & 1;
    if (t + 1 < t_end) {
      load_tile(t + 1, buf ^ 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    const uint32_t kt_u = k_u + buf * KT, vt_u = v_u + buf * VT, key0 = t * LP_BN;
    if (key0 <= wp_last) {  // this warp sees the tile
      float s[LP_BN / 8][4];
#pragma unroll
      for (int j = 0; j < LP_BN / 8; ++j) s[j][0] = s[j][1] = s[j][2] = s[j][3] = 0.f;
#pragma unroll
      for (int ks = 0; ks < KS; ++ks) {
        uint32_t (&a)[4] = qa[Q_IN_REGS ? ks : 0];
        if constexpr (!Q_IN_REGS) ldsm_x4(qs_u + (q_row * LK + ks * 16 + (mat >> 1) * 8) * 2, a[0], a[1], a[2], a[3]);
#pragma unroll
        for (int j2 = 0; j2 < LP_BN / 16; ++j2) {
          const uint32_t row = j2 * 16 + (mat >> 1) * 8 + mr, col = ks * 16 + (mat & 1) * 8;
          uint32_t b0, b1, b2, b3;
          ldsm_x4(kt_u + (row * LK + col) * 2, b0, b1, b2, b3);
          mma_bf16(s[2 * j2], a, b0, b1);
          mma_bf16(s[2 * j2 + 1], a, b2, b3);
        }
      }
      float mx_lo = LA_NEG, mx_hi = LA_NEG;
      const bool all = key0 + LP_BN - 1 <= wp_first;  // every key seen by every token of the warp
#pragma unroll
      for (int j = 0; j < LP_BN / 8; ++j) {
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const uint32_t key = key0 + j * 8 + 2 * tg + (e & 1), pos = e < 2 ? pos_lo : pos_hi;
          const float v = all || key <= pos ? s[j][e] * scale_log2 : -INFINITY;
          s[j][e] = v;
          if (e < 2) mx_lo = fmaxf(mx_lo, v);
          else mx_hi = fmaxf(mx_hi, v);
        }
      }
      mx_lo = fmaxf(mx_lo, __shfl_xor_sync(0xffffffffu, mx_lo, 1));
      mx_lo = fmaxf(mx_lo, __shfl_xor_sync(0xffffffffu, mx_lo, 2));
      mx_hi = fmaxf(mx_hi, __shfl_xor_sync(0xffffffffu, mx_hi, 1));
      mx_hi = fmaxf(mx_hi, __shfl_xor_sync(0xffffffffu, mx_hi, 2));
      const float mn_lo = fmaxf(m_lo, mx_lo), mn_hi = fmaxf(m_hi, mx_hi);
      const float al_lo = exp2f(m_lo - mn_lo), al_hi = exp2f(m_hi - mn_hi);
      m_lo = mn_lo, m_hi = mn_hi;
      float sum_lo = 0.f, sum_hi = 0.f;
#pragma unroll
      for (int j = 0; j < LP_BN / 8; ++j) {
        s[j][0] = exp2f(s[j][0] - m_lo), s[j][1] = exp2f(s[j][1] - m_lo);
        s[j][2] = exp2f(s[j][2] - m_hi), s[j][3] = exp2f(s[j][3] - m_hi);
        sum_lo += s[j][0] + s[j][1];
        sum_hi += s[j][2] + s[j][3];
      }
      l_lo = l_lo * al_lo + sum_lo, l_hi = l_hi * al_hi + sum_hi;
#pragma unroll
      for (int j = 0; j < DV / 8; ++j) o[j][0] *= al_lo, o[j][1] *= al_lo, o[j][2] *= al_hi, o[j][3] *= al_hi;
#pragma unroll
      for (int kk = 0; kk < LP_BN / 16; ++kk) {
        uint32_t ph[4], pl[4];
        split_bf16(s[2 * kk][0], s[2 * kk][1], ph[0], pl[0]);
        split_bf16(s[2 * kk][2], s[2 * kk][3], ph[1], pl[1]);
        split_bf16(s[2 * kk + 1][0], s[2 * kk + 1][1], ph[2], pl[2]);
        split_bf16(s[2 * kk + 1][2], s[2 * kk + 1][3], ph[3], pl[3]);
#pragma unroll
        for (int jd2 = 0; jd2 < DV / 16; ++jd2) {
          const uint32_t row = kk * 16 + (mat & 1) * 8 + mr, col = jd2 * 16 + (mat >> 1) * 8;
          uint32_t b0, b1, b2, b3;
          ldsm_x4_trans(vt_u + (row * LV + col) * 2, b0, b1, b2, b3);
          mma_bf16(o[2 * jd2], ph, b0, b1);
          mma_bf16(o[2 * jd2 + 1], ph, b2, b3);
          mma_bf16(o[2 * jd2], pl, b0, b1);
          mma_bf16(o[2 * jd2 + 1], pl, b2, b3);
        }
      }
    }
    __syncthreads();  // the tile is free for the copy issued two turns from now
  }

  l_lo += __shfl_xor_sync(0xffffffffu, l_lo, 1);
  l_lo += __shfl_xor_sync(0xffffffffu, l_lo, 2);
  l_hi += __shfl_xor_sync(0xffffffffu, l_hi, 1);
  l_hi += __shfl_xor_sync(0xffffffffu, l_hi, 2);
  if (d.sink) l_lo += exp2f(sink - m_lo), l_hi += exp2f(sink - m_hi);
  const float inv_lo = 1.0f / l_lo, inv_hi = 1.0f / l_hi;
#pragma unroll
  for (int j = 0; j < DV / 8; ++j) {
    const uint32_t c = 8 * j + 2 * tg;
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const uint32_t r = e < 2 ? row_lo : row_hi, cc = c + (e & 1);
      if (r < ntok && cc < d.vdim)
        store_out(d.out, d.out_dtype == CUTB_BF16, (size_t)(tok0 + r) * d.ldo + (size_t)h * d.vdim + cc, o[j][e] * (e < 2 ? inv_lo : inv_hi));
    }
  }
}

template <int DK, int DV> int lp_launch(const cutb_latent_attn_desc &d, cudaStream_t stream) {
  constexpr size_t smem = ((size_t)(LP_BM + 2 * LP_BN) * (DK + LP_PAD) + (size_t)2 * LP_BN * (DV + LP_PAD)) * 2;
  CUTB_CUDA_TRY(cudaFuncSetAttribute(latent_prefill_tc_kernel<DK, DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  CUTB_CUDA_TRY(launch_pdl(latent_prefill_tc_kernel<DK, DV>, dim3(d.n_heads, (d.n_tokens + LP_BM - 1) / LP_BM), dim3(LP_THREADS), smem, stream, d));
  return CUTB_OK;
}
template <int DV> int lp_dispatch(const cutb_latent_attn_desc &d, cudaStream_t stream) {
  const uint32_t width = d.dim + d.rot_dim;
  if constexpr (DV <= 128) {
    if (width <= 64) return lp_launch<64, DV>(d, stream);
    if (width <= 128) return lp_launch<128, DV>(d, stream);
    if (width <= 192) return lp_launch<192, DV>(d, stream);
  }
  return lp_launch<256, DV>(d, stream);
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

template <int NC> int ld_launch(const cutb_latent_attn_desc &d, const LatentSplit &sp, uint32_t row_len, cudaStream_t stream) {
  const uint32_t smem = ld_smem_bytes(d);
  CUTB_CUDA_TRY(cudaFuncSetAttribute(latent_decode_tc_kernel<NC>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3((d.n_heads + LD_HEADS - 1) / LD_HEADS, sp.splits * LD_CLUSTER, d.n_tokens);
  cfg.blockDim = dim3(LD_THREADS);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = stream;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = 1;
  attr[0].val.clusterDim.y = LD_CLUSTER;
  attr[0].val.clusterDim.z = 1;
  attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[1].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = 2;
  CUTB_CUDA_TRY(cudaLaunchKernelEx(&cfg, latent_decode_tc_kernel<NC>, d, sp, row_len));
  return CUTB_OK;
}

}  // namespace

bool latent_takes_split_queries(const cutb_latent_attn_desc &d) { return d.n_tokens == 1 && ld_applies(d); }

uint32_t latent_splits(const cutb_latent_attn_desc &d) {
  if (d.n_tokens != 1) return 1;
  DeviceInfo di;
  const uint32_t sms = get_device_info(&di) == CUTB_OK ? (uint32_t)di.sm_count : 148u;
  if (ld_applies(d)) {  // clusters per head group: as many as run at once, at least 16 keys per block at the full context
    const uint32_t groups = (d.n_heads + LD_HEADS - 1) / LD_HEADS;
    uint32_t s = (2 * sms > 40 ? 2 * sms - 40 : 1) / (groups * LD_CLUSTER), most = (d.max_pos + 16 * LD_CLUSTER - 1) / (16 * LD_CLUSTER);
    if (s > most) s = most;
    if (s > 16) s = 16;
    return s < 1 ? 1 : s;
  }
  const uint32_t groups = (d.n_heads + LS_HEADS - 1) / LS_HEADS;
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
  if (ld_applies(d)) {
    if (d.rank <= 128) return ld_launch<1>(d, sp, row_len, stream);
    if (d.rank <= 256) return ld_launch<2>(d, sp, row_len, stream);
    return d.rank <= 512 ? ld_launch<4>(d, sp, row_len, stream) : ld_launch<8>(d, sp, row_len, stream);
  }
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

bool latent_prefill_supported(const cutb_latent_attn_desc &d) {
  return d.kv_dtype == CUTB_BF16 && d.dim % 8 == 0 && d.rot_dim % 8 == 0 && d.vdim % 8 == 0 && d.vdim > 0 && d.dim + d.rot_dim > 0 &&
         d.dim + d.rot_dim <= 256 && d.vdim <= 256 && d.n_heads <= 0x7fffffffu && (d.n_tokens + LP_BM - 1) / LP_BM <= 65535;
}

int latent_prefill_launch(const cutb_latent_attn_desc &d, cudaStream_t stream) {
  if (d.vdim <= 64) return lp_dispatch<64>(d, stream);
  return d.vdim <= 128 ? lp_dispatch<128>(d, stream) : lp_dispatch<256>(d, stream);
}

}  // namespace cutb
