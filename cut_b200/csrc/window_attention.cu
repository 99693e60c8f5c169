// Sliding-window attention over ring caches (position p in row p % ring_rows), with rotary embedding of part of a head,
// mixing of the values with another layer's, and an optional sink in the softmax.  Beside attention.cu / attention_prefill.cu,
// which serve the llama path (whole-context caches, half-split rotation of the whole head).
//
//  * window_kv_write_kernel: a batch of tokens into the ring;
//  * window_attention_tc_kernel: prefill with a bf16 cache.  A block of four warps owns 64 consecutive tokens of one query
//    head; only the key tiles that some token of the block sees are visited, and a warp skips those its own 16 tokens do not
//    see.  K / V tiles of 64 ring rows stream through a two-deep cp.async ring (a tile never wraps: ring_rows is a multiple of
//    64 and tiles are aligned), products are m16n8k16 warp MMAs with fp32 accumulators, the softmax runs online.  The weights
//    enter the value product as the sum of two bf16 terms, so they keep 16 significant bits;
//  * window_attention_simt_kernel: the same in fp32 arithmetic, one warp per (token, head);
//  * window_attention_decode_kernel: one token.  The slices of the window are the blocks of a cluster; every block rotates
//    its query heads itself, the first slice takes the new token's key and value from registers of this step and stores them
//    to the ring (its row holds a key outside the window), and the slices meet through distributed shared memory.
#include <cooperative_groups.h>
#include <cuda_bf16.h>

#include "attn_common.cuh"
#include "common.cuh"
#include "dense_common.cuh"
#include "kernels.h"

namespace cg = cooperative_groups;

namespace cutb {
namespace {

constexpr float WA_NEG = -1e30f;

// element e of a head after rotation at table row `pos`
__device__ __forceinline__ float rotated(const float *x, uint32_t e, uint32_t pos, const cutb_window_attn_desc &d) {
  const float v = x[e];
  if (e >= d.rot_dims) return v;
  const uint32_t half = d.rot_dims / 2;
  uint32_t i, other;
  bool second;
  if (d.rot_pairing) i = e >> 1, second = e & 1, other = e ^ 1u;
  else second = e >= half, i = second ? e - half : e, other = second ? e - half : e + half;
  const float c = __ldg(d.cos_table + (size_t)pos * half + i), s = __ldg(d.sin_table + (size_t)pos * half + i), o = x[other];
  return second ? v * c + o * s : v * c - o * s;
}

// Elements of a head two at a time: pair i < rot_dims / 2 is rotated, the others are (2 i, 2 i + 1) as they are.
struct Pair {
  uint32_t e0, e1;
  float x0, x1, c, s;
};
__device__ __forceinline__ Pair load_pair(const float *x, uint32_t i, uint32_t pos, const cutb_window_attn_desc &d) {
  Pair r;
  const uint32_t half = d.rot_dims / 2;
  const bool rot = i < half;
  r.e0 = d.rot_pairing || !rot ? 2 * i : i, r.e1 = d.rot_pairing || !rot ? 2 * i + 1 : i + half;
  r.x0 = r.e0 < d.dim ? __ldg(x + r.e0) : 0.f, r.x1 = r.e1 < d.dim ? __ldg(x + r.e1) : 0.f;
  r.c = rot ? __ldg(d.cos_table + (size_t)pos * half + i) : 1.f, r.s = rot ? __ldg(d.sin_table + (size_t)pos * half + i) : 0.f;
  return r;
}

__device__ __forceinline__ float mixed_value(const cutb_window_attn_desc &d, uint32_t tok, uint32_t i) {
  const float v = d.v[tok * d.ldqkv + i];
  if (d.v_first_out) d.v_first_out[tok * d.ld_first + i] = v;
  return d.v_first ? (1.0f - d.v_mix) * v + d.v_mix * d.v_first[tok * d.ld_first + i] : v;
}

template <typename KV> __global__ void __launch_bounds__(256) window_kv_write_kernel(const cutb_window_attn_desc d) {
  pdl_enter();
  const uint32_t tok = blockIdx.x, pos = (d.pos_ptr ? *d.pos_ptr : d.pos) + tok;
  if (pos >= d.max_pos) {  // no table row: record it and write nothing
    if (d.status && threadIdx.x == 0) atomicExch(d.status, (int)CUTB_ERR_INVALID);
    return;
  }
  const size_t row = pos % d.ring_rows;
  KV *kc = reinterpret_cast<KV *>(d.k_cache) + row * d.n_kv_heads * d.k_head;
  KV *vc = reinterpret_cast<KV *>(d.v_cache) + row * d.n_kv_heads * d.v_head;
  const uint32_t pairs = d.k_head / 2;
  for (uint32_t i = threadIdx.x; i < d.n_kv_heads * pairs; i += 256) {
    const uint32_t g = i / pairs;
    const Pair x = load_pair(d.k + tok * d.ldqkv + g * d.dim, i - g * pairs, pos, d);  // (zeros past the head's elements)
    KV *dst = kc + g * d.k_head;
    kv_put(dst + x.e0, x.x0 * x.c - x.x1 * x.s);
    kv_put(dst + x.e1, x.x1 * x.c + x.x0 * x.s);
  }
  for (uint32_t i = threadIdx.x; i < d.n_kv_heads * d.vdim; i += 256) kv_put(vc + i / d.vdim * d.v_head + i % d.vdim, mixed_value(d, tok, i));
}

// ---- prefill on the tensor cores -----------------------------------------------------------------------------------
constexpr int WT_BM = 64, WT_BN = 64, WT_THREADS = 128, WT_PAD = 8;

template <int DK, int DV> __global__ void __launch_bounds__(WT_THREADS) window_attention_tc_kernel(const cutb_window_attn_desc d) {
  constexpr int LK = DK + WT_PAD, LV = DV + WT_PAD, KS = DK / 16;
  constexpr uint32_t KT = WT_BN * LK * 2, VT = WT_BN * LV * 2;
  extern __shared__ __align__(16) uint8_t wt_smem[];
  __nv_bfloat16 *Qs = reinterpret_cast<__nv_bfloat16 *>(wt_smem);
  const uint32_t qs_u = smem_u32(wt_smem), k_u = qs_u + WT_BM * LK * 2, v_u = k_u + 2 * KT;

  const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
  // later tokens (which see a full window) first
  const uint32_t tok0 = (gridDim.x - 1 - blockIdx.x) * WT_BM, h = blockIdx.y, G = d.n_kv_heads, kvh = h / (d.n_heads / G);
  pdl_enter();
  const uint32_t p0 = (d.pos_ptr ? *d.pos_ptr : d.pos) + tok0, ntok = min((uint32_t)WT_BM, d.n_tokens - tok0);
  if (p0 + ntok > d.max_pos) {  // no table rows: the cache write has done nothing for them either
    if (d.status && tid == 0 && h == 0) atomicExch(d.status, (int)CUTB_ERR_INVALID);
    return;
  }
  const uint32_t p_last = p0 + ntok - 1, key_lo = p0 + 1 > d.window ? p0 + 1 - d.window : 0;
  const uint32_t t_first = key_lo / WT_BN, t_end = p_last / WT_BN + 1;

  const __nv_bfloat16 *kbase = reinterpret_cast<const __nv_bfloat16 *>(d.k_cache) + (size_t)kvh * d.k_head;
  const __nv_bfloat16 *vbase = reinterpret_cast<const __nv_bfloat16 *>(d.v_cache) + (size_t)kvh * d.v_head;
  const size_t kld = (size_t)G * d.k_head, vld = (size_t)G * d.v_head;
  // Keys nobody in the block sees are zero (a weight of zero times a stray NaN would not be); columns past the head's
  // elements are zeroed once and never written again.
  constexpr uint32_t KC = DK / 8, VC = DV / 8, KR = WT_THREADS / KC, VR = WT_THREADS / VC;  // 16-byte pieces per row, rows per pass
  const uint32_t kr0 = tid / KC, kc = tid % KC, vr0 = tid / VC, vc = tid % VC;
  const bool k_live = kc * 8 < d.k_head, v_live = vc * 8 < d.v_head;
  auto load_tile = [&](uint32_t t, uint32_t buf) {
    const uint32_t ring0 = (t * WT_BN) % d.ring_rows;
    const bool whole = t * WT_BN >= key_lo && t * WT_BN + WT_BN - 1 <= p_last;
    if (k_live) {
      const __nv_bfloat16 *src = kbase + (ring0 + kr0) * kld + kc * 8;
      const uint32_t off = buf * KT + (kr0 * LK + kc * 8) * 2;
#pragma unroll
      for (uint32_t j = 0; j < WT_BN / KR; ++j, src += KR * kld) {
        const uint32_t key = t * WT_BN + kr0 + j * KR;
        if (whole || (key >= key_lo && key <= p_last)) cp_async16(k_u + off + j * KR * LK * 2, src);
        else *reinterpret_cast<uint4 *>(wt_smem + (k_u - qs_u) + off + j * KR * LK * 2) = make_uint4(0, 0, 0, 0);
      }
    }
    if (v_live) {
      const __nv_bfloat16 *src = vbase + (ring0 + vr0) * vld + vc * 8;
      const uint32_t off = buf * VT + (vr0 * LV + vc * 8) * 2;
#pragma unroll
      for (uint32_t j = 0; j < WT_BN / VR; ++j, src += VR * vld) {
        const uint32_t key = t * WT_BN + vr0 + j * VR;
        if (whole || (key >= key_lo && key <= p_last)) cp_async16(v_u + off + j * VR * LV * 2, src);
        else *reinterpret_cast<uint4 *>(wt_smem + (v_u - qs_u) + off + j * VR * LV * 2) = make_uint4(0, 0, 0, 0);
      }
    }
    cp_async_commit();
  };
  if (d.k_head < DK)
    for (uint32_t i = tid; i < 2 * WT_BN * (DK / 8); i += WT_THREADS)
      if (i % (DK / 8) * 8 >= d.k_head)
        *reinterpret_cast<uint4 *>(wt_smem + (k_u - qs_u) + (i / (DK / 8) * LK + i % (DK / 8) * 8) * 2) = make_uint4(0, 0, 0, 0);
  if (d.v_head < DV)
    for (uint32_t i = tid; i < 2 * WT_BN * (DV / 8); i += WT_THREADS)
      if (i % (DV / 8) * 8 >= d.v_head)
        *reinterpret_cast<uint4 *>(wt_smem + (v_u - qs_u) + (i / (DV / 8) * LV + i % (DV / 8) * 8) * 2) = make_uint4(0, 0, 0, 0);
  load_tile(t_first, 0);

  // queries: rotated at their own positions, rounded to bf16; eight pairs in flight per thread
  {
    constexpr uint32_t PP = DK / 2, QU = 8;  // pairs per row
    const uint32_t pi = tid % PP, rr = tid / PP;
    const float *q0 = d.q + (size_t)tok0 * d.ldqkv + (size_t)h * d.dim;
    for (uint32_t r0 = rr; r0 < WT_BM; r0 += QU * (WT_THREADS / PP)) {
      Pair pr[QU];
#pragma unroll
      for (uint32_t u = 0; u < QU; ++u) {
        const uint32_t r = r0 + u * (WT_THREADS / PP), rc = min(r, ntok - 1);  // (rows past the last token repeat it)
        pr[u] = load_pair(q0 + rc * d.ldqkv, pi, p0 + rc, d);
      }
#pragma unroll
      for (uint32_t u = 0; u < QU; ++u) {
        const uint32_t r = r0 + u * (WT_THREADS / PP);
        const Pair &x = pr[u];
        Qs[r * LK + x.e0] = __float2bfloat16_rn(x.x0 * x.c - x.x1 * x.s);
        Qs[r * LK + x.e1] = __float2bfloat16_rn(x.x1 * x.c + x.x0 * x.s);
      }
    }
  }
  __syncthreads();

  const uint32_t g = lane >> 2, tg = lane & 3, mat = lane >> 3, mr = lane & 7;
  uint32_t qa[KS][4];
#pragma unroll
  for (int ks = 0; ks < KS; ++ks) {
    const uint32_t row = warp * 16 + (mat & 1) * 8 + mr, col = ks * 16 + (mat >> 1) * 8;
    ldsm_x4(qs_u + (row * LK + col) * 2, qa[ks][0], qa[ks][1], qa[ks][2], qa[ks][3]);
  }
  const uint32_t row_lo = warp * 16 + g, row_hi = row_lo + 8;
  const uint32_t pos_lo = p0 + row_lo, pos_hi = p0 + row_hi;           // (rows past ntok compute and are not stored)
  const uint32_t wp_first = p0 + warp * 16, wp_last = wp_first + 15;   // this warp's positions
  const float scale_log2 = d.scale * 1.4426950408889634f;

  float o[DV / 8][4];
#pragma unroll
  for (int j = 0; j < DV / 8; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
  // running maxima (log2 units) and sums; a sink is a key of score 0 seen before all others
  float m_lo = d.sink ? 0.f : WA_NEG, m_hi = m_lo, l_lo = 0.f, l_hi = 0.f;

  for (uint32_t t = t_first; t < t_end; ++t) {
    const uint32_t buf = (t - t_first) & 1;
    if (t + 1 < t_end) {
      load_tile(t + 1, buf ^ 1);
      cp_async_wait<1>();
    } else {
      cp_async_wait<0>();
    }
    __syncthreads();
    const uint32_t kt_u = k_u + buf * KT, vt_u = v_u + buf * VT, key0 = t * WT_BN;
    // does this warp see the tile?  (its keys up to wp_last, from wp_first - window + 1 on)
    if (key0 <= wp_last && key0 + WT_BN + d.window > wp_first + 1) {
      float s[WT_BN / 8][4];
#pragma unroll
      for (int j = 0; j < WT_BN / 8; ++j) s[j][0] = s[j][1] = s[j][2] = s[j][3] = 0.f;
#pragma unroll
      for (int ks = 0; ks < KS; ++ks) {
#pragma unroll
        for (int j2 = 0; j2 < WT_BN / 16; ++j2) {
          const uint32_t row = j2 * 16 + (mat >> 1) * 8 + mr, col = ks * 16 + (mat & 1) * 8;
          uint32_t b0, b1, b2, b3;
          ldsm_x4(kt_u + (row * LK + col) * 2, b0, b1, b2, b3);
          mma_bf16(s[2 * j2], qa[ks], b0, b1);
          mma_bf16(s[2 * j2 + 1], qa[ks], b2, b3);
        }
      }
      float mx_lo = WA_NEG, mx_hi = WA_NEG;
      if (key0 + WT_BN - 1 <= wp_first && key0 + d.window > wp_last) {  // every key seen by every token of the warp
#pragma unroll
        for (int j = 0; j < WT_BN / 8; ++j) {
          s[j][0] *= scale_log2, s[j][1] *= scale_log2, s[j][2] *= scale_log2, s[j][3] *= scale_log2;
          mx_lo = fmaxf(mx_lo, fmaxf(s[j][0], s[j][1]));
          mx_hi = fmaxf(mx_hi, fmaxf(s[j][2], s[j][3]));
        }
      } else {
#pragma unroll
        for (int j = 0; j < WT_BN / 8; ++j) {
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const uint32_t key = key0 + j * 8 + 2 * tg + (e & 1), pos = e < 2 ? pos_lo : pos_hi;
            const float v = key <= pos && pos - key < d.window ? s[j][e] * scale_log2 : -INFINITY;
            s[j][e] = v;
            if (e < 2) mx_lo = fmaxf(mx_lo, v);
            else mx_hi = fmaxf(mx_hi, v);
          }
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
      for (int j = 0; j < WT_BN / 8; ++j) {
        s[j][0] = exp2f(s[j][0] - m_lo), s[j][1] = exp2f(s[j][1] - m_lo);
        s[j][2] = exp2f(s[j][2] - m_hi), s[j][3] = exp2f(s[j][3] - m_hi);
        sum_lo += s[j][0] + s[j][1];
        sum_hi += s[j][2] + s[j][3];
      }
      l_lo = l_lo * al_lo + sum_lo, l_hi = l_hi * al_hi + sum_hi;
#pragma unroll
      for (int j = 0; j < DV / 8; ++j) o[j][0] *= al_lo, o[j][1] *= al_lo, o[j][2] *= al_hi, o[j][3] *= al_hi;
#pragma unroll
      for (int kk = 0; kk < WT_BN / 16; ++kk) {
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
  if (d.sink) l_lo += exp2f(-m_lo), l_hi += exp2f(-m_hi);
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

// ---- prefill in fp32 arithmetic: a warp per (token, query head), 32 keys at a time --------------------------------------
constexpr int WS_WARPS = 8, WS_MAX_D = 256;

template <typename KV> __global__ void __launch_bounds__(32 * WS_WARPS) window_attention_simt_kernel(const cutb_window_attn_desc d) {
  __shared__ __align__(16) float qs[WS_WARPS][WS_MAX_D];
  pdl_enter();
  const uint32_t lane = threadIdx.x & 31, warp = threadIdx.x >> 5, tok = blockIdx.x * WS_WARPS + warp, h = blockIdx.y, G = d.n_kv_heads;
  if (tok >= d.n_tokens) return;
  const uint32_t pos = (d.pos_ptr ? *d.pos_ptr : d.pos) + tok;
  if (pos >= d.max_pos) {
    if (d.status && lane == 0) atomicExch(d.status, (int)CUTB_ERR_INVALID);
    return;
  }
  const uint32_t kvh = h / (d.n_heads / G);
  for (uint32_t e = lane; e < d.k_head; e += 32)
    qs[warp][e] = e < d.dim ? rotated(d.q + (size_t)tok * d.ldqkv + (size_t)h * d.dim, e, pos, d) * d.scale : 0.f;
  __syncwarp();
  const KV *kb = reinterpret_cast<const KV *>(d.k_cache) + (size_t)kvh * d.k_head;
  const KV *vb = reinterpret_cast<const KV *>(d.v_cache) + (size_t)kvh * d.v_head;
  const size_t kld = (size_t)G * d.k_head, vld = (size_t)G * d.v_head;
  float m = d.sink ? 0.f : WA_NEG, l = d.sink ? 1.f : 0.f, acc[WS_MAX_D / 32];
#pragma unroll
  for (int i = 0; i < WS_MAX_D / 32; ++i) acc[i] = 0.f;
  const uint32_t lo = pos + 1 > d.window ? pos + 1 - d.window : 0;
  for (uint32_t k0 = lo; k0 <= pos; k0 += 32) {
    const uint32_t key = k0 + lane;
    float s = -INFINITY;
    if (key <= pos) {
      const KV *kr = kb + (size_t)(key % d.ring_rows) * kld;
      s = 0.f;
      for (uint32_t e = 0; e < d.k_head; e += 8) {
        float kv[8];
        kv_unpack8(kv_raw8(kr + e), kv);
#pragma unroll
        for (int j = 0; j < 8; ++j) s = fmaf(qs[warp][e + j], kv[j], s);
      }
    }
    float mx = s;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
    const float mn = fmaxf(m, mx), al = expf(m - mn), pr = expf(s - mn);
    m = mn;
    float sum = pr;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
    l = fmaf(l, al, sum);
#pragma unroll
    for (int i = 0; i < WS_MAX_D / 32; ++i) acc[i] *= al;
    const uint32_t cnt = min(32u, pos - k0 + 1);
    for (uint32_t j = 0; j < cnt; ++j) {
      const float w = __shfl_sync(0xffffffffu, pr, j);
      const KV *vr = vb + (size_t)((k0 + j) % d.ring_rows) * vld;
#pragma unroll
      for (int i = 0; i < WS_MAX_D / 32; ++i) {
        const uint32_t e = lane + 32 * i;
        if (e < d.vdim) acc[i] = fmaf(w, kvf(vr[e]), acc[i]);
      }
    }
  }
  const float inv = 1.0f / l;
#pragma unroll
  for (int i = 0; i < WS_MAX_D / 32; ++i) {
    const uint32_t e = lane + 32 * i;
    if (e < d.vdim) store_out(d.out, d.out_dtype == CUTB_BF16, (size_t)tok * d.ldo + (size_t)h * d.vdim + e, acc[i] * inv);
  }
}

// ---- decode ------------------------------------------------------------------------------------------------------------
constexpr int WD_THREADS = 256, WD_WARPS = WD_THREADS / 32, WD_CHUNK = 512, WD_MAX_D = 256, WD_MAX_SPLITS = 8;

// grid = (n_kv_heads * head groups, S), cluster (1, S, 1); a block serves up to RG query heads of one KV head over its slice
// of the window.
template <typename KV, int RG> __global__ void __launch_bounds__(WD_THREADS) window_attention_decode_kernel(const cutb_window_attn_desc d) {
  extern __shared__ __align__(16) float wd_smem[];  // [WD_WARPS][RG][v_head] partial value sums
  __shared__ __align__(16) float qs[RG][WD_MAX_D], kn[WD_MAX_D], vn[WD_MAX_D];
  __shared__ float sc[RG][WD_CHUNK];
  __shared__ float head_m[RG], head_l[RG], fac[RG], p_new[RG];
  __shared__ float pacc[RG][WD_MAX_D];
  using Raw = typename RawOf<KV>::type;

  cg::cluster_group cluster = cg::this_cluster();
  const uint32_t tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, split = blockIdx.y, S = gridDim.y, G = d.n_kv_heads;
  const uint32_t rep = d.n_heads / G, ngrp = (rep + RG - 1) / RG, kvh = blockIdx.x / ngrp, grp = blockIdx.x % ngrp;
  const uint32_t h0 = kvh * rep + grp * RG, nr = min((uint32_t)RG, rep - grp * RG);
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");  // (a mat-vec behind this starts its weight stream)
  pdl_enter();
  const uint32_t pos = d.pos_ptr ? *d.pos_ptr : d.pos;
  if (pos >= d.max_pos) {  // (the same in every block of the cluster)
    if (d.status && tid == 0) atomicExch(d.status, (int)CUTB_ERR_INVALID);
    return;
  }
  const KV *kb = reinterpret_cast<const KV *>(d.k_cache) + (size_t)kvh * d.k_head;
  const KV *vb = reinterpret_cast<const KV *>(d.v_cache) + (size_t)kvh * d.v_head;
  const size_t kld = (size_t)G * d.k_head, vld = (size_t)G * d.v_head;
  // lanes per cache row: eight elements each
  uint32_t lpk = 1, lpv = 1;
  while (lpk * 8 < d.k_head) lpk *= 2;
  while (lpv * 8 < d.v_head) lpv *= 2;
  const uint32_t ke = lane % lpk * 8, ksub = lane / lpk, kpw = 32 / lpk;  // element, key within a pass, keys per warp and pass
  const uint32_t ve = lane % lpv * 8, vsub = lane / lpv, vpw = 32 / lpv;
  // keys before this token, dealt to the slices
  const uint32_t n_old = min(d.window - 1, pos), per = (n_old + S - 1) / S;
  const uint32_t s0 = min(split * per, n_old), s1 = min(s0 + per, n_old), row0 = (pos - n_old) % d.ring_rows;
  constexpr int U = 4;  // passes in flight
  auto load_k = [&](Raw (&raw)[U], uint32_t c0, uint32_t i0, uint32_t cnt) {
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const uint32_t i = i0 + u * WD_WARPS * kpw + ksub;
      uint32_t row = row0 + c0 + i;
      if (row >= d.ring_rows) row -= d.ring_rows;
      if (i < cnt && ke < d.k_head) raw[u] = kv_raw8(kb + (size_t)row * kld + ke);
      else kv_zero8(raw[u]);
    }
  };
  auto load_v = [&](Raw (&raw)[U], uint32_t c0, uint32_t i0, uint32_t cnt) {
#pragma unroll
    for (int u = 0; u < U; ++u) {
      const uint32_t i = i0 + u * WD_WARPS * vpw + vsub;
      uint32_t row = row0 + c0 + i;
      if (row >= d.ring_rows) row -= d.ring_rows;
      if (i < cnt && ve < d.v_head) raw[u] = kv_raw8(vb + (size_t)row * vld + ve);
      else kv_zero8(raw[u]);
    }
  };
  // the first keys and values are on their way while the queries are rotated
  Raw kr0[U], vr0[U];
  const uint32_t cnt0 = min((uint32_t)WD_CHUNK, s1 - s0);
  load_k(kr0, s0, warp * kpw, cnt0);
  load_v(vr0, s0, warp * vpw, cnt0);

  {  // pairs of the query heads, 32 lanes along a head
    const uint32_t pairs = d.k_head / 2;
#pragma unroll
    for (uint32_t r = 0; r < RG; ++r)
      if (r % WD_WARPS == warp || RG < WD_WARPS) {
        // fewer heads than warps: the warps of a head share its pairs
        constexpr uint32_t SH = RG < WD_WARPS ? WD_WARPS / RG : 1;
        if (RG < WD_WARPS && warp / SH != r) continue;
        for (uint32_t i = (RG < WD_WARPS ? warp % SH : 0) * 32 + lane; i < pairs; i += 32 * SH) {
          if (r < nr) {
            const Pair x = load_pair(d.q + (size_t)(h0 + r) * d.dim, i, pos, d);
            qs[r][x.e0] = (x.x0 * x.c - x.x1 * x.s) * d.scale;
            qs[r][x.e1] = (x.x1 * x.c + x.x0 * x.s) * d.scale;
          } else {
            qs[r][2 * i] = qs[r][2 * i + 1] = 0.f;
          }
        }
      }
  }
  if (split == 0) {  // this token's key and value, rounded as the cache holds them
    const bool store = grp == 0;
    KV *kw = reinterpret_cast<KV *>(d.k_cache) + (size_t)(pos % d.ring_rows) * kld + (size_t)kvh * d.k_head;
    KV *vw = reinterpret_cast<KV *>(d.v_cache) + (size_t)(pos % d.ring_rows) * vld + (size_t)kvh * d.v_head;
    for (uint32_t e = tid; e < d.k_head; e += WD_THREADS) {
      const float v = e < d.dim ? rotated(d.k + (size_t)kvh * d.dim, e, pos, d) : 0.f;
      kn[e] = kv_round(v, (const KV *)nullptr);
      if (store && e < d.dim) kv_put(kw + e, v);
    }
    for (uint32_t e = tid; e < d.v_head; e += WD_THREADS) {
      const float v = e < d.vdim ? mixed_value(d, 0, kvh * d.vdim + e) : 0.f;
      vn[e] = kv_round(v, (const KV *)nullptr);
      if (store && e < d.vdim) kv_put(vw + e, v);
    }
  }
  if (tid < RG) head_m[tid] = WA_NEG, head_l[tid] = 0.f, p_new[tid] = 0.f;
  __syncthreads();
  float qr[RG][8];
#pragma unroll
  for (int r = 0; r < RG; ++r)
#pragma unroll
    for (int j = 0; j < 8; ++j) qr[r][j] = ke < d.k_head ? qs[r][ke + j] : 0.f;
  float acc[RG][8];
#pragma unroll
  for (int r = 0; r < RG; ++r)
#pragma unroll
    for (int j = 0; j < 8; ++j) acc[r][j] = 0.f;

  // (the first slice has the new key to add even when there are no others)
  for (uint32_t c0 = s0; c0 < s1 || (c0 == s0 && split == 0); c0 += WD_CHUNK) {
    const uint32_t cnt = min((uint32_t)WD_CHUNK, s1 - c0);
    for (uint32_t i0 = warp * kpw; i0 < cnt; i0 += WD_WARPS * kpw * U) {
      Raw raw[U];
      if (c0 == s0 && i0 == warp * kpw) {
#pragma unroll
        for (int u = 0; u < U; ++u) raw[u] = kr0[u];
      } else {
        load_k(raw, c0, i0, cnt);
      }
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const uint32_t i = i0 + u * WD_WARPS * kpw + ksub;
        float kv[8], dot[RG];
        kv_unpack8(raw[u], kv);
#pragma unroll
        for (int r = 0; r < RG; ++r) {
          dot[r] = 0.f;
#pragma unroll
          for (int j = 0; j < 8; ++j) dot[r] = fmaf(qr[r][j], kv[j], dot[r]);
        }
        for (uint32_t o = lpk >> 1; o > 0; o >>= 1)
#pragma unroll
          for (int r = 0; r < RG; ++r) dot[r] += __shfl_xor_sync(0xffffffffu, dot[r], o);
        if (i < cnt && ke == 0) {
#pragma unroll
          for (int r = 0; r < RG; ++r) sc[r][i] = dot[r];
        }
      }
    }
    if (c0 != s0) load_v(vr0, c0, warp * vpw, cnt);  // on their way while the softmax runs
    __syncthreads();
    for (uint32_t r = warp; r < RG; r += WD_WARPS) {
      const bool fresh = c0 == s0 && split == 0;  // the new token's key, and the sink as a key of score 0
      float m = head_m[r], s_new = 0.f;
      if (fresh) {
        for (uint32_t e = lane; e < d.k_head; e += 32) s_new = fmaf(qs[r][e], kn[e], s_new);
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) s_new += __shfl_xor_sync(0xffffffffu, s_new, o);
        m = d.sink ? fmaxf(s_new, 0.f) : s_new;
      }
      for (uint32_t i = lane; i < cnt; i += 32) m = fmaxf(m, sc[r][i]);
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
      const float f = expf(head_m[r] - m);
      float l = 0.f;
      for (uint32_t i = lane; i < cnt; i += 32) {
        const float e = expf(sc[r][i] - m);
        sc[r][i] = e;
        l += e;
      }
#pragma unroll
      for (int o = 16; o > 0; o >>= 1) l += __shfl_xor_sync(0xffffffffu, l, o);
      __syncwarp();
      if (lane == 0) {
        if (fresh) {
          const float p = expf(s_new - m);
          p_new[r] = p;
          l += p + (d.sink ? expf(-m) : 0.f);
        }
        head_l[r] = fmaf(head_l[r], f, l), head_m[r] = m, fac[r] = f;
      }
    }
    __syncthreads();
    if (c0 != s0) {
#pragma unroll
      for (int r = 0; r < RG; ++r)
#pragma unroll
        for (int j = 0; j < 8; ++j) acc[r][j] *= fac[r];
    } else if (split == 0 && warp == 0 && vsub == 0 && ve < d.v_head) {
#pragma unroll
      for (int r = 0; r < RG; ++r)
#pragma unroll
        for (int j = 0; j < 8; ++j) acc[r][j] = p_new[r] * vn[ve + j];
    }
    for (uint32_t i0 = warp * vpw; i0 < cnt; i0 += WD_WARPS * vpw * U) {
      Raw raw[U];
      if (i0 == warp * vpw) {
#pragma unroll
        for (int u = 0; u < U; ++u) raw[u] = vr0[u];
      } else {
        load_v(raw, c0, i0, cnt);
      }
#pragma unroll
      for (int u = 0; u < U; ++u) {
        const uint32_t i = i0 + u * WD_WARPS * vpw + vsub;
        if (i >= cnt) continue;
        float vv[8];
        kv_unpack8(raw[u], vv);
#pragma unroll
        for (int r = 0; r < RG; ++r) {
          const float w = sc[r][i];
#pragma unroll
          for (int j = 0; j < 8; ++j) acc[r][j] = fmaf(w, vv[j], acc[r][j]);
        }
      }
    }
    __syncthreads();  // the next chunk overwrites the scores
  }

  // sums of a warp's key groups, of the block's warps, then of the cluster's slices
#pragma unroll
  for (int r = 0; r < RG; ++r)
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      for (uint32_t o = lpv; o < 32; o <<= 1) acc[r][j] += __shfl_xor_sync(0xffffffffu, acc[r][j], o);
      if (vsub == 0 && ve < d.v_head) wd_smem[(warp * RG + r) * d.v_head + ve + j] = acc[r][j];
    }
  __syncthreads();
  for (uint32_t i = tid; i < RG * d.vdim; i += WD_THREADS) {
    const uint32_t r = i / d.vdim, e = i % d.vdim;
    float s = 0.f;
#pragma unroll
    for (int w = 0; w < WD_WARPS; ++w) s += wd_smem[(w * RG + r) * d.v_head + e];
    pacc[r][e] = s;
  }
  cluster.sync();
  for (uint32_t i = split * WD_THREADS + tid; i < nr * d.vdim; i += S * WD_THREADS) {
    const uint32_t r = i / d.vdim, e = i % d.vdim;
    float mk[WD_MAX_SPLITS], lk[WD_MAX_SPLITS], ak[WD_MAX_SPLITS], m = WA_NEG, l = 0.f, s = 0.f;
#pragma unroll
    for (uint32_t k = 0; k < WD_MAX_SPLITS; ++k) {  // every remote read in flight at once
      const uint32_t from = k < S ? k : 0;
      mk[k] = *cluster.map_shared_rank(&head_m[r], from);
      lk[k] = *cluster.map_shared_rank(&head_l[r], from);
      ak[k] = *cluster.map_shared_rank(&pacc[r][e], from);
    }
#pragma unroll
    for (uint32_t k = 0; k < WD_MAX_SPLITS; ++k)
      if (k < S) m = fmaxf(m, mk[k]);
#pragma unroll
    for (uint32_t k = 0; k < WD_MAX_SPLITS; ++k)
      if (k < S) {
        const float w = expf(mk[k] - m);
        l = fmaf(w, lk[k], l);
        s = fmaf(w, ak[k], s);
      }
    store_out(d.out, d.out_dtype == CUTB_BF16, (size_t)(h0 + r) * d.vdim + e, s / l);
  }
  cluster.sync();  // nobody leaves while its shared memory may still be read
}

template <int DK, int DV> int wt_launch(const cutb_window_attn_desc &d, cudaStream_t stream) {
  constexpr size_t smem = ((size_t)(WT_BM + 2 * WT_BN) * (DK + WT_PAD) + (size_t)2 * WT_BN * (DV + WT_PAD)) * 2;
  CUTB_CUDA_TRY(cudaFuncSetAttribute(window_attention_tc_kernel<DK, DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  CUTB_CUDA_TRY(launch_pdl(window_attention_tc_kernel<DK, DV>, dim3((d.n_tokens + WT_BM - 1) / WT_BM, d.n_heads), dim3(WT_THREADS), smem,
                           stream, d));
  return CUTB_OK;
}

template <typename KV, int RG> int wd_launch(const cutb_window_attn_desc &d, cudaStream_t stream) {
  const uint32_t rep = d.n_heads / d.n_kv_heads, keys = d.window < d.max_pos ? d.window : d.max_pos;
  uint32_t S = 1;
  while (S < WD_MAX_SPLITS && keys > 32 * S) S *= 2;
  const size_t smem = (size_t)WD_WARPS * RG * d.v_head * sizeof(float);
  CUTB_CUDA_TRY(cudaFuncSetAttribute(window_attention_decode_kernel<KV, RG>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(d.n_kv_heads * ((rep + RG - 1) / RG), S);
  cfg.blockDim = dim3(WD_THREADS);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = stream;
  cudaLaunchAttribute attr[2];
  attr[0].id = cudaLaunchAttributeClusterDimension;
  attr[0].val.clusterDim.x = 1;
  attr[0].val.clusterDim.y = S;
  attr[0].val.clusterDim.z = 1;
  attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[1].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = 2;
  CUTB_CUDA_TRY(cudaLaunchKernelEx(&cfg, window_attention_decode_kernel<KV, RG>, d));
  return CUTB_OK;
}
// Query heads per block: one as long as the blocks fit the GPU twice over (keys and values then come from L2 once per head;
// the kernel is bound by latency, not by bytes), more for models with many heads.
template <typename KV> int wd_dispatch(const cutb_window_attn_desc &d, cudaStream_t stream) {
  const uint32_t rep = d.n_heads / d.n_kv_heads;
  if (rep == 1 || d.n_heads <= 48) return wd_launch<KV, 1>(d, stream);
  if (rep == 2 || d.n_heads <= 96) return wd_launch<KV, 2>(d, stream);
  return wd_launch<KV, 4>(d, stream);
}

}  // namespace

int window_kv_write_launch(const cutb_window_attn_desc &d, cudaStream_t stream) {
  if (d.kv_dtype == CUTB_BF16) CUTB_CUDA_TRY(launch_pdl(window_kv_write_kernel<__nv_bfloat16>, dim3(d.n_tokens), dim3(256), 0, stream, d));
  else CUTB_CUDA_TRY(launch_pdl(window_kv_write_kernel<float>, dim3(d.n_tokens), dim3(256), 0, stream, d));
  return CUTB_OK;
}

int window_attention_launch(const cutb_window_attn_desc &d, cudaStream_t stream) {
  if (d.kv_dtype == CUTB_BF16 && d.dim <= 128 && d.vdim <= 128) {
    if (d.dim <= 64) return d.vdim <= 64 ? wt_launch<64, 64>(d, stream) : wt_launch<64, 128>(d, stream);
    return d.vdim <= 64 ? wt_launch<128, 64>(d, stream) : wt_launch<128, 128>(d, stream);
  }
  const dim3 grid((d.n_tokens + WS_WARPS - 1) / WS_WARPS, d.n_heads);
  if (d.kv_dtype == CUTB_BF16) CUTB_CUDA_TRY(launch_pdl(window_attention_simt_kernel<__nv_bfloat16>, grid, dim3(32 * WS_WARPS), 0, stream, d));
  else CUTB_CUDA_TRY(launch_pdl(window_attention_simt_kernel<float>, grid, dim3(32 * WS_WARPS), 0, stream, d));
  return CUTB_OK;
}

int window_attention_decode_launch(const cutb_window_attn_desc &d, cudaStream_t stream) {
  return d.kv_dtype == CUTB_BF16 ? wd_dispatch<__nv_bfloat16>(d, stream) : wd_dispatch<float>(d, stream);
}

}  // namespace cutb
