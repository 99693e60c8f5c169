// Prefill GEMM over dense bf16 weights, C[M, N] = unary(A[M, K] W[N, K]^T + bias), and its 32-bit companion.
//
// dense_gemm_tc_kernel: persistent, warp-specialised tcgen05 kernel.  A CTA tile is 128 tokens x BN weight rows (64 / 128 /
// 256); tokens are the MMA's M operand (one per tensor-memory lane), weight rows its N operand.
//   warp 0      one lane copies the 64-k stages of both operands by TMA (128-byte swizzle; rows and k past the matrices read as
//               zero) into a ring that fills shared memory;
//   warp 1      allocates tensor memory (two accumulators of BN columns); one lane issues four K = 16 MMAs per stage and
//               commits them to the stage's "empty" barrier, and after the last stage to the accumulator's "full" barrier;
//   warps 2..5  epilogue of the previous tile meanwhile: tcgen05.ld (lane = token, 32 columns at a time), bias, elementwise
//               op, 16-byte stores along the row.
// GROUPED (experts): the rows of A are sorted by expert, expert e's are offsets[e] .. offsets[e + 1] - 1, and they meet its own N
// rows of the stacked weight.  Every CTA derives the list of tiles from the offsets on the device; a tile's copy may run into
// the next expert's rows, whose products are not stored.  Neighbouring outputs may pass through a gated unit (gate, up).
// Few tiles and a long K: the K stages of a tile are shared out over CTAs, partial sums go to the workspace and a second
// kernel adds them in a fixed order and applies the epilogue.
// Every wait is bounded; on expiry the CTA records CUTB_ERR_TIMEOUT in the caller's status word, waits (bounded) for its own
// copies in flight, frees its tensor memory and returns.
//
// dense_gemm_simt_kernel: fp32 fused multiply-adds (bf16 weights are exact in fp32), for the true 32-bit mode.
#include <cuda.h>
#include <cuda_bf16.h>

#include "common.cuh"
#include "dense_common.cuh"
#include "kernels.h"
#include "tcgen05.cuh"

namespace cutb {
namespace {

constexpr int DG_BM = 128, DG_BK = 64, DG_THREADS = 192;
constexpr uint32_t DG_A_BYTES = DG_BM * DG_BK * 2;
__host__ __device__ constexpr int dg_stages(int bn) { return bn == 256 ? 4 : (bn == 128 ? 6 : 8); }
__host__ __device__ constexpr uint32_t dg_stage_bytes(int bn) { return DG_A_BYTES + (uint32_t)bn * DG_BK * 2; }
constexpr uint32_t dg_smem(int bn) { return 1024 + dg_stages(bn) * dg_stage_bytes(bn); }

struct DgParams {
  const float *bias;
  void *C;
  float *partial;  // [ksplit][M][N] when K is split
  int *status;
  uint32_t M, K, N, ldc;
  uint32_t tiles_m, tiles_n, ksplit, nk, nk_per, a_box_rows;
  int c_bf16, unary;
  const uint32_t *offsets;  // grouped
  uint32_t experts;
  GluParams glu;
};
constexpr uint32_t DG_MAX_EXPERTS = 1024;

struct DgJob {
  uint32_t m0, m_end, n0, w0, k0, nk, z;  // rows m0 .. m_end - 1 are stored; w0 = row of the stacked weight
};

template <int BN, bool GROUPED>
__global__ void __launch_bounds__(DG_THREADS, 1) dense_gemm_tc_kernel(const __grid_constant__ CUtensorMap map_a,
                                                                      const __grid_constant__ CUtensorMap map_w, const DgParams p) {
  constexpr int S = dg_stages(BN);
  constexpr uint32_t STAGE = dg_stage_bytes(BN), COLS = 2 * BN;
  extern __shared__ __align__(1024) uint8_t dg_raw[];
  uint8_t *ring = reinterpret_cast<uint8_t *>((reinterpret_cast<uintptr_t>(dg_raw) + 1023) & ~uintptr_t(1023));
  __shared__ __align__(8) uint64_t bars[2 * S + 4];  // full[S], empty[S], accumulator full[2], accumulator empty[2]
  __shared__ uint32_t tmem_slot, abort_flag;
  __shared__ uint32_t offs[GROUPED ? DG_MAX_EXPERTS + 1 : 1], first_tile[GROUPED ? DG_MAX_EXPERTS + 1 : 1];
  const uint32_t tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const uint32_t full_u = smem_u32(bars), empty_u = full_u + S * 8, afull_u = empty_u + S * 8, aempty_u = afull_u + 16;
  const uint32_t ring_u = smem_u32(ring);

  if (tid == 0) {
    for (int s = 0; s < S; ++s) mbar_init(full_u + s * 8, 1), mbar_init(empty_u + s * 8, 1);
    for (int a = 0; a < 2; ++a) mbar_init(afull_u + a * 8, 1), mbar_init(aempty_u + a * 8, 4);
    abort_flag = 0;
    fence_mbar_init();
  }
  if (warp == 1) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&tmem_slot)), "r"(COLS) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  if (GROUPED && warp == 2) {  // row tiles before each expert
    uint32_t before = 0;
    for (uint32_t e0 = 0; e0 < p.experts; e0 += 32) {
      const uint32_t e = e0 + lane, lo = min(p.offsets[min(e, p.experts)], p.M), hi = min(p.offsets[min(e + 1, p.experts)], p.M);
      const uint32_t tiles = e < p.experts && hi > lo ? (hi - lo + DG_BM - 1) / DG_BM : 0;
      uint32_t sum = tiles;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const uint32_t v = __shfl_up_sync(0xffffffffu, sum, o);
        if (lane >= (uint32_t)o) sum += v;
      }
      if (e < p.experts) offs[e] = lo, first_tile[e] = before + sum - tiles;
      if (e + 1 == p.experts) offs[e + 1] = hi;
      before += __shfl_sync(0xffffffffu, sum, 31);
    }
    if (lane == 0) first_tile[p.experts] = before;
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = tmem_slot;
  auto give_up = [&]() {
    if (p.status) atomicExch(p.status, (int)CUTB_ERR_TIMEOUT);
    atomicExch(&abort_flag, 1u);
  };
  auto aborted = [&]() { return *reinterpret_cast<volatile uint32_t *>(&abort_flag) != 0; };

  const uint32_t jobs = GROUPED ? first_tile[p.experts] * p.tiles_n : p.tiles_m * p.tiles_n * p.ksplit;
  // job -> token tile fastest (CTAs that run together share weight rows), then weight tile, then share of K; grouped: expert by
  // expert (a role's jobs ascend, so its cursor `e` only moves forward)
  uint32_t e = 0;
  auto job_of = [&](uint32_t j) {
    DgJob b;
    if constexpr (GROUPED) {
      while (j >= first_tile[e + 1] * p.tiles_n) ++e;
      const uint32_t rel = j - first_tile[e] * p.tiles_n, tm = first_tile[e + 1] - first_tile[e];
      b.m0 = offs[e] + rel % tm * DG_BM, b.m_end = offs[e + 1];
      b.n0 = rel / tm * BN, b.w0 = e * p.N + b.n0;
      b.z = b.k0 = 0, b.nk = p.nk;
    } else {
      b.m0 = j % p.tiles_m * DG_BM, b.m_end = p.M;
      b.n0 = b.w0 = j / p.tiles_m % p.tiles_n * BN;
      b.z = j / (p.tiles_m * p.tiles_n);
      b.k0 = b.z * p.nk_per;
      b.nk = min(p.nk_per, p.nk - b.k0);  // (the launcher leaves no share empty)
    }
    return b;
  };

  // The copy and MMA warps run converged, with one elected lane issuing: loop variables stay warp-uniform.  A wait that runs
  // out marks the warp dead; it then runs through its remaining steps without waiting, so that every loop ends.
  if (warp == 0) {
    const bool leader = elect_one();
    uint32_t s = 0, ph = 1;  // (a fresh barrier lets a wait on the phase before its first pass)
    const uint32_t bytes = p.a_box_rows * DG_BK * 2 + BN * DG_BK * 2;
    bool dead = false;
    for (uint32_t j = blockIdx.x; j < jobs; j += gridDim.x) {
      const DgJob b = job_of(j);
      for (uint32_t ks = 0; ks < b.nk; ++ks) {
        if (!dead && !mbar_spin_bounded(empty_u + s * 8, ph)) {
          give_up();
          dead = true;
        }
        const uint32_t bar = full_u + s * 8, dst = ring_u + s * STAGE, x = (b.k0 + ks) * DG_BK;
        if (leader && !dead) {
          mbar_arrive_expect_tx(bar, bytes);
          tma_load_2d(dst, &map_a, x, b.m0, bar);
          tma_load_2d(dst + DG_A_BYTES, &map_w, x, b.w0, bar);
        }
        if (++s == S) s = 0, ph ^= 1u;
      }
    }
    // do not retire with copies still landing in shared memory: every stage's last fill (bounded; a stage that was never
    // filled, or whose fill the MMA warp has consumed, answers at once or runs into the small limit of an aborted launch)
    if (aborted()) {
      for (uint32_t i = 0; i < S; ++i) {
        if (s == 0) s = S, ph ^= 1u;
        --s;
        mbar_wait_bounded(full_u + s * 8, ph ^ 1u, 1u << 8);
      }
    }
    __syncwarp();
  } else if (warp == 1) {
    const bool leader = elect_one();
    const uint64_t proto = umma_desc_sw128(0);
    const uint32_t desc_hi = (uint32_t)(proto >> 32), base = (uint32_t)proto + ((ring_u & 0x3FFFFu) >> 4);
    const uint32_t idesc = umma_idesc_bf16(DG_BM, BN);
    uint32_t s = 0, ph = 0, turn = 0;
    bool dead = false;
    for (uint32_t j = blockIdx.x; j < jobs; j += gridDim.x, ++turn) {
      const uint32_t nk = job_of(j).nk, a = turn & 1, d = tmem + a * BN;
      if (turn >= 2 && !dead && !mbar_spin_bounded(aempty_u + a * 8, ((turn >> 1) - 1) & 1u)) {
        give_up();
        dead = true;
      }
      tc_fence_after();
      for (uint32_t ks = 0; ks < nk; ++ks) {
        if (!dead && !mbar_spin_bounded(full_u + s * 8, ph)) {
          give_up();
          dead = true;
        }
        tc_fence_after();
        const uint32_t at = base + s * (STAGE >> 4), wt = at + (DG_A_BYTES >> 4);
        if (leader) {
          umma_f16(d, at, wt, desc_hi, idesc, ks != 0);
          umma_f16(d, at + 2, wt + 2, desc_hi, idesc, 1);
          umma_f16(d, at + 4, wt + 4, desc_hi, idesc, 1);
          umma_f16(d, at + 6, wt + 6, desc_hi, idesc, 1);
          umma_commit(empty_u + s * 8);
        }
        if (++s == S) s = 0, ph ^= 1u;
      }
      if (leader) umma_commit(afull_u + a * 8);
    }
    __syncwarp();
  } else {
    const uint32_t quarter = warp & 3;  // tensor-memory lanes this warp may read
    uint32_t turn = 0;
    for (uint32_t j = blockIdx.x; j < jobs; j += gridDim.x, ++turn) {
      const DgJob b = job_of(j);
      const uint32_t a = turn & 1;
      uint32_t ok = 1;
      if (lane == 0) ok = !aborted() && mbar_wait_bounded(afull_u + a * 8, (turn >> 1) & 1u);
      ok = __shfl_sync(0xffffffffu, ok, 0);
      if (!ok) {
        if (lane == 0) give_up();
        break;
      }
      tc_fence_after();
      const uint32_t m = b.m0 + quarter * 32 + lane;
#pragma unroll 1
      for (uint32_t c0 = 0; c0 < BN; c0 += 32) {
        const uint32_t n = b.n0 + c0;
        if (n >= p.N) break;
        uint32_t v[32];
        tmem_ld32(tmem + ((quarter * 32) << 16) + a * BN + c0, v);
        if (m >= b.m_end) continue;
        const bool whole = n + 32 <= p.N;
        if constexpr (GROUPED) {
          if (p.glu.kind) {  // N is even: outputs 2 i and 2 i + 1 make one
            float y[16];
#pragma unroll
            for (int i = 0; i < 16; ++i) y[i] = glu(p.glu, __uint_as_float(v[2 * i]), __uint_as_float(v[2 * i + 1]));
            const size_t base = (size_t)m * p.ldc + n / 2;
            if (whole && p.ldc % 8 == 0 && p.c_bf16) {
              uint4 *dst = reinterpret_cast<uint4 *>(reinterpret_cast<__nv_bfloat16 *>(p.C) + base);
#pragma unroll
              for (int i = 0; i < 2; ++i)
                dst[i] = make_uint4(pack_bf16(y[8 * i], y[8 * i + 1]), pack_bf16(y[8 * i + 2], y[8 * i + 3]),
                                    pack_bf16(y[8 * i + 4], y[8 * i + 5]), pack_bf16(y[8 * i + 6], y[8 * i + 7]));
            } else {
#pragma unroll
              for (int i = 0; i < 16; ++i)
                if (n + 2 * i < p.N) store_out(p.C, p.c_bf16, base + i, y[i]);
            }
            continue;
          }
        } else if (p.ksplit > 1) {
          float *dst = p.partial + ((size_t)b.z * p.M + m) * p.N + n;
          if (whole && p.N % 4 == 0) {
#pragma unroll
            for (int i = 0; i < 8; ++i) reinterpret_cast<uint4 *>(dst)[i] = make_uint4(v[4 * i], v[4 * i + 1], v[4 * i + 2], v[4 * i + 3]);
          } else {
#pragma unroll
            for (int i = 0; i < 32; ++i)
              if (n + i < p.N) dst[i] = __uint_as_float(v[i]);
          }
          continue;
        }
        float x[32];
#pragma unroll
        for (int i = 0; i < 32; ++i) x[i] = __uint_as_float(v[i]) + (p.bias && n + i < p.N ? __ldg(p.bias + n + i) : 0.f);
        if (p.unary == CUTB_UNARY_RELU_SQUARE) {
#pragma unroll
          for (int i = 0; i < 32; ++i) x[i] = fmaxf(x[i], 0.f) * fmaxf(x[i], 0.f);
        } else if (p.unary) {
          float (&x8)[32] = x;
          const float none[32] = {};
          apply_epilogue_n<32>(x8, none, CUTB_FUSION_UNARY, p.unary);
        }
        const size_t base = (size_t)m * p.ldc + n;
        if (whole && p.ldc % 8 == 0) {
          if (p.c_bf16) {
            uint4 *dst = reinterpret_cast<uint4 *>(reinterpret_cast<__nv_bfloat16 *>(p.C) + base);
#pragma unroll
            for (int i = 0; i < 4; ++i)
              dst[i] = make_uint4(pack_bf16(x[8 * i], x[8 * i + 1]), pack_bf16(x[8 * i + 2], x[8 * i + 3]),
                                  pack_bf16(x[8 * i + 4], x[8 * i + 5]), pack_bf16(x[8 * i + 6], x[8 * i + 7]));
          } else {
            float4 *dst = reinterpret_cast<float4 *>(reinterpret_cast<float *>(p.C) + base);
#pragma unroll
            for (int i = 0; i < 8; ++i) dst[i] = make_float4(x[4 * i], x[4 * i + 1], x[4 * i + 2], x[4 * i + 3]);
          }
        } else {
#pragma unroll
          for (int i = 0; i < 32; ++i)
            if (n + i < p.N) store_out(p.C, p.c_bf16, base + i, x[i]);
        }
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(aempty_u + a * 8);
    }
  }

  tc_fence_before();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after();
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(COLS) : "memory");
  }
}

__global__ void __launch_bounds__(256) dense_splitk_reduce_kernel(const DgParams p) {
  const size_t idx = (size_t)blockIdx.x * 256 + threadIdx.x, total = (size_t)p.M * p.N;
  if (idx >= total) return;
  const uint32_t m = (uint32_t)(idx / p.N), n = (uint32_t)(idx % p.N);
  float sum = 0.f;
#pragma unroll 4
  for (uint32_t z = 0; z < p.ksplit; ++z) sum += p.partial[z * total + idx];
  store_out(p.C, p.c_bf16, (size_t)m * p.ldc + n, dense_unary(sum + (p.bias ? __ldg(p.bias + n) : 0.f), p.unary));
}

// 64 x 64 outputs per block of 256 threads, 4 x 4 per thread, k in steps of 16.  blockIdx.z = product of a batch; with `offsets`
// blockIdx.y = tile of an expert's rows.
struct DsParams {
  const void *A;
  const __nv_bfloat16 *W;
  const float *bias;
  void *C;
  uint32_t lda, ldw, ldc, M, N, K, a_batch, c_batch;
  int c_bf16, unary;
  const uint32_t *offsets;
  uint32_t experts;
  GluParams glu;
};

template <typename TA> __global__ void __launch_bounds__(256) dense_gemm_simt_kernel(const DsParams p) {
  __shared__ __align__(16) float as[16][64 + 4], ws[16][64 + 4];
  __shared__ uint32_t where[3];  // expert, first row, end of its rows
  pdl_enter();
  const uint32_t tid = threadIdx.x, tx = tid % 16, ty = tid / 16, n0 = blockIdx.x * 64, N = p.N, K = p.K, lda = p.lda, ldw = p.ldw;
  uint32_t m0 = blockIdx.y * 64, M = p.M;
  const TA *A = reinterpret_cast<const TA *>(p.A) + (size_t)blockIdx.z * p.a_batch;
  const __nv_bfloat16 *W = p.W + (size_t)blockIdx.z * N * ldw;
  if (p.offsets) {
    if (tid == 0) {
      uint32_t before = 0, e = 0, lo = 0, hi = 0;
      for (; e < p.experts; ++e) {
        lo = min(p.offsets[e], M), hi = min(p.offsets[e + 1], M);
        const uint32_t tiles = hi > lo ? (hi - lo + 63) / 64 : 0;
        if (blockIdx.y < before + tiles) break;
        before += tiles;
      }
      where[0] = e, where[1] = lo + (blockIdx.y - before) * 64, where[2] = hi;
    }
    __syncthreads();
    if (where[0] >= p.experts) return;  // (the grid is an upper bound)
    m0 = where[1], M = where[2];
    W += (size_t)where[0] * N * ldw;
  }
  float acc[4][4] = {};
  for (uint32_t k0 = 0; k0 < K; k0 += 16) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const uint32_t r = tid / 16 + 16 * i, k = k0 + tid % 16;
      as[tid % 16][r] = m0 + r < M && k < K ? (float)A[(size_t)(m0 + r) * lda + k] : 0.f;
      ws[tid % 16][r] = n0 + r < N && k < K ? __bfloat162float(W[(size_t)(n0 + r) * ldw + k]) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < 16; ++k) {
      const float4 a = *reinterpret_cast<const float4 *>(&as[k][ty * 4]), w = *reinterpret_cast<const float4 *>(&ws[k][tx * 4]);
      const float av[4] = {a.x, a.y, a.z, a.w}, wv[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(av[i], wv[j], acc[i][j]);
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const uint32_t m = m0 + ty * 4 + i, n = n0 + tx * 4;
    if (m >= M) continue;
    const size_t at = (size_t)m * p.ldc + (size_t)blockIdx.z * p.c_batch;
    if (p.glu.kind) {
#pragma unroll
      for (int j = 0; j < 4; j += 2)
        if (n + j < N) store_out(p.C, p.c_bf16, at + (n + j) / 2, glu(p.glu, acc[i][j], acc[i][j + 1]));
      continue;
    }
#pragma unroll
    for (int j = 0; j < 4; ++j)
      if (n + j < N) store_out(p.C, p.c_bf16, at + n + j, dense_unary(acc[i][j] + (p.bias ? __ldg(p.bias + n + j) : 0.f), p.unary));
  }
}

struct DgPlan {
  int bn;
  uint32_t tiles_m, tiles_n, ksplit, nk, nk_per;
};
// Tile width by the time of its waves; K split when even narrow tiles leave most SMs idle.
DgPlan dg_plan(const cutb_dense_desc &d, uint32_t sms) {
  DgPlan b{};
  uint64_t best = ~0ull;
  const uint32_t tm = (d.M + DG_BM - 1) / DG_BM;
  // measured time of a wave of tiles, relative: a 64-k stage costs at least what its operands take to arrive
  const struct { int bn; uint32_t cost; } kinds[] = {{256, 100}, {128, 66}, {64, 62}};
  for (const auto &kind : kinds) {
    const int bn = kind.bn;
    const uint32_t tn = (d.N + bn - 1) / bn;
    const uint64_t cost = (uint64_t)((tm * tn + sms - 1) / sms) * kind.cost;
    if (cost < best) best = cost, b.bn = bn, b.tiles_m = tm, b.tiles_n = tn;
  }
  b.nk = (d.K + DG_BK - 1) / DG_BK;
  if (tm * ((d.N + 127) / 128) * 2 <= sms && b.nk >= 16) {
    b.bn = 128;
    b.tiles_n = (d.N + 127) / 128;
    uint32_t want = sms / (b.tiles_m * b.tiles_n);
    if (want > b.nk / 4) want = b.nk / 4;
    if (want > 16) want = 16;
    if (want < 1) want = 1;
    b.nk_per = (b.nk + want - 1) / want;
    b.ksplit = (b.nk + b.nk_per - 1) / b.nk_per;
  } else {
    b.ksplit = 1, b.nk_per = b.nk;
  }
  return b;
}

template <int BN, bool GROUPED> int dg_launch(const CUtensorMap &ma, const CUtensorMap &mw, const DgParams &p, uint32_t sms, cudaStream_t stream) {
  static bool configured[64] = {};
  int dev = 0;
  CUTB_CUDA_TRY(cudaGetDevice(&dev));
  if (dev < 0 || dev >= 64 || !configured[dev]) {
    CUTB_CUDA_TRY(cudaFuncSetAttribute(dense_gemm_tc_kernel<BN, GROUPED>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)dg_smem(BN)));
    if (dev >= 0 && dev < 64) configured[dev] = true;
  }
  const uint32_t jobs = p.tiles_m * p.tiles_n * p.ksplit;  // (grouped: an upper bound)
  dense_gemm_tc_kernel<BN, GROUPED><<<jobs < sms ? jobs : sms, DG_THREADS, dg_smem(BN), stream>>>(ma, mw, p);
  CUTB_CUDA_TRY(cudaGetLastError());
  return CUTB_OK;
}

}  // namespace

uint64_t dense_gemm_tc_workspace(const cutb_dense_desc &d) {
  DeviceInfo di;
  const uint32_t sms = get_device_info(&di) == CUTB_OK ? (uint32_t)di.sm_count : 148u;
  const DgPlan pl = dg_plan(d, sms);
  return pl.ksplit > 1 ? (uint64_t)pl.ksplit * d.M * d.N * sizeof(float) : 0;
}

bool dense_gemm_tc_supported(const cutb_dense_desc &d) {
  return d.a_dtype == CUTB_BF16 && d.lda % 8 == 0 && reinterpret_cast<uintptr_t>(d.A) % 16 == 0;
}

int dense_gemm_tc_launch(const cutb_dense_desc &d, cudaStream_t stream) {
  DeviceInfo di;
  if (int rc = get_device_info(&di)) return rc;
  DgPlan pl = dg_plan(d, (uint32_t)di.sm_count);
  if (pl.ksplit > 1 && (!d.workspace || d.workspace_bytes < (uint64_t)pl.ksplit * d.M * d.N * sizeof(float) ||
                        reinterpret_cast<uintptr_t>(d.workspace) % 16 != 0))
    pl.ksplit = 1, pl.nk_per = pl.nk;
  DgParams p{};
  p.bias = d.bias, p.C = d.C, p.status = d.status, p.M = d.M, p.K = d.K, p.N = d.N, p.ldc = d.ldc;
  p.partial = pl.ksplit > 1 ? reinterpret_cast<float *>(d.workspace) : nullptr;
  p.tiles_m = pl.tiles_m, p.tiles_n = pl.tiles_n, p.ksplit = pl.ksplit, p.nk = pl.nk, p.nk_per = pl.nk_per;
  p.a_box_rows = d.M >= DG_BM ? DG_BM : (d.M + 7) / 8 * 8;  // (rows of the tile that are not copied only feed outputs that are not stored)
  p.c_bf16 = d.c_dtype == CUTB_BF16, p.unary = d.unary_op;
  CUtensorMap ma, mw;
  if (int rc = make_tmap_sw128(&ma, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, d.A, d.M, d.K, (uint64_t)d.lda * 2, p.a_box_rows)) return rc;
  if (int rc = make_tmap_sw128(&mw, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, d.W, d.N, d.K, (uint64_t)d.ldw * 2, (uint32_t)pl.bn)) return rc;
  int rc = pl.bn == 256 ? dg_launch<256, false>(ma, mw, p, (uint32_t)di.sm_count, stream)
         : pl.bn == 128 ? dg_launch<128, false>(ma, mw, p, (uint32_t)di.sm_count, stream)
                        : dg_launch<64, false>(ma, mw, p, (uint32_t)di.sm_count, stream);
  if (rc != CUTB_OK || pl.ksplit <= 1) return rc;
  dense_splitk_reduce_kernel<<<(unsigned)(((size_t)d.M * d.N + 255) / 256), 256, 0, stream>>>(p);
  CUTB_CUDA_TRY(cudaGetLastError());
  return CUTB_OK;
}

int moe_gemm_tc_launch(const cutb_moe_desc &d, cudaStream_t stream) {
  DeviceInfo di;
  if (int rc = get_device_info(&di)) return rc;
  const uint32_t sms = (uint32_t)di.sm_count, rows = d.n_tokens * d.top;
  DgParams p{};
  p.C = d.C, p.status = d.status, p.M = rows, p.K = d.K, p.N = d.N, p.ldc = (uint32_t)d.ldc;
  p.offsets = d.offsets, p.experts = d.experts, p.glu = GluParams{d.glu, d.alpha, d.beta, d.limit};
  p.c_bf16 = d.c_dtype == CUTB_BF16;
  p.nk = p.nk_per = (d.K + DG_BK - 1) / DG_BK, p.ksplit = 1;
  p.a_box_rows = rows >= DG_BM ? DG_BM : (rows + 7) / 8 * 8;
  // row tiles: every expert in use ends in a part-filled one.  Widths by the time of their waves, as in dg_plan.
  const uint32_t used = d.experts < rows ? d.experts : rows, likely = rows / DG_BM + (used + 1) / 2;
  int bn = 256;
  uint64_t best = ~0ull;
  const struct { int bn; uint32_t cost; } kinds[] = {{256, 100}, {128, 66}, {64, 62}};
  for (const auto &kind : kinds) {
    const uint64_t cost = (uint64_t)((likely * ((d.N + kind.bn - 1) / kind.bn) + sms - 1) / sms) * kind.cost;
    if (cost < best) best = cost, bn = kind.bn;
  }
  p.tiles_m = rows / DG_BM + used, p.tiles_n = (d.N + bn - 1) / bn;
  CUtensorMap ma, mw;
  if (int rc = make_tmap_sw128(&ma, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, d.A, rows, d.K, d.lda * 2, p.a_box_rows)) return rc;
  if (int rc = make_tmap_sw128(&mw, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, d.W, d.experts * d.N, d.K, (uint64_t)d.ldw * 2, (uint32_t)bn)) return rc;
  return bn == 256 ? dg_launch<256, true>(ma, mw, p, sms, stream)
       : bn == 128 ? dg_launch<128, true>(ma, mw, p, sms, stream)
                   : dg_launch<64, true>(ma, mw, p, sms, stream);
}

namespace {
int ds_launch(const DsParams &p, bool a_bf16, uint32_t tiles_m, uint32_t batch, cudaStream_t stream) {
  const dim3 grid((p.N + 63) / 64, tiles_m, batch);
  if (a_bf16) CUTB_CUDA_TRY(launch_pdl(dense_gemm_simt_kernel<__nv_bfloat16>, grid, dim3(256), 0, stream, p));
  else CUTB_CUDA_TRY(launch_pdl(dense_gemm_simt_kernel<float>, grid, dim3(256), 0, stream, p));
  return CUTB_OK;
}
}  // namespace

int dense_gemm_simt_launch(const cutb_dense_desc &d, cudaStream_t stream) {
  DsParams p{};
  p.A = d.A, p.W = reinterpret_cast<const __nv_bfloat16 *>(d.W), p.bias = d.bias, p.C = d.C;
  p.lda = d.lda, p.ldw = d.ldw, p.ldc = d.ldc, p.M = d.M, p.N = d.N, p.K = d.K, p.a_batch = d.a_batch, p.c_batch = d.c_batch;
  p.c_bf16 = d.c_dtype == CUTB_BF16, p.unary = d.unary_op;
  return ds_launch(p, d.a_dtype == CUTB_BF16, (d.M + 63) / 64, d.batch ? d.batch : 1, stream);
}

int moe_gemm_simt_launch(const cutb_moe_desc &d, cudaStream_t stream) {
  DsParams p{};
  const uint32_t rows = d.n_tokens * d.top, used = d.experts < rows ? d.experts : rows;
  p.A = d.A, p.W = reinterpret_cast<const __nv_bfloat16 *>(d.W), p.C = d.C;
  p.lda = (uint32_t)d.lda, p.ldw = d.ldw, p.ldc = (uint32_t)d.ldc, p.M = rows, p.N = d.N, p.K = d.K;
  p.c_bf16 = d.c_dtype == CUTB_BF16, p.offsets = d.offsets, p.experts = d.experts, p.glu = GluParams{d.glu, d.alpha, d.beta, d.limit};
  return ds_launch(p, d.a_dtype == CUTB_BF16, rows / 64 + used, 1, stream);
}

}  // namespace cutb
