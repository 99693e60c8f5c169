// Decode mat-vecs of a mixture of experts for one token, with a dense matrix beside the experts in the same launch, so that a
// layer whose mixer and feed-forward read one normed input needs no launches of its own for the experts.  bf16 weights, fp32
// activations and accumulation, HBM-bound: only the chosen experts' rows are read, each once.
//
// UP    the router's choice is made by every block from the logits (a few hundred cycles); tiles are row pairs: first the dense
//       matrix's (whose input may be RMS-normed on the way in), then gate and up rows of every chosen expert, whose outputs meet
//       in the gated unit, scaled by the expert's weight.
// DOWN  a tile is one output row: the dense matrix's row and the same row of every chosen expert, one running sum.
//
// A tile belongs to one warp, tiles are dealt over the SMs first; a lane takes every 32nd 16-byte piece, two steps of loads are
// in flight.  The first steps of the dense rows are issued before the wait for the previous kernel.
#include <cuda_bf16.h>

#include "common.cuh"
#include "dense_common.cuh"
#include "kernels.h"
#include "moe_common.cuh"
#include "norm_stage.cuh"

namespace cutb {
namespace {

constexpr int EX_MIN_WARPS = 16;
constexpr int ex_max_warps(bool up) { return up ? 24 : 28; }
constexpr uint32_t EX_MAX_TOP = 64;

struct ExParams {
  const uint4 *Wd, *W;
  const float *logits, *x, *xd, *xd_norm_w;
  float *act, *C;
  uint32_t *ids;
  uint32_t experts, top, width, ff;
  uint32_t Nd, Kd, Kd8, ldwd8;  // Kd8 0: no dense companion
  uint32_t K8, ldw8;            // pieces of an expert's row
  uint32_t dense_tiles, ntiles;
  float eps;
  GluParams glu;
};

template <bool UP> __global__ void __launch_bounds__(32 * ex_max_warps(UP), 1) expert_matvec_kernel(const ExParams p) {
  constexpr int R = UP ? 2 : 1, UNR = UP ? 2 : 4;
  extern __shared__ __align__(16) float ex_smem[];
  __shared__ uint32_t ids[EX_MAX_TOP];
  __shared__ float weights[EX_MAX_TOP];
  const uint32_t x8 = p.Kd8 + (UP ? p.K8 : p.top * p.K8);  // pieces of the staged input
  float4 *lo = reinterpret_cast<float4 *>(ex_smem), *hi = lo + x8;
  float *stage = ex_smem + 8 * x8;  // UP: logits, then the norm's rows
  const uint32_t tid = threadIdx.x, nt = blockDim.x, lane = tid & 31, warp = tid >> 5;
  const uint32_t tstep = gridDim.x * (nt >> 5), first = warp * gridDim.x + blockIdx.x;
  asm volatile("griddepcontrol.launch_dependents;" ::: "memory");

  // a tile is a sequence of segments (one in UP): consecutive pieces of R rows against a stretch of the staged input
  struct Segment {
    const uint4 *w;
    uint32_t step, k8;  // distance of the rows (0: there is no second one), pieces
  };
  auto is_dense = [&](uint32_t tile, uint32_t s) { return UP ? tile < p.dense_tiles : p.Kd8 && s == 0; };
  auto segment = [&](uint32_t tile, uint32_t s) {
    Segment g;
    if constexpr (UP) {
      if (tile < p.dense_tiles) {
        g.w = p.Wd + (size_t)tile * R * p.ldwd8, g.step = tile * R + 1 < p.Nd ? p.ldwd8 : 0, g.k8 = p.Kd8;
      } else {
        const uint32_t t = tile - p.dense_tiles, k = t / p.ff;
        g.w = p.W + ((size_t)ids[k] * 2 * p.ff + 2 * (t - k * p.ff)) * p.ldw8, g.step = p.ldw8, g.k8 = p.K8;
      }
    } else {
      const uint32_t k = s - (p.Kd8 ? 1 : 0);
      if (p.Kd8 && s == 0) g.w = p.Wd + (size_t)tile * p.ldwd8, g.k8 = p.Kd8;
      else g.w = p.W + ((size_t)ids[k] * p.width + tile) * p.ldw8, g.k8 = p.K8;
      g.step = 0;
    }
    return g;
  };
  const uint32_t nseg = UP ? 1 : p.top + (p.Kd8 ? 1 : 0);
  uint32_t l_tile = first, l_s = 0, l_k = lane;
  bool l_new = true;  // the segment under the load cursor has not been looked up (that of an expert needs its number)
  Segment lg{};
  auto load = [&](uint4 (&w)[UNR][R]) {
    if (l_tile >= p.ntiles) return;
    if (l_new) lg = segment(l_tile, l_s), l_new = false;
#pragma unroll
    for (int u = 0; u < UNR; ++u)
#pragma unroll
      for (int r = 0; r < R; ++r) {
        const uint32_t k = l_k + 32 * u;
        w[u][r] = k < lg.k8 && (r == 0 || lg.step) ? ld_stream(lg.w + (size_t)r * lg.step + k) : make_uint4(0, 0, 0, 0);
      }
    l_k += 32 * UNR;
    if (l_k >= lg.k8 + lane) {  // (the same step in every lane)
      l_k = lane, l_new = true;
      if (++l_s == nseg) l_s = 0, l_tile += tstep;
    }
  };
  // loads of the dense matrix are on their way before the wait for the previous kernel; the experts are not known then
  uint4 wa[UNR][R], wb[UNR][R];
  uint32_t early = 0;
  if (l_tile < p.ntiles && is_dense(l_tile, l_s)) {
    load(wa);
    early = 1;
    if (l_tile < p.ntiles && is_dense(l_tile, l_s)) {
      load(wb);
      early = 2;
    }
  }
  asm volatile("griddepcontrol.wait;" ::: "memory");

  auto put1 = [&](uint32_t at, uint32_t i, float v) { ex_smem[(i & 4 ? 4 * x8 : 0) + (at + (i >> 3)) * 4 + (i & 3)] = v; };
  auto put_row = [&](uint32_t at, const float *x, uint32_t n, uint32_t pieces) {
    for (uint32_t i = tid; i < 8 * pieces; i += nt) put1(at, i, i < n ? x[i] : 0.f);
  };
  if constexpr (UP) {
    const uint32_t epad = (p.experts + 3) / 4 * 4;
    float *z = stage;
    for (uint32_t e = tid; e < epad; e += nt) z[e] = e < p.experts ? p.logits[e] : -INFINITY;
    if (tid < EX_MAX_TOP) ids[tid] = 0;
    put_row(p.Kd8, p.x, p.width, p.K8);
    if (p.Kd8) {
      if (p.xd_norm_w) {
        for (uint32_t i = p.Kd + tid; i < 8 * p.Kd8; i += nt) put1(0, i, 0.f);
        NormStage n{};
        n.x = p.xd, n.pre_w = p.xd_norm_w, n.dim = p.Kd, n.groups = 1, n.eps = p.eps;
        auto n1 = [&](uint32_t i, float v) { put1(0, i, v); };
        auto n4 = [&](uint32_t i, float4 v) { (i & 4 ? hi : lo)[i >> 3] = v; };
        if (norm_stage_fits(p.Kd, 1, nt, 2)) stage_norm_regs<2, true>(n, z + epad, nullptr, false, n4);
        else stage_norm(n, z + epad, false, n4, n1);
      } else {
        put_row(0, p.xd, p.Kd, p.Kd8);
      }
    }
    __syncthreads();
    choose_experts(z, p.experts, p.top, tid, nt, ids);
    __syncthreads();
    if (tid < p.top) {
      weights[tid] = choice_weight(z, ids, p.top, tid);
      if (blockIdx.x == 0) p.ids[tid] = ids[tid];
    }
  } else {
    if (tid < p.top) ids[tid] = min(p.ids[tid], p.experts - 1);
    if (p.Kd8) put_row(0, p.xd, p.Kd, p.Kd8);
    for (uint32_t k = 0; k < p.top; ++k) put_row(p.Kd8 + k * p.K8, p.act + (size_t)k * p.ff, p.ff, p.K8);
  }
  __syncthreads();

  uint32_t tile = first, seg = 0, k = lane, c_k8 = 0, c_x8 = 0;
  auto at = [&]() {
    if constexpr (UP) c_k8 = tile < p.dense_tiles ? p.Kd8 : p.K8, c_x8 = tile < p.dense_tiles ? 0 : p.Kd8;
    else if (p.Kd8 && seg == 0) c_k8 = p.Kd8, c_x8 = 0;
    else c_k8 = p.K8, c_x8 = p.Kd8 + (seg - (p.Kd8 ? 1 : 0)) * p.K8;
  };
  at();
  float acc[R];
#pragma unroll
  for (int r = 0; r < R; ++r) acc[r] = 0.f;
  auto use = [&](const uint4 (&w)[UNR][R]) {
#pragma unroll
    for (int u = 0; u < UNR; ++u)
      if (k + 32 * u < c_k8) {
        const float4 a = lo[c_x8 + k + 32 * u], b = hi[c_x8 + k + 32 * u];
#pragma unroll
        for (int r = 0; r < R; ++r) fma8(acc[r], w[u][r], a, b);
      }
    k += 32 * UNR;
    if (k < c_k8 + lane) return;
    k = lane;
    if (++seg < nseg) {
      at();
      return;
    }
    // the tile's last piece
    seg = 0;
#pragma unroll
    for (int r = 0; r < R; ++r) acc[r] = warp_sum(acc[r]);
    if constexpr (UP) {
      if (tile < p.dense_tiles) {
        if (lane < R && tile * R + lane < p.Nd) p.C[tile * R + lane] = lane ? acc[R - 1] : acc[0];
      } else if (lane == 0) {
        const uint32_t t = tile - p.dense_tiles;
        p.act[t] = weights[t / p.ff] * glu(p.glu, acc[0], acc[R - 1]);
      }
    } else {
      if (lane == 0) p.C[tile] = acc[0];
    }
#pragma unroll
    for (int r = 0; r < R; ++r) acc[r] = 0.f;
    tile += tstep;
    at();
  };
  if (early < 1) load(wa);
  if (early < 2) load(wb);
  while (tile < p.ntiles) {
    use(wa);
    load(wa);
    if (tile >= p.ntiles) break;
    use(wb);
    load(wb);
  }
}

uint32_t ex_smem_bytes(const cutb_expert_desc &d, bool up) {
  const uint32_t Kd8 = d.Wd ? (d.Kd + 7) / 8 : 0, K8 = ((up ? d.width : d.ff) + 7) / 8;
  return 4 * (8 * (Kd8 + (up ? K8 : d.top * K8)) + (up ? (d.experts + 3) / 4 * 4 + (d.Wd && d.xd_norm_w ? norm_stage_floats(d.Kd, 1) : 0) : 0));
}

template <bool UP> int ex_launch(const cutb_expert_desc &d, cudaStream_t stream) {
  DeviceInfo di;
  if (int rc = get_device_info(&di)) return rc;
  ExParams p{};
  p.Wd = reinterpret_cast<const uint4 *>(d.Wd), p.W = reinterpret_cast<const uint4 *>(d.W);
  p.logits = d.logits, p.x = d.x, p.xd = d.xd, p.xd_norm_w = d.xd_norm_w, p.act = d.act, p.C = d.C, p.ids = d.ids;
  p.experts = d.experts, p.top = d.top, p.width = d.width, p.ff = d.ff;
  if (d.Wd) p.Nd = d.Nd, p.Kd = d.Kd, p.Kd8 = (d.Kd + 7) / 8, p.ldwd8 = d.ldwd / 8;
  p.K8 = ((UP ? d.width : d.ff) + 7) / 8, p.ldw8 = d.ldw / 8;
  p.dense_tiles = UP ? (p.Nd + 1) / 2 : 0, p.ntiles = UP ? p.dense_tiles + d.top * d.ff : d.width;
  p.eps = d.eps, p.glu = GluParams{CUTB_GLU_CLAMPED, d.alpha, d.beta, d.limit};
  static bool configured[64] = {};
  int dev = 0;
  CUTB_CUDA_TRY(cudaGetDevice(&dev));
  if (dev < 0 || dev >= 64 || !configured[dev]) {
    CUTB_CUDA_TRY(cudaFuncSetAttribute(expert_matvec_kernel<UP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)di.smem_optin - 2048));
    if (dev >= 0 && dev < 64) configured[dev] = true;
  }
  const uint32_t sms = (uint32_t)di.sm_count, per_sm = (p.ntiles + sms - 1) / sms, most = ex_max_warps(UP), turns = (per_sm + most - 1) / most;
  uint32_t warps = (per_sm + turns - 1) / turns;
  if (warps < EX_MIN_WARPS) warps = EX_MIN_WARPS;
  const dim3 grid(p.ntiles < sms ? p.ntiles : sms), block(32 * warps);
  const uint32_t smem = ex_smem_bytes(d, UP);
  if (d.flags & CUTB_FLAG_NO_OVERLAP) {
    expert_matvec_kernel<UP><<<grid, block, smem, stream>>>(p);
    CUTB_CUDA_TRY(cudaGetLastError());
  } else {
    CUTB_CUDA_TRY(launch_pdl(expert_matvec_kernel<UP>, grid, block, smem, stream, p));
  }
  return CUTB_OK;
}

}  // namespace

bool expert_matvec_supported(const cutb_expert_desc &d, bool up) { return d.top <= EX_MAX_TOP && ex_smem_bytes(d, up) <= 220 * 1024; }
int expert_up_launch(const cutb_expert_desc &d, cudaStream_t stream) { return ex_launch<true>(d, stream); }
int expert_down_launch(const cutb_expert_desc &d, cudaStream_t stream) { return ex_launch<false>(d, stream); }

}  // namespace cutb
