// Mixture of experts: routing, dispatch and the experts' matrix products.
//
//   moe_route      one warp per token: softmax or sigmoid of the router logits (fp32, from a GEMM output or its split-K
//                  partials), the best groups of neighbouring experts by their largest score, the `top` largest scores
//                  inside those groups; each choice takes a ticket of its expert's counter
//   moe_dispatch   segment offsets from the counters, one copy of every chosen token's row into its expert's segment,
//                  multiplied by the choice's weight if the weights belong to the experts' inputs
//   moe_gemm       grouped GEMM on tcgen05: one persistent launch over the tiles of every expert's segment, the
//                  number of rows of a segment is read on the device (nothing about the routing reaches the host, so a
//                  decode step with a mixture is captured in a CUDA graph like any other); gelu, squared relu or
//                  silu(gate) * up in the epilogue. With one always-on segment it is a dense feed-forward's first product.
// The (weighted) sum of a token's expert outputs is taken by the kernel that updates the residual stream (residual_norm.cu,
// stream_update.cu).
//
// Equal scores: the expert (or group) with the smaller number wins.
#include "act_io.cuh"
#include "moe_segments.cuh"
#include "rpeg_kernels.h"

namespace rpeg {

constexpr int MOE_MAX_SEGMENTS = 1024;
constexpr int ROUTE_WARPS = 4;

// Index of the largest of the non-negative values v[lane + 32 j] whose bit j is set in the lane's mask, ties to the smaller
// index; every lane returns it (-1: no bit set anywhere). Non-negative floats order like their bit patterns.
__device__ __forceinline__ int warp_argmax(const float* v, int n, uint32_t mask, int lane) {
  uint32_t best = 0u;
  int at = 0x7fffffff;
  for (int j = 0, i = lane; i < n; ++j, i += 32) {
    const uint32_t key = (mask >> j) & 1u ? __float_as_uint(v[i]) + 1u : 0u;
    if (key > best) { best = key; at = i; }
  }
  const uint32_t top = __reduce_max_sync(0xffffffffu, best);
  if (top == 0u) return -1;
  return static_cast<int>(__reduce_min_sync(0xffffffffu, best == top ? static_cast<uint32_t>(at) : 0x7fffffffu));
}

__global__ void __launch_bounds__(ROUTE_WARPS * 32)
moe_route_kernel(const float* __restrict__ logits, int splits, long long stride, int ld, int rows, int E, int n_groups, int keep, int top,
                 int renorm, int sigmoid, int* __restrict__ ids, float* __restrict__ wts, int* __restrict__ ticket, int* __restrict__ counts) {
  griddep_launch();
  griddep_wait();
  extern __shared__ float route_sm[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int t = blockIdx.x * ROUTE_WARPS + warp;
  if (t >= rows) return;
  float* sc = route_sm + warp * (E + n_groups + top);     // per warp: E scores, n_groups group scores, the choices
  float* gs = sc + E;
  int* pick = reinterpret_cast<int*>(gs + n_groups);
  const float* lr = logits + static_cast<size_t>(t) * ld;
  float mx = -INFINITY;
  for (int e = lane; e < E; e += 32) {
    float z = lr[e];
#pragma unroll 8
    for (int s = 1; s < splits; ++s) z += lr[s * stride + e];
    sc[e] = z;
    mx = fmaxf(mx, z);
  }
  if (sigmoid) {
    for (int e = lane; e < E; e += 32) sc[e] = sigmoidf(sc[e]);
  } else {
    mx = warp_max(mx);
    float sum = 0.f;
    for (int e = lane; e < E; e += 32) {
      const float p = expf(sc[e] - mx);
      sc[e] = p;
      sum += p;
    }
    const float inv = 1.f / warp_sum(sum);
    for (int e = lane; e < E; e += 32) sc[e] *= inv;
  }
  __syncwarp();
  const int per = E / n_groups;
  uint32_t open = 0xffffffffu;                             // bit j: expert lane + 32 j may still be chosen (E <= 1024)
  if (keep < n_groups) {
    for (int g = lane; g < n_groups; g += 32) {
      float b = sc[g * per];
      for (int i = 1; i < per; ++i) b = fmaxf(b, sc[g * per + i]);
      gs[g] = b;
    }
    __syncwarp();
    open = 0u;
    uint32_t gopen = 0xffffffffu;
    for (int k = 0; k < keep; ++k) {
      const int g = max(warp_argmax(gs, n_groups, gopen, lane), 0);
      if ((g & 31) == lane) gopen &= ~(1u << (g >> 5));
      for (int j = 0, e = lane; e < E; ++j, e += 32)
        if (e >= g * per && e < (g + 1) * per) open |= 1u << j;
    }
  }
  float chosen = 0.f;
  for (int k = 0; k < top; ++k) {
    const int e = max(warp_argmax(sc, E, open, lane), 0);  // the host guarantees top <= keep * per
    if ((e & 31) == lane) open &= ~(1u << (e >> 5));
    chosen += sc[e];
    if (lane == 0) pick[k] = e;
  }
  __syncwarp();
  const float scale = renorm ? 1.f / chosen : 1.f;
  for (int k = lane; k < top; k += 32) {
    const int e = pick[k];
    const size_t o = static_cast<size_t>(t) * top + k;
    ids[o] = e;
    wts[o] = sc[e] * scale;
    ticket[o] = atomicAdd(&counts[e], 1);
  }
}

// One CTA per token. Every CTA sums the counters below its token's experts itself (a few hundred words from L2).
// `wts`: weights of the choices, multiplied into the copies (null: plain copies).
__device__ __forceinline__ uint4 scaled(uint4 v, float w, const float*) {
  return make_uint4(__float_as_uint(__uint_as_float(v.x) * w), __float_as_uint(__uint_as_float(v.y) * w), __float_as_uint(__uint_as_float(v.z) * w),
                    __float_as_uint(__uint_as_float(v.w) * w));
}
__device__ __forceinline__ uint4 scaled(uint4 v, float w, const __nv_bfloat16*) {
  auto two = [&](uint32_t u) -> uint32_t {
    const float2 f = unpack_bf16x2(u);
    return pack_bf16x2(f.x * w, f.y * w);
  };
  return make_uint4(two(v.x), two(v.y), two(v.z), two(v.w));
}

template <typename T>
__global__ void __launch_bounds__(128)
moe_dispatch_kernel(const T* __restrict__ x, int dp, const int* __restrict__ ids, const int* __restrict__ ticket, const float* __restrict__ wts,
                    const int* __restrict__ counts, int E, int top, T* __restrict__ xs, int* __restrict__ row_of, int* __restrict__ seg_off) {
  griddep_launch();
  griddep_wait();
  extern __shared__ int off_sm[];             // [E + 1] segment offsets, then [top] rows
  int* rows_sm = off_sm + E + 1;
  const int t = blockIdx.x;
  if (threadIdx.x < 32) {
    int carry = 0;
    for (int e0 = 0; e0 < E; e0 += 32) {
      const int e = e0 + threadIdx.x;
      int v = e < E ? counts[e] : 0;
      const int own = v;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int u = __shfl_up_sync(0xffffffffu, v, o);
        if (static_cast<int>(threadIdx.x) >= o) v += u;
      }
      if (e < E) off_sm[e] = carry + v - own;
      carry += __shfl_sync(0xffffffffu, v, 31);
    }
    if (threadIdx.x == 0) off_sm[E] = carry;
  }
  __syncthreads();
  for (int k = threadIdx.x; k < top; k += blockDim.x) {
    const size_t o = static_cast<size_t>(t) * top + k;
    const int r = off_sm[ids[o]] + ticket[o];
    rows_sm[k] = r;
    row_of[o] = r;
  }
  if (t == 0)
    for (int e = threadIdx.x; e <= E; e += blockDim.x) seg_off[e] = off_sm[e];
  __syncthreads();
  const int nv = static_cast<int>(dp * sizeof(T) / 16);
  const uint4* src = reinterpret_cast<const uint4*>(x + static_cast<size_t>(t) * dp);
  for (int i = threadIdx.x; i < nv; i += blockDim.x) {
    const uint4 v = src[i];
    for (int k = 0; k < top; ++k)
      reinterpret_cast<uint4*>(xs + static_cast<size_t>(rows_sm[k]) * dp)[i] = wts == nullptr ? v : scaled(v, wts[static_cast<size_t>(t) * top + k], x);
  }
}

// ---------------------------------------------------------------------------------- grouped GEMM
//   C[r, 0..N) = act( A[r, 0..K) * B_s[0..N, 0..K)^T )   for every row r of segment s;  B_s = rows [s * N, s * N + N) of B
// (gated: B_s has 2 N rows, gate then up; a tile of BN accumulator columns holds BN / 2 gate columns and the BN / 2 up columns of
// the same outputs)
// Same structure as the dense kernel in gemm.cu (TMA producer warp, one MMA-issuing thread, four epilogue warps,
// accumulator double buffered in TMEM). A tile is 128 rows of ONE segment: it starts at any row (the row coordinate
// of a TMA box is free) and the rows that belong to the next segment are computed and not stored. Always-on
// segments may read their rows from a second operand (the tokens in their original order) instead of a copy.
constexpr int MG_BM = 128, MG_BK = 64, MG_THREADS = 192;
constexpr int MG_SMEM_BUDGET = 227 * 1024 - 2048 - (MOE_MAX_SEGMENTS + 1) * 4;

template <int BN>
struct MoeGemmCfg {
  static constexpr int A_BYTES = MG_BM * MG_BK * 2;
  static constexpr int B_BYTES = BN * MG_BK * 2;
  static constexpr int STAGE_BYTES = A_BYTES + B_BYTES;
  static constexpr int STAGES = MG_SMEM_BUDGET / STAGE_BYTES > 8 ? 8 : MG_SMEM_BUDGET / STAGE_BYTES;
  static constexpr int TMEM_COLS = 2 * BN;
  static constexpr int SMEM_BYTES = STAGES * STAGE_BYTES + 1024 + 512 + (MOE_MAX_SEGMENTS + 1) * 4;
};

template <int BN, int ACT>
__global__ void __launch_bounds__(MG_THREADS, 1)
moe_gemm_kernel(const __grid_constant__ CUtensorMap tmap_a, const __grid_constant__ CUtensorMap tmap_x,
                const __grid_constant__ CUtensorMap tmap_b, __nv_bfloat16* __restrict__ C, const int* __restrict__ seg_off, int n_routed,
                int n_shared, int seg_rows, int shared_from_x, int N, int K, int ldc, int a_rows, int* status) {
  using Cfg = MoeGemmCfg<BN>;
  constexpr int STAGES = Cfg::STAGES;
  constexpr int TN = ACT == FF_SWIGLU ? BN / 2 : BN;   // output columns per tile
  const uint32_t stage_tx = static_cast<uint32_t>(Cfg::B_BYTES + a_rows * MG_BK * 2);
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint64_t* full_bar = reinterpret_cast<uint64_t*>(smem + STAGES * Cfg::STAGE_BYTES);
  uint64_t* empty_bar = full_bar + STAGES;
  uint64_t* tfull_bar = empty_bar + STAGES;
  uint64_t* tempty_bar = tfull_bar + 2;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(tempty_bar + 2);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  int* mt0 = reinterpret_cast<int*>(smem + STAGES * Cfg::STAGE_BYTES + 512);   // [segments + 1] first M tile of a segment

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int S = n_routed + n_shared;
  if (threadIdx.x == 0) {
    for (int s = 0; s < STAGES; ++s) { mbar_init(&full_bar[s], 1); mbar_init(&empty_bar[s], 1); }
    for (int b = 0; b < 2; ++b) { mbar_init(&tfull_bar[b], 1); mbar_init(&tempty_bar[b], 4); }
    *abort_flag = 0;
    fence_mbar_init();
  }
  if (warp == 0 && lane == 0) {
    tma_prefetch_desc(&tmap_a);
    tma_prefetch_desc(&tmap_x);
    tma_prefetch_desc(&tmap_b);
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, Cfg::TMEM_COLS);
    tmem_relinquish();
  }
  griddep_launch();
  griddep_wait();
  if (warp == 2) {                              // M tiles before every segment
    int carry = 0;
    for (int s0 = 0; s0 < S; s0 += 32) {
      const int s = s0 + lane;
      int v = s < S ? (moe_segment(seg_off, n_routed, seg_rows, s).rows + MG_BM - 1) / MG_BM : 0;
      const int own = v;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int u = __shfl_up_sync(0xffffffffu, v, o);
        if (lane >= o) v += u;
      }
      if (s < S) mt0[s] = carry + v - own;
      carry += __shfl_sync(0xffffffffu, v, 31);
    }
    if (lane == 0) mt0[S] = carry;
  }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem_base = *tmem_slot;
  const int n_tiles = (N + TN - 1) / TN;
  const int num_items = mt0[S] * n_tiles;
  const int num_kb = (K + MG_BK - 1) / MG_BK;

  // Items of a segment: its M tiles vary fastest, so the CTAs that run side by side share a weight tile.
  struct Item { int seg, tm, tn; };
  auto item = [&](int w) -> Item {
    int lo = 0, hi = S;                         // largest s with mt0[s] * n_tiles <= w and a non-empty segment
    while (hi - lo > 1) {
      const int mid = (lo + hi) >> 1;
      if (mt0[mid] * n_tiles <= w) lo = mid; else hi = mid;
    }
    const int m_tiles = mt0[lo + 1] - mt0[lo];
    const int r = w - mt0[lo] * n_tiles;
    return {lo, r % m_tiles, r / m_tiles};
  };

  if (warp == 0) {
    if (lane == 0) {
      int stage = 0;
      uint32_t phase = 0;
      for (int w = blockIdx.x; w < num_items; w += gridDim.x) {
        const Item it = item(w);
        const MoeSegment sg = moe_segment(seg_off, n_routed, seg_rows, it.seg);
        const bool from_x = shared_from_x && it.seg >= n_routed;
        const CUtensorMap* ta = from_x ? &tmap_x : &tmap_a;
        const int m0 = it.tm * MG_BM + (from_x ? 0 : static_cast<int>(sg.row0));
        const int b0 = it.seg * (ACT == FF_SWIGLU ? 2 * N : N) + it.tn * TN;
        for (int kb = 0; kb < num_kb; ++kb) {
          if (!mbar_wait(&empty_bar[stage], phase ^ 1u, abort_flag, status, 700)) goto producer_done;
          uint8_t* sa = smem + stage * Cfg::STAGE_BYTES;
          mbar_expect_tx(&full_bar[stage], stage_tx);
          tma_load_2d(sa + Cfg::A_BYTES, &tmap_b, &full_bar[stage], kb * MG_BK, b0);
          if constexpr (ACT == FF_SWIGLU)      // the boxes are TN rows high: gate rows, then the up rows of the same columns
            tma_load_2d(sa + Cfg::A_BYTES + TN * MG_BK * 2, &tmap_b, &full_bar[stage], kb * MG_BK, b0 + N);
          tma_load_2d(sa, ta, &full_bar[stage], kb * MG_BK, m0);
          if (++stage == STAGES) { stage = 0; phase ^= 1u; }
        }
      }
    producer_done:;
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t idesc = make_idesc_bf16(MG_BM, BN, 0, 0);
      int stage = 0, buf = 0;
      uint32_t phase = 0, acc_phase = 0;
      for (int w = blockIdx.x; w < num_items; w += gridDim.x) {
        if (!mbar_wait(&tempty_bar[buf], acc_phase ^ 1u, abort_flag, status, 710)) goto mma_done;
        tc_fence_after_sync();
        const uint32_t tacc = tmem_base + static_cast<uint32_t>(buf * BN);
        for (int kb = 0; kb < num_kb; ++kb) {
          if (!mbar_wait(&full_bar[stage], phase, abort_flag, status, 711)) goto mma_done;
          tc_fence_after_sync();
          const uint32_t sa = smem_u32(smem + stage * Cfg::STAGE_BYTES);
          const uint32_t sb = sa + Cfg::A_BYTES;
#pragma unroll
          for (int k = 0; k < MG_BK / 16; ++k)
            umma_bf16_ss(tacc, make_smem_desc_sw128(sa + k * 32, 16, 1024), make_smem_desc_sw128(sb + k * 32, 16, 1024), idesc,
                         (kb | k) != 0 ? 1u : 0u);
          umma_commit(&empty_bar[stage]);
          if (++stage == STAGES) { stage = 0; phase ^= 1u; }
        }
        umma_commit(&tfull_bar[buf]);
        if (++buf == 2) { buf = 0; acc_phase ^= 1u; }
      }
    mma_done:;
    }
  } else {
    const int quad = warp & 3;
    int buf = 0;
    uint32_t acc_phase = 0;
    for (int w = blockIdx.x; w < num_items; w += gridDim.x) {
      const Item it = item(w);
      const MoeSegment sg = moe_segment(seg_off, n_routed, seg_rows, it.seg);
      const int r = it.tm * MG_BM + quad * 32 + lane;
      const bool live = r < sg.rows;
      const bool warp_live = it.tm * MG_BM + quad * 32 < sg.rows;    // decode: most quads of a tile hold no row at all
      const int n0 = it.tn * TN;
      if (!__all_sync(0xffffffffu, mbar_wait(&tfull_bar[buf], acc_phase, abort_flag, status, 720))) break;
      tc_fence_after_sync();
      const uint32_t taddr = tmem_base + (static_cast<uint32_t>(quad * 32) << 16) + static_cast<uint32_t>(buf * BN);
      if (warp_live) {
        __nv_bfloat16* crow = C + static_cast<size_t>(sg.row0 + r) * ldc;
#pragma unroll 1
        for (int c = 0; c < TN / 32; ++c) {
          const int col0 = n0 + c * 32;
          if (col0 >= N) break;                                      // uniform over the warp
          uint32_t v[32], u[ACT == FF_SWIGLU ? 32 : 1];
          tmem_ld_32x32(taddr + c * 32, v);
          if constexpr (ACT == FF_SWIGLU) tmem_ld_32x32(taddr + TN + c * 32, u);
          tmem_wait_ld();
          if (live) {
#pragma unroll
            for (int q = 0; q < 4; ++q) {
              if (col0 + q * 8 < N) {
                uint32_t o[4];
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                  float a = __uint_as_float(v[q * 8 + 2 * e]), b = __uint_as_float(v[q * 8 + 2 * e + 1]);
                  if constexpr (ACT == FF_SWIGLU) {
                    a = silu_mul(a, __uint_as_float(u[q * 8 + 2 * e]));
                    b = silu_mul(b, __uint_as_float(u[q * 8 + 2 * e + 1]));
                  } else {
                    a = ff_act<ACT>(a);
                    b = ff_act<ACT>(b);
                  }
                  o[e] = pack_bf16x2(a, b);
                }
                *reinterpret_cast<uint4*>(crow + col0 + q * 8) = make_uint4(o[0], o[1], o[2], o[3]);
              }
            }
          }
        }
      }
      tc_fence_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(&tempty_bar[buf]);
      if (++buf == 2) { buf = 0; acc_phase ^= 1u; }
    }
  }

  __syncwarp();
  if (*abort_flag) __nanosleep(200000);
  tc_fence_before_sync();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after_sync();
    tmem_dealloc(tmem_base, Cfg::TMEM_COLS);
  }
}

int make_tmap_bf16_2d(CUtensorMap* out, const void* ptr, uint64_t inner, uint64_t outer, uint64_t ld, uint32_t box_inner,
                      uint32_t box_outer);

template <int BN, int ACT>
static int launch_moe_gemm(const CUtensorMap& ta, const CUtensorMap& tx, const CUtensorMap& tb, void* C, const int* seg_off, int n_routed,
                           int n_shared, int seg_rows, int from_x, int N, int K, int ldc, int a_rows, long long max_tiles, int num_sms,
                           int* status, cudaStream_t stream) {
  using Cfg = MoeGemmCfg<BN>;
  auto kern = moe_gemm_kernel<BN, ACT>;
  static bool configured = false;
  if (!configured) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, Cfg::SMEM_BYTES) != cudaSuccess) return -20;
    configured = true;
  }
  const unsigned grid = static_cast<unsigned>(max_tiles < num_sms ? max_tiles : num_sms);
  const cudaError_t e = launch_pdl(kern, dim3(grid), dim3(MG_THREADS), static_cast<size_t>(Cfg::SMEM_BYTES), stream, ta, tx, tb,
                                   static_cast<__nv_bfloat16*>(C), seg_off, n_routed, n_shared, seg_rows, from_x, N, K, ldc, a_rows, status);
  return e == cudaSuccess ? 0 : -21;
}

}  // namespace rpeg

using namespace rpeg;
#define STREAM(s) reinterpret_cast<cudaStream_t>(s)

extern "C" int rpeg_moe_route(const float* logits, int splits, long long stride, int ld, int rows, int E, int n_groups, int keep, int top,
                              int renorm, int sigmoid, int* ids, float* wts, int* ticket, int* counts, void* stream) {
  if (rows <= 0) return 0;
  if (E < 1 || n_groups < 1 || E % n_groups || keep < 1 || keep > n_groups || top < 1 || top > keep * (E / n_groups)) return -2;
  if (E > MOE_MAX_SEGMENTS) return -3;
  const size_t smem = static_cast<size_t>(ROUTE_WARPS) * (E + n_groups + top) * 4;
  if (smem > 48 * 1024) return -3;
  const cudaError_t e = launch_pdl(moe_route_kernel, dim3((rows + ROUTE_WARPS - 1) / ROUTE_WARPS), dim3(ROUTE_WARPS * 32), smem,
                                   STREAM(stream), logits, splits, stride, ld, rows, E, n_groups, keep, top, renorm, sigmoid, ids, wts, ticket, counts);
  return e == cudaSuccess ? 0 : -21;
}

extern "C" int rpeg_moe_dispatch(const void* x, int dp, const int* ids, const int* ticket, const float* wts, const int* counts, int rows,
                                 int E, int top, void* xs, int* row_of, int* seg_off, int f32, void* stream) {
  if (rows <= 0) return 0;
  if ((dp & 7) || E < 1 || E > MOE_MAX_SEGMENTS || top < 1 || top > E) return -2;
  const size_t smem = static_cast<size_t>(E + 1 + top) * 4;
  const cudaError_t e =
      f32 ? launch_pdl(moe_dispatch_kernel<float>, dim3(rows), dim3(128), smem, STREAM(stream), static_cast<const float*>(x), dp, ids, ticket,
                       wts, counts, E, top, static_cast<float*>(xs), row_of, seg_off)
          : launch_pdl(moe_dispatch_kernel<__nv_bfloat16>, dim3(rows), dim3(128), smem, STREAM(stream), static_cast<const __nv_bfloat16*>(x),
                       dp, ids, ticket, wts, counts, E, top, static_cast<__nv_bfloat16*>(xs), row_of, seg_off);
  return e == cudaSuccess ? 0 : -21;
}

// A [a_rows_total, K]: routed rows (and the always-on ones unless X is given); X [seg_rows, K] or null; B [(n_routed +
// n_shared) * N, K] (2 N rows per segment for FF_SWIGLU); C rows as A's segments. `choices` = routed rows in total (seg_rows * top), for the grid size.
extern "C" int rpeg_moe_gemm(const void* A, long long a_rows_total, const void* X, const void* B, void* C, const int* seg_off, int n_routed,
                             int n_shared, int seg_rows, long long choices, int N, int K, int lda, int ldx, int ldb, int ldc, int act,
                             int bn_hint, int* status, void* stream) {
  if (seg_rows <= 0 || N <= 0 || K <= 0) return 0;
  const int S = n_routed + n_shared;
  if (S < 1 || S > MOE_MAX_SEGMENTS) return -3;
  if ((reinterpret_cast<uintptr_t>(A) | reinterpret_cast<uintptr_t>(B) | reinterpret_cast<uintptr_t>(C) | reinterpret_cast<uintptr_t>(X)) & 15)
    return -1;
  if ((lda | ldb | ldc | ldx | N) & 7) return -2;
  static int num_sms = 0;
  if (num_sms == 0) {
    int dev = 0;
    cudaGetDevice(&dev);
    cudaDeviceGetAttribute(&num_sms, cudaDevAttrMultiProcessorCount, dev);
  }
  // A routed segment has at most min(seg_rows, choices) rows; the number of M tiles is bounded by full tiles plus one
  // ragged tile per segment that can be non-empty.
  const long long active = choices < n_routed ? choices : n_routed;
  const long long m_tiles = choices / MG_BM + active + static_cast<long long>(n_shared) * ((seg_rows + MG_BM - 1) / MG_BM);
  int bn = bn_hint;
  if (bn == 0) {
    // widest tile that still gives every SM one, unless it wastes much more of the last column tile than a narrower one
    bn = 256;
    const int cols = act == FF_SWIGLU ? 2 * N : N;
    while (bn > 64 && (m_tiles * ((cols + bn - 1) / bn) < num_sms || (cols + bn - 1) / bn * bn * 8 > ((cols + 127) / 128 * 128) * 9)) bn >>= 1;
  }
  const int tn = act == FF_SWIGLU ? bn / 2 : bn;
  const int a_rows = seg_rows <= 32 ? 32 : (seg_rows <= 64 ? 64 : MG_BM);
  CUtensorMap ta, tx, tb;
  int rc = make_tmap_bf16_2d(&ta, A, K, a_rows_total, lda, MG_BK, a_rows);
  if (rc) return rc;
  rc = X != nullptr ? make_tmap_bf16_2d(&tx, X, K, seg_rows, ldx, MG_BK, a_rows) : make_tmap_bf16_2d(&tx, A, K, a_rows_total, lda, MG_BK, a_rows);
  if (rc) return rc - 100;
  rc = make_tmap_bf16_2d(&tb, B, K, static_cast<uint64_t>(S) * N * (act == FF_SWIGLU ? 2 : 1), ldb, MG_BK, tn);
  if (rc) return rc - 200;
  const long long max_tiles = m_tiles * ((N + tn - 1) / tn);
#define RPEG_MG_ACT(BN_, ACT_)                                                                                                       \
  return launch_moe_gemm<BN_, ACT_>(ta, tx, tb, C, seg_off, n_routed, n_shared, seg_rows, X != nullptr, N, K, ldc, a_rows, max_tiles, \
                                    num_sms, status, STREAM(stream));
#define RPEG_MG_CASE(BN_)                             \
  case BN_:                                           \
    switch (act) {                                    \
      case FF_NONE: RPEG_MG_ACT(BN_, FF_NONE)         \
      case FF_GELU: RPEG_MG_ACT(BN_, FF_GELU)         \
      case FF_SWIGLU: RPEG_MG_ACT(BN_, FF_SWIGLU)     \
      case FF_RELU2: RPEG_MG_ACT(BN_, FF_RELU2)       \
      default: return -4;                             \
    }
  switch (bn) {
    RPEG_MG_CASE(256)
    RPEG_MG_CASE(128)
    RPEG_MG_CASE(64)
    default:
      return -4;
  }
#undef RPEG_MG_ACT
#undef RPEG_MG_CASE
}
