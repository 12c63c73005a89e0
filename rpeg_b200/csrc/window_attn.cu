// Attention over the paged cache for layers whose visible keys are limited to the query's own chunk of the sequence,
// whose softmax has a sink, and whose head size is not fixed: chunk size (0 = none), sink (null = none), scale,
// rotary size and head size (up to 256) are arguments.
//
// Cache layout per layer: K pages and V pages [num_pages, H_kv, PAGE, dp], dp = head size padded to a multiple of 8
// (padding is zero), so one (page, head) block is contiguous and is fetched with one bulk copy.
//
//   rotary_append   interleaved rotary embedding on the first dimensions, optional weight-free RMS norm per head after
//                   it, q to a buffer, k (rotated, normalised) and v (as projected) to the cache. v may be the keys'
//                   own projection (`v_col0 == k_col0`).
//   rows_attn       one query row per (CTA, group of up to 8 query heads of one KV head): decode, and any prompt the
//                   tensor-core kernel below does not take. Pages stream through shared memory (bulk copies, mbarrier
//                   ring), each K / V element is read once for all heads of the group, split over the pages.
// The tensor-core kernel for prompts is in window_prefill.cu.
#include "act_io.cuh"
#include "rpeg_kernels.h"

namespace rpeg {

constexpr int WPAGE = RPEG_KV_PAGE;

// One warp per HPW heads of a token (query heads, then KV heads). A lane owns runs of 4 elements, i.e. whole pairs
// (2i, 2i + 1), so the rotation is local; a rotation keeps the sum of squares, so the norm is known before it. Prompts take
// four heads per warp (the angles are read once for all of them), decode one (more warps for few tokens).
template <typename T, bool PARTIALS, int HPW>
__global__ void __launch_bounds__(256)
rotary_append_kernel(const void* __restrict__ src_v, int splits, long long stride, int ld, int q_col0, int k_col0, int v_col0,
                     const int* __restrict__ slot, const int* __restrict__ pos, const float* __restrict__ cos_t,
                     const float* __restrict__ sin_t, const int* __restrict__ page_table, int max_pages, T* __restrict__ q_out, int ldq,
                     T* __restrict__ kcache, T* __restrict__ vcache, int rows, int H, int Hkv, int dim, int dp, int rot_dims, int do_norm,
                     float eps) {
  griddep_launch();
  griddep_wait();
  const unsigned jobs = (H + Hkv + HPW - 1) / HPW;
  const unsigned wid = blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);     // below 2^31, checked on the host
  if (wid >= static_cast<unsigned>(rows) * jobs) return;
  const int lane = threadIdx.x & 31;
  const int t = static_cast<int>(wid / jobs), job0 = static_cast<int>(wid % jobs) * HPW;
  const int p = pos[t];
  const int half = rot_dims >> 1, nq = dp >> 2;
  auto read = [&](int col) -> float4 {
    const size_t off = static_cast<size_t>(t) * ld + col;
    if constexpr (PARTIALS) {
      const float* s = static_cast<const float*>(src_v) + off;
      float4 a = load4(s);
#pragma unroll 8
      for (int k = 1; k < splits; ++k) a = add4(a, load4(s + k * stride));
      return a;
    } else {
      return load4(static_cast<const T*>(src_v) + off);
    }
  };
  float4 v[HPW][2];
#pragma unroll
  for (int g = 0; g < HPW; ++g) {
    const int job = job0 + g;
    const int col0 = job < H ? q_col0 + job * dp : k_col0 + (job - H) * dp;
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      v[g][j] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (lane + 32 * j < nq && job < H + Hkv) v[g][j] = read(col0 + 4 * (lane + 32 * j));
    }
  }
  float2 cs[2][2];                                          // (cos, sin) of the lane's two pairs
#pragma unroll
  for (int j = 0; j < 2; ++j)
#pragma unroll
    for (int e = 0; e < 2; ++e) {
      const int pr = 2 * (lane + 32 * j) + e;
      cs[j][e] = pr < half ? make_float2(cos_t[static_cast<size_t>(p) * half + pr], sin_t[static_cast<size_t>(p) * half + pr])
                           : make_float2(1.f, 0.f);
    }
  size_t page_row = 0;
  if (job0 + HPW > H) page_row = static_cast<size_t>(page_table[static_cast<size_t>(slot[t]) * max_pages + p / WPAGE]) * Hkv;
#pragma unroll
  for (int g = 0; g < HPW; ++g) {
    const int job = job0 + g;
    if (job >= H + Hkv) break;
    const bool is_q = job < H;
    float r = 1.f;
    if (do_norm) {
      float ss = 0.f;
#pragma unroll
      for (int j = 0; j < 2; ++j) ss += v[g][j].x * v[g][j].x + v[g][j].y * v[g][j].y + v[g][j].z * v[g][j].z + v[g][j].w * v[g][j].w;
      r = rsqrtf(warp_sum(ss) / static_cast<float>(dim) + eps);
    }
    const size_t dst = is_q ? 0 : ((page_row + (job - H)) * WPAGE + (p % WPAGE)) * dp;
    T* out = is_q ? q_out + static_cast<size_t>(t) * ldq + job * dp : kcache + dst;
#pragma unroll
    for (int j = 0; j < 2; ++j) {
      const int i = lane + 32 * j;
      if (i >= nq) break;
      const float4 u = v[g][j];
      if (!is_q) store4(vcache + dst + 4 * i, v_col0 == k_col0 ? u : read(v_col0 + (job - H) * dp + 4 * i));
      const float2 a = cs[j][0], b = cs[j][1];
      store4(out + 4 * i, make_float4((u.x * a.x - u.y * a.y) * r, (u.y * a.x + u.x * a.y) * r, (u.z * b.x - u.w * b.y) * r,
                                      (u.w * b.x + u.z * b.y) * r));
    }
  }
}

// ---------------------------------------------------------------------------------- rows attention
constexpr int RA_THREADS = 128;
constexpr size_t RA_SMEM_TARGET = 72 * 1024;     // pages in flight per CTA: three CTAs of one SM together keep the copy rate up

struct RowsAttn {
  const void* q; int ldq;
  const void* kc; const void* vc;
  const int* page_table; int max_pages;
  const int* slot; const int* pos; const int* lens;              // lens null: pos + 1 keys
  const void* sink;
  void* out; int ldo;
  float* partial; int* arrive;                                   // split results [row, head, split, dp + 2]
  int H, Hkv, dp, window, nsplit, stages;
  float scale_log2;
  int* status;
};

__device__ __forceinline__ void load8(const __nv_bfloat16* p, uint64_t (&o)[4]) {
  const uint4 v = *reinterpret_cast<const uint4*>(p);
  const uint32_t w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const float2 f = unpack_bf16x2(w[i]);
    o[i] = pack2(f.x, f.y);
  }
}
__device__ __forceinline__ void load8(const float* p, uint64_t (&o)[4]) {
  const float4 a = load4(p), b = load4(p + 4);
  o[0] = pack2(a.x, a.y); o[1] = pack2(a.z, a.w); o[2] = pack2(b.x, b.y); o[3] = pack2(b.z, b.w);
}
__device__ __forceinline__ void bulk_load(void* smem_dst, const void* src, uint32_t bytes, uint64_t* bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(smem_u32(smem_dst)),
               "l"(reinterpret_cast<uint64_t>(src)), "r"(bytes), "r"(smem_u32(bar))
               : "memory");
}

// LPK lanes hold one key (8 dimensions each), a warp scores 32 / LPK keys side by side and RA_KEYS of them per lane
// group in a row, for RA_HEADS query heads of the KV head (4 or 8, whichever leaves fewer idle). The RA_KEYS x RA_HEADS
// partial dot products of a lane are summed across its group by a transposing
// butterfly after which lane c holds the finished scores number c * VPL .. of the list (key major), so every exponential
// is computed once; the weights go back to all lanes of the group by shuffles for P V.
template <typename T, int LPK, int RA_HEADS, int RA_KEYS>
__global__ void __launch_bounds__(RA_THREADS)
rows_attn_kernel(const RowsAttn a) {
  constexpr int GPW = 32 / LPK, NV = RA_KEYS * RA_HEADS, VPL = NV / LPK, ITERS = (WPAGE / 4) / (RA_KEYS * GPW);
  constexpr int GROUPS = 4 * GPW, WIDTH = LPK * 8;
  constexpr int HL = RA_HEADS / VPL;                    // lanes that hold the scores of one key
  static_assert(VPL >= 1 && HL >= 1 && ITERS >= 1, "lane split");
  griddep_launch();
  griddep_wait();
  extern __shared__ __align__(128) uint8_t ra_smem[];
  __shared__ uint64_t full_bar[4];
  __shared__ int abort_word, is_last;
  __shared__ float share[RA_HEADS][64];
  __shared__ float red_m[GROUPS][RA_HEADS], red_l[GROUPS][RA_HEADS];
  const int row = blockIdx.x, split = blockIdx.z;
  const int R = a.H / a.Hkv;                            // query heads per KV head
  const int blocks_per_kv = (R + RA_HEADS - 1) / RA_HEADS;
  const int hk = blockIdx.y / blocks_per_kv;
  const int r0 = (blockIdx.y % blocks_per_kv) * RA_HEADS;
  const int nh = min(RA_HEADS, R - r0), h0 = hk * R + r0;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int grp = lane / LPK, c = lane % LPK;
  const int dp = a.dp;
  const bool has_dims = c * 8 < dp;
  const int L = a.lens != nullptr ? a.lens[row] : a.pos[row] + 1;
  const int key0 = a.window > 0 && L > 0 ? (L - 1) / a.window * a.window : 0;
  const int pg0 = key0 / WPAGE, pg1 = L > 0 ? (L + WPAGE - 1) / WPAGE : pg0;
  const int per = (pg1 - pg0 + a.nsplit - 1) / a.nsplit;
  const int pa = min(pg1, pg0 + split * per), pb = min(pg1, pa + per);
  const uint32_t block_bytes = static_cast<uint32_t>(WPAGE * dp * sizeof(T));
  const int stages = a.stages;
  const int* pt = a.page_table + static_cast<size_t>(a.slot[row]) * a.max_pages;
  const T* kc = static_cast<const T*>(a.kc);
  const T* vc = static_cast<const T*>(a.vc);
  auto fetch = [&](int pg, int st) {
    const size_t off = (static_cast<size_t>(pt[pg]) * a.Hkv + hk) * WPAGE * dp;
    uint8_t* dst = ra_smem + static_cast<size_t>(st) * 2 * block_bytes;
    mbar_expect_tx(&full_bar[st], 2 * block_bytes);
    bulk_load(dst, kc + off, block_bytes, &full_bar[st]);
    bulk_load(dst + block_bytes, vc + off, block_bytes, &full_bar[st]);
  };
  if (threadIdx.x == 0) {
    for (int s = 0; s < stages; ++s) mbar_init(&full_bar[s], 1);
    abort_word = 0;
    fence_mbar_init();
    for (int i = 0; i < stages && pa + i < pb; ++i) fetch(pa + i, i);
  }
  uint64_t q2[RA_HEADS][4];
#pragma unroll
  for (int h = 0; h < RA_HEADS; ++h) {
#pragma unroll
    for (int k = 0; k < 4; ++k) q2[h][k] = 0ull;
    if (h < nh && has_dims) {
      load8(static_cast<const T*>(a.q) + static_cast<size_t>(row) * a.ldq + (h0 + h) * dp + c * 8, q2[h]);
      const uint64_t sc = pack2(a.scale_log2, a.scale_log2);
#pragma unroll
      for (int k = 0; k < 4; ++k) q2[h][k] = mul2(q2[h][k], sc);
    }
  }
  uint64_t acc[RA_HEADS][4];
#pragma unroll
  for (int h = 0; h < RA_HEADS; ++h)
#pragma unroll
    for (int k = 0; k < 4; ++k) acc[h][k] = 0ull;
  float m[VPL], l[VPL];
#pragma unroll
  for (int i = 0; i < VPL; ++i) { m[i] = -INFINITY; l[i] = 0.f; }
  const int u_own = c * VPL / RA_HEADS;                 // which of the RA_KEYS keys this lane's finished scores belong to
  const int gbase = grp * LPK;
  __syncthreads();

  for (int pg = pa; pg < pb; ++pg) {
    const int st = (pg - pa) % stages;
    const bool ok = mbar_wait(&full_bar[st], static_cast<uint32_t>((pg - pa) / stages) & 1u, &abort_word, a.status, 800);
    if (ok) {
      const T* ks = reinterpret_cast<const T*>(ra_smem + static_cast<size_t>(st) * 2 * block_bytes);
      const T* vs = ks + static_cast<size_t>(WPAGE) * dp;
#pragma unroll 1
      for (int it = 0; it < ITERS; ++it) {
        const int kbase = warp * (WPAGE / 4) + it * RA_KEYS * GPW + grp;          // key u of this group: kbase + u * GPW
        const int j0 = pg * WPAGE + kbase;
        // keys of a warp's iteration lie in one run of RA_KEYS * GPW positions
        const int run0 = pg * WPAGE + warp * (WPAGE / 4) + it * RA_KEYS * GPW;
        if (run0 >= L || run0 + RA_KEYS * GPW <= key0) continue;                  // uniform over the warp
        float v[NV];
#pragma unroll
        for (int u = 0; u < RA_KEYS; ++u) {
          uint64_t k2[4] = {0ull, 0ull, 0ull, 0ull};
          if (has_dims) load8(ks + (kbase + u * GPW) * dp + c * 8, k2);
#pragma unroll
          for (int h = 0; h < RA_HEADS; ++h) {
            uint64_t d = mul2(q2[h][0], k2[0]);
            d = fma2(q2[h][1], k2[1], d);
            d = fma2(q2[h][2], k2[2], d);
            d = fma2(q2[h][3], k2[3], d);
            const float2 f = unpack2(d);
            v[u * RA_HEADS + h] = f.x + f.y;
          }
        }
        int n = NV;
#pragma unroll
        for (int mask = LPK / 2; mask >= 1; mask >>= 1) {
          n >>= 1;
          const bool up = lane & mask;
#pragma unroll
          for (int i = 0; i < NV / 2; ++i) {
            if (i < n) {
              const float send = up ? v[i] : v[i + n];
              const float keep = up ? v[i + n] : v[i];
              v[i] = keep + __shfl_xor_sync(0xffffffffu, send, mask);
            }
          }
        }
        const int j = j0 + u_own * GPW;
        const bool valid = j >= key0 && j < L;
        bool grew = false;
        float nm[VPL];
#pragma unroll
        for (int i = 0; i < VPL; ++i) {
          if (!valid) v[i] = -INFINITY;
          float b = v[i];
#pragma unroll
          for (int o = HL; o < LPK; o <<= 1) b = fmaxf(b, __shfl_xor_sync(0xffffffffu, b, o));
          nm[i] = fmaxf(m[i], b);
          grew |= nm[i] > m[i];
        }
        if (__any_sync(0xffffffffu, grew)) {
          float al[VPL];
#pragma unroll
          for (int i = 0; i < VPL; ++i) {
            al[i] = nm[i] == -INFINITY ? 1.f : exp2f(m[i] - nm[i]);
            l[i] *= al[i];
            m[i] = nm[i];
          }
#pragma unroll
          for (int h = 0; h < RA_HEADS; ++h) {
            const float s = __shfl_sync(0xffffffffu, al[h % VPL], gbase + h / VPL);
            const uint64_t s2 = pack2(s, s);
#pragma unroll
            for (int k = 0; k < 4; ++k) acc[h][k] = mul2(acc[h][k], s2);
          }
        }
#pragma unroll
        for (int i = 0; i < VPL; ++i) {
          v[i] = valid ? exp2f(v[i] - m[i]) : 0.f;
          l[i] += v[i];
        }
#pragma unroll
        for (int u = 0; u < RA_KEYS; ++u) {
          uint64_t v2[4] = {0ull, 0ull, 0ull, 0ull};
          const int ju = j0 + u * GPW;
          if (has_dims && ju >= key0 && ju < L) load8(vs + (kbase + u * GPW) * dp + c * 8, v2);
#pragma unroll
          for (int h = 0; h < RA_HEADS; ++h) {
            const float ph = __shfl_sync(0xffffffffu, v[h % VPL], gbase + (u * RA_HEADS + h) / VPL);
            const uint64_t p2 = pack2(ph, ph);
#pragma unroll
            for (int k = 0; k < 4; ++k) acc[h][k] = fma2(p2, v2[k], acc[h][k]);
          }
        }
      }
    }
    if (!__syncthreads_and(ok ? 1 : 0)) break;
    if (threadIdx.x == 0 && pg + stages < pb) fetch(pg + stages, st);
  }
  // After a wait that ran out, copies may still be in flight into this CTA's shared memory: let them land.
  if (abort_word) __nanosleep(200000);
  __syncthreads();

  // merge the lane groups: every group leaves (m, l, o) of its share of the keys
  float* red_o = reinterpret_cast<float*>(ra_smem);     // [GROUPS][RA_HEADS][WIDTH]
  const int gi = warp * GPW + grp;
#pragma unroll
  for (int i = 0; i < VPL; ++i) {
#pragma unroll
    for (int o = HL; o < LPK; o <<= 1) l[i] += __shfl_xor_sync(0xffffffffu, l[i], o);
    if (u_own == 0) {
      red_m[gi][c * VPL + i] = m[i];
      red_l[gi][c * VPL + i] = l[i];
    }
  }
#pragma unroll
  for (int h = 0; h < RA_HEADS; ++h)
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      const float2 f = unpack2(acc[h][k]);
      *reinterpret_cast<float2*>(red_o + (static_cast<size_t>(gi) * RA_HEADS + h) * WIDTH + c * 8 + 2 * k) = f;
    }
  __syncthreads();
  const float* sink = static_cast<const float*>(a.sink);
  T* out = static_cast<T*>(a.out) + static_cast<size_t>(row) * a.ldo;
  for (int e = threadIdx.x; e < nh * dp; e += RA_THREADS) {
    const int h = e / dp, d = e % dp;
    float gm = -INFINITY;
#pragma unroll
    for (int g = 0; g < GROUPS; ++g) gm = fmaxf(gm, red_m[g][h]);
    float gl = 0.f, o = 0.f;
#pragma unroll
    for (int g = 0; g < GROUPS; ++g) {
      const float w = red_m[g][h] == -INFINITY ? 0.f : exp2f(red_m[g][h] - gm);
      gl += red_l[g][h] * w;
      o += red_o[(static_cast<size_t>(g) * RA_HEADS + h) * WIDTH + d] * w;
    }
    if (a.nsplit == 1) {
      if (sink != nullptr) {
        const float sl = sink[h0 + h] * 1.4426950408889634f, nm = fmaxf(gm, sl);
        const float w = gm == -INFINITY ? 0.f : exp2f(gm - nm);
        o *= w;
        gl = gl * w + exp2f(sl - nm);
      }
      const float r = gl > 0.f ? o / gl : 0.f;
      if constexpr (sizeof(T) == 2) out[(h0 + h) * dp + d] = __float2bfloat16(r); else out[(h0 + h) * dp + d] = r;
    } else {
      float* pp = a.partial + ((static_cast<size_t>(row) * a.H + h0 + h) * a.nsplit + split) * (dp + 2);
      pp[d] = o;
      if (d == 0) { pp[dp] = gm; pp[dp + 1] = gl; }
    }
  }
  if (a.nsplit == 1) return;
  // The last split of a (row, head group) to arrive merges all of them and resets the counter for the next launch.
  int* counter = a.arrive + static_cast<size_t>(row) * gridDim.y + blockIdx.y;
  __threadfence();
  __syncthreads();
  if (threadIdx.x == 0) is_last = atomicAdd(counter, 1) == a.nsplit - 1 ? 1 : 0;
  __syncthreads();
  if (!is_last) return;
  if (threadIdx.x == 0) *counter = 0;
  __threadfence();
  const float* parts = a.partial + (static_cast<size_t>(row) * a.H + h0) * a.nsplit * (dp + 2);
  if (warp < nh)                                        // share of every split in its head's result
    for (int h = warp; h < nh; h += RA_THREADS / 32) {
      const float* pp = parts + static_cast<size_t>(h) * a.nsplit * (dp + 2) + dp;
      const float sl = sink != nullptr ? sink[h0 + h] * 1.4426950408889634f : -INFINITY;
      float ms[2], ls[2], gm = sl;
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        const int s = lane + 32 * j;
        ms[j] = s < a.nsplit ? __ldcg(pp + s * (dp + 2)) : -INFINITY;
        ls[j] = s < a.nsplit ? __ldcg(pp + s * (dp + 2) + 1) : 0.f;
        gm = fmaxf(gm, ms[j]);
      }
      gm = warp_max(gm);
      float gl = 0.f;
#pragma unroll
      for (int j = 0; j < 2; ++j) {
        ms[j] = ms[j] == -INFINITY ? 0.f : exp2f(ms[j] - gm);
        gl += ls[j] * ms[j];
      }
      gl = warp_sum(gl) + (sink != nullptr ? exp2f(sl - gm) : 0.f);
#pragma unroll
      for (int j = 0; j < 2; ++j)
        if (lane + 32 * j < a.nsplit) share[h][lane + 32 * j] = gl > 0.f ? ms[j] / gl : 0.f;
    }
  __syncthreads();
  for (int e = threadIdx.x; e < nh * dp; e += RA_THREADS) {
    const int h = e / dp, d = e % dp;
    const float* pp = parts + static_cast<size_t>(h) * a.nsplit * (dp + 2) + d;
    float r = 0.f;
#pragma unroll 8
    for (int s = 0; s < a.nsplit; ++s) r += __ldcg(pp + s * (dp + 2)) * share[h][s];
    if constexpr (sizeof(T) == 2) out[(h0 + h) * dp + d] = __float2bfloat16(r); else out[(h0 + h) * dp + d] = r;
  }
}

template <typename T, int LPK, int HEADS, int KEYS>
static int launch_rows_attn(RowsAttn a, int rows, cudaStream_t stream) {
  auto kern = rows_attn_kernel<T, LPK, HEADS, KEYS>;
  const size_t stage = static_cast<size_t>(2) * WPAGE * a.dp * sizeof(T);
  const size_t merge = static_cast<size_t>(4 * (32 / LPK)) * HEADS * LPK * 8 * 4;
  int st = static_cast<int>((RA_SMEM_TARGET) / stage);
  a.stages = st < 1 ? 1 : (st > 4 ? 4 : st);
  size_t smem = a.stages * stage;
  if (smem < merge) smem = merge;
  if (smem > 224 * 1024) return -3;
  static size_t configured = 0;
  if (smem > configured) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)) != cudaSuccess) return -20;
    configured = smem;
  }
  const int R = a.H / a.Hkv;
  const dim3 grid(rows, a.Hkv * ((R + HEADS - 1) / HEADS), a.nsplit);
  return launch_pdl(kern, grid, dim3(RA_THREADS), smem, stream, a) == cudaSuccess ? 0 : -21;
}

template <typename T>
static int dispatch_rows_attn(const RowsAttn& a, int rows, cudaStream_t stream) {
  const int R = a.H / a.Hkv;
  const bool narrow = (R - 1) % 8 < 4 && R <= 12;            // blocks of 4 heads leave fewer idle
  if (narrow) {
    if (a.dp <= 64) return launch_rows_attn<T, 8, 4, 4>(a, rows, stream);
    if (a.dp <= 128) return launch_rows_attn<T, 16, 4, 8>(a, rows, stream);
    return launch_rows_attn<T, 32, 4, 8>(a, rows, stream);
  }
  if (a.dp <= 64) return launch_rows_attn<T, 8, 8, 4>(a, rows, stream);
  if (a.dp <= 128) return launch_rows_attn<T, 16, 8, 4>(a, rows, stream);
  return launch_rows_attn<T, 32, 8, 4>(a, rows, stream);
}

}  // namespace rpeg

using namespace rpeg;
#define STREAM(s) reinterpret_cast<cudaStream_t>(s)

extern "C" int rpeg_rotary_append(const void* src, int splits, long long stride, int ld, int q_col0, int k_col0, int v_col0, const int* slot,
                                  const int* pos, const float* cos_t, const float* sin_t, const int* page_table, int max_pages, void* q_out,
                                  int ldq, void* kcache, void* vcache, int rows, int H, int Hkv, int dim, int dp, int rot_dims, int do_norm,
                                  float eps, int f32, void* stream) {
  if (rows <= 0) return 0;
  if ((dp & 7) || dp > 256 || dim < 1 || dim > dp || rot_dims < 0 || rot_dims > dim || (rot_dims & 1) || ((ld | ldq | q_col0 | k_col0 | v_col0) & 3)) return -2;
  if (H < 1 || Hkv < 1 || H % Hkv) return -3;
  const int hpw = rows >= 1024 && !f32 && splits == 0 ? 4 : 1;
  const long long warps = static_cast<long long>(rows) * ((H + Hkv + hpw - 1) / hpw);
  if (warps > 0x7fffffffll) return -2;
  const dim3 grid(static_cast<unsigned>((warps + 7) / 8));
#define RPEG_RA(T_, P_, H_)                                                                                                           \
  return launch_pdl(rotary_append_kernel<T_, P_, H_>, grid, dim3(256), 0, STREAM(stream), src, splits, stride, ld, q_col0, k_col0, v_col0, \
                    slot, pos, cos_t, sin_t, page_table, max_pages, static_cast<T_*>(q_out), ldq, static_cast<T_*>(kcache),            \
                    static_cast<T_*>(vcache), rows, H, Hkv, dim, dp, rot_dims, do_norm, eps) == cudaSuccess ? 0 : -21;
  if (f32) { RPEG_RA(float, false, 1) }
  if (splits > 0) { RPEG_RA(__nv_bfloat16, true, 1) }
  if (hpw == 4) { RPEG_RA(__nv_bfloat16, false, 4) }
  RPEG_RA(__nv_bfloat16, false, 1)
#undef RPEG_RA
}

// floats of scratch for `rows` rows split `nsplit` ways (plus, in ints, rows * H arrival counters that start at zero)
extern "C" long long rpeg_rows_attn_scratch(int rows, int H, int dp, int nsplit) {
  return nsplit > 1 ? static_cast<long long>(rows) * H * nsplit * (dp + 2) : 0;
}

extern "C" int rpeg_rows_attn(const void* q, int ldq, const void* kcache, const void* vcache, const int* page_table, int max_pages,
                              const int* slot, const int* pos, const int* lens, const float* sink, void* out, int ldo, float* scratch,
                              int* arrive, int rows, int H, int Hkv, int dp, int window, int nsplit, float scale, int f32, int* status,
                              void* stream) {
  if (rows <= 0) return 0;
  if ((dp & 7) || dp < 8 || dp > 256 || H < 1 || Hkv < 1 || H % Hkv || window < 0 || nsplit < 1 || nsplit > 64) return -2;
  if (nsplit > 1 && (scratch == nullptr || arrive == nullptr)) return -6;
  if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(kcache) | reinterpret_cast<uintptr_t>(vcache)) & 15) return -1;
  if (ldq & 7) return -2;
  RowsAttn a{q, ldq, kcache, vcache, page_table, max_pages, slot, pos, lens, sink, out, ldo, scratch, arrive,
             H, Hkv, dp, window, nsplit, 1, scale * 1.4426950408889634f, status};
  return f32 ? dispatch_rows_attn<float>(a, rows, STREAM(stream)) : dispatch_rows_attn<__nv_bfloat16>(a, rows, STREAM(stream));
}
