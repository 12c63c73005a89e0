// Prompt attention on the tensor cores, keys and values read from the paged cache, head size up to 128 (bf16).
//
//   O = softmax(Q K^T * scale  [visible keys], sink) V
//
// Row i of a request's portion stands at position p = (cached tokens) + i and sees the keys [floor(p / window) * window, p]
// (window = 0: [0, p]). The portion's own keys were appended to the cache before, so a whole prompt, a portion of one
// and a batch of unequal portions are the same launch: nothing depends on where a prompt was cut.
//
// One CTA = 128 query rows of one head; the pipeline is the one of flash_attn.cu (TMA warp, MMA warp, four softmax
// warps; S double buffered in TMEM, P in TMEM columns of its own, lazy rescaling of O). Differences:
//   * a key tile is two 64-token cache pages, fetched by TMA through the request's page-table row; tiles start at the
//     page that holds the first key any row of the CTA sees;
//   * heads narrower than the tile (64 or 128) are padded by the TMA unit (out-of-bounds columns read as zero);
//   * the sink opens the softmax: the running maximum starts no lower than the sink's logit and the running sum with its
//     exponential, so it needs no key and no pass of its own.
#include "common.cuh"
#include "rpeg_kernels.h"

namespace rpeg {

constexpr int WP_BM = 128, WP_BN = 128, WP_THREADS = 192, WP_STAGES = 2;
constexpr float WP_RESCALE = 8.0f;

template <int HDT>
struct PrefillCfg {
  static constexpr int TILE = 128 * HDT * 2;               // HDT / 64 atoms of 128 rows x 128 bytes
  static constexpr int SMEM = TILE * (1 + 2 * WP_STAGES) + 1024 + 256;
};

struct Prefill {
  const int* cu; const int* pos; const int* slot;
  const int* page_table; int max_pages;
  const float* sink;
  __nv_bfloat16* out; int ldo;
  int H, Hkv, dp, window;
  float scale_log2;
  int* status;
};

// Largest raw score of the row among the visible keys [lo, hi] of the tile that starts at k0.
template <bool MASK>
__device__ __forceinline__ float wp_max_pass(uint32_t ts, int k0, int lo, int hi) {
  uint32_t a[32], b[32];
  float tmax = -INFINITY;
  tmem_ld_32x32(ts, a);
#pragma unroll
  for (int c = 0; c < 4; ++c) {
    tmem_wait_ld();
    uint32_t(&cur)[32] = (c & 1) ? b : a;
    if (c + 1 < 4) tmem_ld_32x32(ts + (c + 1) * 32, (c & 1) ? a : b);
#pragma unroll
    for (int i = 0; i < 32; ++i) {
      const int kj = k0 + c * 32 + i;
      if (!MASK || (kj >= lo && kj <= hi)) tmax = fmaxf(tmax, __uint_as_float(cur[i]));
    }
  }
  return tmax;
}

// P = exp2(s * scale - m_ref) as packed bf16, its row sum, and the largest raw score seen.
template <bool MASK>
__device__ __forceinline__ void wp_exp_pass(uint32_t ts, uint32_t tp, float scale_log2, float m_ref, int k0, int lo, int hi, float& lsum,
                                            float& smax) {
  uint32_t a[32], b[32];
  tmem_ld_32x32(ts, a);
#pragma unroll
  for (int c = 0; c < 4; ++c) {
    tmem_wait_ld();
    uint32_t(&cur)[32] = (c & 1) ? b : a;
    if (c + 1 < 4) tmem_ld_32x32(ts + (c + 1) * 32, (c & 1) ? a : b);
    uint32_t pk[16];
#pragma unroll
    for (int i = 0; i < 16; ++i) {
      const int kj = k0 + c * 32 + 2 * i;
      const float s0 = __uint_as_float(cur[2 * i]), s1 = __uint_as_float(cur[2 * i + 1]);
      float p0, p1;
      if (MASK) {
        const bool v0 = kj >= lo && kj <= hi, v1 = kj + 1 >= lo && kj + 1 <= hi;
        if (v0) smax = fmaxf(smax, s0);
        if (v1) smax = fmaxf(smax, s1);
        p0 = v0 ? exp2f(fmaf(s0, scale_log2, -m_ref)) : 0.f;
        p1 = v1 ? exp2f(fmaf(s1, scale_log2, -m_ref)) : 0.f;
      } else {
        smax = fmaxf(smax, fmaxf(s0, s1));
        p0 = exp2f(fmaf(s0, scale_log2, -m_ref));
        p1 = exp2f(fmaf(s1, scale_log2, -m_ref));
      }
      lsum += p0 + p1;
      pk[i] = pack_bf16x2(p0, p1);
    }
    tmem_st_32x16(tp + c * 16, pk);
  }
}

template <int HDT>
__global__ void __launch_bounds__(WP_THREADS, 1)
window_prefill_kernel(const __grid_constant__ CUtensorMap tmap_q, const __grid_constant__ CUtensorMap tmap_k,
                      const __grid_constant__ CUtensorMap tmap_v, const Prefill a) {
  using Cfg = PrefillCfg<HDT>;
  constexpr int ATOMS = HDT / 64, TILE = Cfg::TILE;
  const int b = blockIdx.z, h = blockIdx.y;
  const int qt = gridDim.x - 1 - blockIdx.x;
  const int tok0 = a.cu[b], L = a.cu[b + 1] - tok0;
  const int q0 = qt * WP_BM;
  if (q0 >= L) return;
  const int hk = h / (a.H / a.Hkv);
  const int p0 = a.pos[tok0] + q0;                          // position of the CTA's first row
  const int p_last = p0 + min(WP_BM, L - q0) - 1;
  const int first_key = a.window > 0 ? p0 / a.window * a.window : 0;
  const int last_lo = a.window > 0 ? p_last / a.window * a.window : 0;
  const int kb = first_key & ~(RPEG_KV_PAGE - 1);
  const int n_tiles = (p_last + 1 - kb + WP_BN - 1) / WP_BN;

  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* q_sm = smem;
  uint8_t* k_sm = smem + TILE;
  uint8_t* v_sm = k_sm + WP_STAGES * TILE;
  uint64_t* bars = reinterpret_cast<uint64_t*>(v_sm + WP_STAGES * TILE);
  uint64_t* q_full = bars;
  uint64_t* k_full = bars + 1;
  uint64_t* k_empty = k_full + WP_STAGES;
  uint64_t* v_full = k_empty + WP_STAGES;
  uint64_t* v_empty = v_full + WP_STAGES;
  uint64_t* s_full = v_empty + WP_STAGES;   // [2]
  uint64_t* p_full = s_full + 2;            // [2]
  uint64_t* pv_done = p_full + 2;           // [2]: PV_j completes pv_done[j & 1]
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(pv_done + 2);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int s = 0; s < WP_STAGES; ++s) {
      mbar_init(&k_full[s], 1); mbar_init(&k_empty[s], 1);
      mbar_init(&v_full[s], 1); mbar_init(&v_empty[s], 1);
    }
    for (int s = 0; s < 2; ++s) { mbar_init(&s_full[s], 1); mbar_init(&p_full[s], 4); mbar_init(&pv_done[s], 1); }
    *abort_flag = 0;
    fence_mbar_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, 512);
    tmem_relinquish();
  }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem_base = *tmem_slot;
  const uint32_t tmem_o = tmem_base + 256;

  if (warp == 0) {
    if (lane == 0) {
      const int* pt = a.page_table + static_cast<size_t>(a.slot[tok0]) * a.max_pages;
      auto load_tile = [&](const CUtensorMap* map, uint8_t* dst, uint64_t* bar, int j) {
        mbar_expect_tx(bar, TILE);
#pragma unroll
        for (int hf = 0; hf < 2; ++hf) {
          const int pi = kb / RPEG_KV_PAGE + 2 * j + hf;
          // a page past the row's last one is never visible: any valid page will do
          const int page = pi * RPEG_KV_PAGE <= p_last ? pt[pi] : 0;
          const int y = (page * a.Hkv + hk) * RPEG_KV_PAGE;
#pragma unroll
          for (int c = 0; c < ATOMS; ++c) tma_load_2d(dst + c * 16384 + hf * 8192, map, bar, c * 64, y);
        }
      };
      mbar_expect_tx(q_full, TILE);
#pragma unroll
      for (int c = 0; c < ATOMS; ++c) tma_load_3d(q_sm + c * 16384, &tmap_q, q_full, c * 64, h, tok0 + q0);
      for (int j = 0; j < n_tiles; ++j) {
        const int st = j % WP_STAGES;
        const uint32_t ph = static_cast<uint32_t>(j / WP_STAGES) & 1u;
        if (!mbar_wait(&k_empty[st], ph ^ 1u, abort_flag, a.status, 900)) break;
        load_tile(&tmap_k, k_sm + st * TILE, &k_full[st], j);
        if (!mbar_wait(&v_empty[st], ph ^ 1u, abort_flag, a.status, 901)) break;
        load_tile(&tmap_v, v_sm + st * TILE, &v_full[st], j);
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t idesc_qk = make_idesc_bf16(128, 128, 0, 0);
      constexpr uint32_t idesc_pv = make_idesc_bf16(128, HDT, 0, 1);
      const uint32_t q_addr = smem_u32(q_sm);
      auto issue_qk = [&](int j) {
        const int st = j % WP_STAGES;
        const uint32_t k_addr = smem_u32(k_sm + st * TILE);
        const uint32_t ts = tmem_base + static_cast<uint32_t>((j & 1) * 128);
#pragma unroll
        for (int k = 0; k < HDT / 16; ++k) {
          const uint32_t off = static_cast<uint32_t>((k >> 2) * 16384 + (k & 3) * 32);
          umma_bf16_ss(ts, make_smem_desc_sw128(q_addr + off, 16, 1024), make_smem_desc_sw128(k_addr + off, 16, 1024), idesc_qk,
                       k != 0 ? 1u : 0u);
        }
        umma_commit(&k_empty[st]);
        umma_commit(&s_full[j & 1]);
      };
      bool ok = mbar_wait(q_full, 0, abort_flag, a.status, 910);
      if (ok) ok = mbar_wait(&k_full[0], 0, abort_flag, a.status, 911);
      if (ok) {
        tc_fence_after_sync();
        issue_qk(0);
        for (int j = 0; j < n_tiles; ++j) {
          const int st = j % WP_STAGES;
          const uint32_t ph = static_cast<uint32_t>(j / WP_STAGES) & 1u;
          if (j + 1 < n_tiles) {
            const int st1 = (j + 1) % WP_STAGES;
            const uint32_t ph1 = static_cast<uint32_t>((j + 1) / WP_STAGES) & 1u;
            if (!mbar_wait(&k_full[st1], ph1, abort_flag, a.status, 912)) break;
            tc_fence_after_sync();
            issue_qk(j + 1);
          }
          if (!mbar_wait(&p_full[j & 1], static_cast<uint32_t>(j >> 1) & 1u, abort_flag, a.status, 913)) break;
          if (!mbar_wait(&v_full[st], ph, abort_flag, a.status, 914)) break;
          tc_fence_after_sync();
          const uint32_t v_addr = smem_u32(v_sm + st * TILE);
          const uint32_t tp = tmem_base + 384u + static_cast<uint32_t>((j & 1) * 64);
#pragma unroll
          for (int k = 0; k < 8; ++k)
            umma_bf16_ts(tmem_o, tp + k * 8, make_smem_desc_sw128(v_addr + k * 2048, 16384, 1024), idesc_pv, (j | k) != 0 ? 1u : 0u);
          umma_commit(&v_empty[st]);
          umma_commit(&pv_done[j & 1]);
        }
      }
    }
  } else {
    const int quad = warp & 3;
    const int r = quad * 32 + lane;
    const bool row_valid = q0 + r < L;
    const int qi = p0 + r;
    // an absent row sees nothing
    const int lo = row_valid ? (a.window > 0 ? qi / a.window * a.window : 0) : 1;
    const int hi = row_valid ? qi : 0;
    const uint32_t lane_base = static_cast<uint32_t>(quad * 32) << 16;
    const float sink_l2 = a.sink != nullptr ? a.sink[h] * 1.4426950408889634f : -INFINITY;
    float m_ref = -INFINITY, l = 0.f;
    bool ok = true;
    // why a parity wait on pv_done is enough: see flash_attn.cu
    auto wait_pv = [&](int tile, int where) -> bool {
      return __all_sync(0xffffffffu, mbar_wait(&pv_done[tile & 1], static_cast<uint32_t>(tile >> 1) & 1u, abort_flag, a.status, where));
    };
    for (int j = 0; j < n_tiles && ok; ++j) {
      const uint32_t ts = tmem_base + lane_base + static_cast<uint32_t>((j & 1) * 128);
      const uint32_t tp = tmem_base + lane_base + 384u + static_cast<uint32_t>((j & 1) * 64);
      if (!__all_sync(0xffffffffu, mbar_wait(&s_full[j & 1], static_cast<uint32_t>(j >> 1) & 1u, abort_flag, a.status, 920))) { ok = false; break; }
      tc_fence_after_sync();
      const int k0 = kb + j * WP_BN;
      const bool need_mask = k0 + WP_BN - 1 > p0 || k0 < last_lo || p_last - p0 < WP_BM - 1;
      if (j == 0) {
        // scale > 0, so the largest score is the scaled largest product
        const float t0 = need_mask ? wp_max_pass<true>(ts, k0, lo, hi) : wp_max_pass<false>(ts, k0, lo, hi);
        m_ref = fmaxf(t0 * a.scale_log2, sink_l2);
        if (sink_l2 != -INFINITY) l = exp2f(sink_l2 - m_ref);
      }
      float lsum = 0.f, smax = -INFINITY;
      // a row that has seen no key and has no sink keeps an infinite reference: whatever this pass gives it is
      // recomputed below as soon as the tile holds a key it sees
      if (need_mask) wp_exp_pass<true>(ts, tp, a.scale_log2, m_ref, k0, lo, hi, lsum, smax);
      else wp_exp_pass<false>(ts, tp, a.scale_log2, m_ref, k0, lo, hi, lsum, smax);
      if (j > 0) {
        const float tmax = smax * a.scale_log2;
        const bool need = smax != -INFINITY && tmax > m_ref + WP_RESCALE;
        if (__any_sync(0xffffffffu, need)) {
          if (!wait_pv(j - 1, 921)) { ok = false; break; }
          tc_fence_after_sync();
          const float alpha = need ? exp2f(m_ref - tmax) : 1.f;
          if (need) { m_ref = tmax; l *= alpha; }
#pragma unroll 1
          for (int c = 0; c < HDT / 32; ++c) {
            uint32_t v[32];
            tmem_ld_32x32(tmem_o + lane_base + c * 32, v);
            tmem_wait_ld();
#pragma unroll
            for (int i = 0; i < 32; ++i) v[i] = __float_as_uint(__uint_as_float(v[i]) * alpha);
            tmem_st_32x32(tmem_o + lane_base + c * 32, v);
          }
          lsum = 0.f;
          float unused = -INFINITY;
          if (need_mask) wp_exp_pass<true>(ts, tp, a.scale_log2, m_ref, k0, lo, hi, lsum, unused);
          else wp_exp_pass<false>(ts, tp, a.scale_log2, m_ref, k0, lo, hi, lsum, unused);
        }
      }
      l += lsum;
      tmem_wait_st();
      tc_fence_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(&p_full[j & 1]);
    }
    if (ok && wait_pv(n_tiles - 1, 922)) {
      tc_fence_after_sync();
      const float inv_l = l > 0.f ? 1.f / l : 0.f;
      __nv_bfloat16* orow = a.out + static_cast<size_t>(tok0 + q0 + r) * a.ldo + h * a.dp;
#pragma unroll 1
      for (int c = 0; c < HDT / 32; ++c) {
        uint32_t v[32];
        tmem_ld_32x32(tmem_o + lane_base + c * 32, v);
        tmem_wait_ld();
        if (row_valid) {
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            if (c * 32 + i * 8 < a.dp) {
              uint4 o;
              o.x = pack_bf16x2(__uint_as_float(v[i * 8 + 0]) * inv_l, __uint_as_float(v[i * 8 + 1]) * inv_l);
              o.y = pack_bf16x2(__uint_as_float(v[i * 8 + 2]) * inv_l, __uint_as_float(v[i * 8 + 3]) * inv_l);
              o.z = pack_bf16x2(__uint_as_float(v[i * 8 + 4]) * inv_l, __uint_as_float(v[i * 8 + 5]) * inv_l);
              o.w = pack_bf16x2(__uint_as_float(v[i * 8 + 6]) * inv_l, __uint_as_float(v[i * 8 + 7]) * inv_l);
              *reinterpret_cast<uint4*>(orow + c * 32 + i * 8) = o;
            }
          }
        }
      }
    }
  }

  __syncwarp();
  if (*abort_flag) __nanosleep(200000);
  tc_fence_before_sync();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after_sync();
    tmem_dealloc(tmem_base, 512);
  }
}

int make_tmap_bf16_2d(CUtensorMap* out, const void* ptr, uint64_t inner, uint64_t outer, uint64_t ld, uint32_t box_inner,
                      uint32_t box_outer);
int make_tmap_bf16_3d(CUtensorMap* out, const void* ptr, uint64_t d0, uint64_t d1, uint64_t d2, uint64_t ld1, uint64_t ld2, uint32_t b0,
                      uint32_t b1, uint32_t b2);

template <int HDT>
static int launch_window_prefill(const CUtensorMap& tq, const CUtensorMap& tk, const CUtensorMap& tv, const Prefill& a, int B, int max_len,
                                 cudaStream_t stream) {
  auto kern = window_prefill_kernel<HDT>;
  static bool configured = false;
  if (!configured) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, PrefillCfg<HDT>::SMEM) != cudaSuccess) return -20;
    configured = true;
  }
  const dim3 grid((max_len + WP_BM - 1) / WP_BM, a.H, B);
  kern<<<grid, WP_THREADS, PrefillCfg<HDT>::SMEM, stream>>>(tq, tk, tv, a);
  return cudaGetLastError() == cudaSuccess ? 0 : -21;
}

}  // namespace rpeg

using namespace rpeg;

// q [T, ldq] bf16 with head h at column h * dp; caches [num_pages, Hkv, PAGE, dp]; cu [B + 1] rows of every request's portion, pos [T]
// its positions, slot [T] its page-table row; out [T, ldo].
extern "C" int rpeg_window_prefill(const void* q, int ldq, const void* kcache, const void* vcache, long long num_pages, const int* page_table,
                                   int max_pages, const int* cu, const int* pos, const int* slot, const float* sink, void* out, int ldo, int T,
                                   int B, int max_len, int H, int Hkv, int dp, int window, float scale, int* status, void* stream) {
  if (T <= 0 || B <= 0 || max_len <= 0) return 0;
  if ((dp & 7) || dp < 8 || dp > 128 || H < 1 || Hkv < 1 || H % Hkv || window < 0 || !(scale > 0.f) || B > 65535 || H > 65535) return -2;
  if ((ldq & 7) || (ldo & 7)) return -2;
  if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(kcache) | reinterpret_cast<uintptr_t>(vcache) |
       reinterpret_cast<uintptr_t>(out)) & 15)
    return -1;
  CUtensorMap tq, tk, tv;
  int rc = make_tmap_bf16_3d(&tq, q, dp, H, T, dp, ldq, 64, 1, WP_BM);
  if (rc) return rc;
  const uint64_t cache_rows = static_cast<uint64_t>(num_pages) * Hkv * RPEG_KV_PAGE;
  rc = make_tmap_bf16_2d(&tk, kcache, dp, cache_rows, dp, 64, RPEG_KV_PAGE);
  if (rc) return rc - 100;
  rc = make_tmap_bf16_2d(&tv, vcache, dp, cache_rows, dp, 64, RPEG_KV_PAGE);
  if (rc) return rc - 200;
  const Prefill a{cu, pos, slot, page_table, max_pages, sink, static_cast<__nv_bfloat16*>(out), ldo, H, Hkv, dp, window,
                  scale * 1.4426950408889634f, status};
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  return dp <= 64 ? launch_window_prefill<64>(tq, tk, tv, a, B, max_len, st) : launch_window_prefill<128>(tq, tk, tv, a, B, max_len, st);
}
