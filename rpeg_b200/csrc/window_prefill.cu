// Prompt attention on the tensor cores, keys and values read from the paged cache, head size up to 128 (bf16).
//
//   O = softmax(Q K^T * scale  [visible keys], sink) V
//
// Row i of a request's portion stands at position p = (cached tokens) + i and sees the keys [floor(p / window) * window, p]
// (window = 0: [0, p]). The portion's own keys were appended to the cache before, so a whole prompt, a portion of one
// and a batch of unequal portions are the same launch: nothing depends on where a prompt was cut.
//
// One CTA works on two 128-row query tiles ("units") over the same key tiles: the same rows of two heads of one KV head,
// or, when the KV head has an odd number of query heads, two neighbouring row tiles of one head. While the softmax warps of one
// unit turn its scores into weights, the tensor cores multiply for the other one. Roles: a TMA warp, an MMA warp, four softmax
// warps per unit (thread = query row).
//   * TMEM: S (128 columns) and O (up to 128) of each unit. A unit's weights replace its scores in place, 32-key chunk by
//     chunk: a weight is handed to the tensor cores as the sum of two bf16 numbers (16 bits), so that rounding the operands
//     of P V does not show; its two parts take 16 of the chunk's 32 columns each.
//   * The commit behind Q K^T of a unit's next tile also covers that unit's P V before it, so the softmax warps need no
//     other signal before they rescale O or overwrite S.
//   * O is rescaled only when a row's maximum grew by more than 8 (log2); a stale reference is exact after the final division.
//   * A key tile is two 64-token cache pages, fetched by TMA through the request's page-table row; tiles start at the page that
//     holds the first key any row of the CTA sees. Heads narrower than the tile (64 or 128) are padded by the TMA unit
//     (out-of-bounds columns read as zero).
//   * The sink opens the softmax: the running maximum starts no lower than the sink's logit and the running sum with its
//     exponential, so it needs no key and no pass of its own.
#include "prefill_softmax.cuh"
#include "rpeg_kernels.h"

namespace rpeg {

constexpr int WP_BM = 128, WP_BN = 128, WP_THREADS = 320, WP_STAGES = 2;

template <int HDT>
struct PrefillCfg {
  static constexpr int TILE = 128 * HDT * 2;               // HDT / 64 atoms of 128 rows x 128 bytes
  static constexpr int SMEM = TILE * (2 + 2 * WP_STAGES) + 1024 + 256;
};

struct Prefill {
  const int* cu; const int* pos; const int* slot;
  const int* page_table; int max_pages;
  const float* sink;
  __nv_bfloat16* out; int ldo;
  int H, Hkv, dp, window;
  int pair_heads;                           // units: two heads of one KV head (1) or two row tiles of one head (0)
  float scale_log2;
  int* status;
};

// One unit: its rows' positions and the key tiles [jb, je) of the CTA that any of its rows sees (je = jb: absent).
struct PrefillUnit {
  int h, q0, p0, p_last, last_lo, jb, je;
};

template <int HDT>
__global__ void __launch_bounds__(WP_THREADS, 1)
window_prefill_kernel(const __grid_constant__ CUtensorMap tmap_q, const __grid_constant__ CUtensorMap tmap_k,
                      const __grid_constant__ CUtensorMap tmap_v, const Prefill a) {
  using Cfg = PrefillCfg<HDT>;
  constexpr int ATOMS = HDT / 64, TILE = Cfg::TILE;
  const int b = blockIdx.z;
  const int bx = gridDim.x - 1 - blockIdx.x;                // late tiles have the most keys: first
  const int tok0 = a.cu[b], L = a.cu[b + 1] - tok0;
  const int q_first = bx * (a.pair_heads ? WP_BM : 2 * WP_BM);
  if (q_first >= L) return;
  const int start = a.pos[tok0];
  const int kb = (a.window > 0 ? (start + q_first) / a.window * a.window : 0) & ~(RPEG_KV_PAGE - 1);
  auto unit = [&](int u) -> PrefillUnit {
    PrefillUnit w;
    w.h = a.pair_heads ? blockIdx.y * 2 + u : blockIdx.y;
    w.q0 = a.pair_heads ? q_first : q_first + u * WP_BM;
    w.p0 = start + w.q0;
    w.p_last = w.p0 + min(WP_BM, L - w.q0) - 1;
    const int first = a.window > 0 ? w.p0 / a.window * a.window : 0;
    w.last_lo = a.window > 0 ? w.p_last / a.window * a.window : 0;
    w.jb = (first - kb) > 0 ? (first - kb) / WP_BN : 0;
    w.je = w.q0 < L ? (w.p_last - kb) / WP_BN + 1 : w.jb;
    return w;
  };
  const PrefillUnit u0 = unit(0), u1 = unit(1);
  const bool has1 = u1.je > u1.jb;
  const int n_tiles = has1 ? max(u0.je, u1.je) : u0.je;
  const int hk = u0.h / (a.H / a.Hkv);

  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* q_sm = smem;                                      // [2]
  uint8_t* k_sm = smem + 2 * TILE;
  uint8_t* v_sm = k_sm + WP_STAGES * TILE;
  uint64_t* bars = reinterpret_cast<uint64_t*>(v_sm + WP_STAGES * TILE);
  uint64_t* q_full = bars;
  uint64_t* k_full = bars + 1;
  uint64_t* k_empty = k_full + WP_STAGES;
  uint64_t* v_full = k_empty + WP_STAGES;
  uint64_t* v_empty = v_full + WP_STAGES;
  uint64_t* s_full = v_empty + WP_STAGES;   // [2], per unit: S of its next tile is complete (and its P V before that)
  uint64_t* p_half = s_full + 2;            // [2], per unit: its weights for the first 64 keys are in place
  uint64_t* p_full = p_half + 2;            // [2], per unit: and for the others
  uint64_t* o_full = p_full + 2;            // [2], per unit: O is final
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(o_full + 2);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int s = 0; s < WP_STAGES; ++s) {
      mbar_init(&k_full[s], 1); mbar_init(&k_empty[s], 1);
      mbar_init(&v_full[s], 1); mbar_init(&v_empty[s], 1);
    }
    for (int u = 0; u < 2; ++u) { mbar_init(&s_full[u], 1); mbar_init(&p_half[u], 4); mbar_init(&p_full[u], 4); mbar_init(&o_full[u], 1); }
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

  if (warp == 0) {
    if (lane == 0) {
      const int* pt = a.page_table + static_cast<size_t>(a.slot[tok0]) * a.max_pages;
      const int last_key = has1 ? max(u0.p_last, u1.p_last) : u0.p_last;
      auto load_tile = [&](const CUtensorMap* map, uint8_t* dst, uint64_t* bar, int j) {
        mbar_expect_tx(bar, TILE);
#pragma unroll
        for (int hf = 0; hf < 2; ++hf) {
          const int pi = kb / RPEG_KV_PAGE + 2 * j + hf;
          // a page past the row's last one is never visible: any valid page will do
          const int page = pi * RPEG_KV_PAGE <= last_key ? pt[pi] : 0;
          const int y = (page * a.Hkv + hk) * RPEG_KV_PAGE;
#pragma unroll
          for (int c = 0; c < ATOMS; ++c) tma_load_2d(dst + c * 16384 + hf * 8192, map, bar, c * 64, y);
        }
      };
      mbar_expect_tx(q_full, has1 ? 2 * TILE : TILE);
#pragma unroll
      for (int u = 0; u < 2; ++u)
        if (u == 0 || has1) {
#pragma unroll
          for (int c = 0; c < ATOMS; ++c)
            tma_load_3d(q_sm + u * TILE + c * 16384, &tmap_q, q_full, c * 64, u ? u1.h : u0.h, tok0 + (u ? u1.q0 : u0.q0));
        }
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
      auto active = [&](int u, int j) -> bool { return u == 0 ? j >= u0.jb && j < u0.je : has1 && j >= u1.jb && j < u1.je; };
      // Q K^T of unit u over tile j; the tile's K buffer is free again once the last unit has used it
      auto issue_qk = [&](int u, int j) {
        const int st = j % WP_STAGES;
        if (active(u, j)) {
          const uint32_t q_addr = smem_u32(q_sm + u * TILE), k_addr = smem_u32(k_sm + st * TILE);
#pragma unroll
          for (int k = 0; k < HDT / 16; ++k) {
            const uint32_t off = static_cast<uint32_t>((k >> 2) * 16384 + (k & 3) * 32);
            umma_bf16_ss(tmem_base + u * 128, make_smem_desc_sw128(q_addr + off, 16, 1024), make_smem_desc_sw128(k_addr + off, 16, 1024),
                         idesc_qk, k != 0 ? 1u : 0u);
          }
          umma_commit(&s_full[u]);
        }
        if (u == 1) umma_commit(&k_empty[st]);
      };
      bool ok = mbar_wait(q_full, 0, abort_flag, a.status, 910);
      if (ok) ok = mbar_wait(&k_full[0], 0, abort_flag, a.status, 911);
      if (ok) {
        tc_fence_after_sync();
        issue_qk(0, 0);
        issue_qk(1, 0);
        for (int j = 0; j < n_tiles && ok; ++j) {
          const int st = j % WP_STAGES, st1 = (j + 1) % WP_STAGES;
          if (!mbar_wait(&v_full[st], static_cast<uint32_t>(j / WP_STAGES) & 1u, abort_flag, a.status, 915)) break;
          if (j + 1 < n_tiles &&
              !mbar_wait(&k_full[st1], static_cast<uint32_t>((j + 1) / WP_STAGES) & 1u, abort_flag, a.status, 912)) break;
          const uint32_t v_addr = smem_u32(v_sm + st * TILE);
#pragma unroll
          for (int u = 0; u < 2; ++u) {
            if (active(u, j)) {
              const int n = j - (u ? u1.jb : u0.jb);         // tiles of this unit before this one
              const uint32_t tp = tmem_base + u * 128, to = tmem_base + 256 + u * 128;
#pragma unroll
              for (int half = 0; half < 2 && ok; ++half) {   // the first keys are multiplied while the last ones are exponentiated
                ok = mbar_wait(half ? &p_full[u] : &p_half[u], static_cast<uint32_t>(n) & 1u, abort_flag, a.status, 913 + half);
                if (!ok) break;
                tc_fence_after_sync();
#pragma unroll
                for (int part = 0; part < 2; ++part)
#pragma unroll
                  for (int k = half * 4; k < half * 4 + 4; ++k)   // 16 keys: 8 packed columns of P, 16 rows (2 KiB) of the V tile
                    umma_bf16_ts(to, tp + (k >> 1) * 32 + part * 16 + (k & 1) * 8, make_smem_desc_sw128(v_addr + k * 2048, 16384, 1024), idesc_pv,
                                 (n | half | part | (k & 3)) != 0 ? 1u : 0u);
              }
              if (!ok) break;
              if (j + 1 == (u ? u1.je : u0.je)) umma_commit(&o_full[u]);
            }
            if (u == 1) umma_commit(&v_empty[st]);
            tc_fence_after_sync();
            if (j + 1 < n_tiles) issue_qk(u, j + 1);
          }
        }
      }
    }
  } else {
    const int ui = (warp - 2) >> 2;
    const PrefillUnit w = ui ? u1 : u0;
    const int quad = warp & 3;
    const int r = quad * 32 + lane;
    const bool row_valid = w.q0 + r < L;
    const int qi = w.p0 + r;
    // an absent row sees nothing
    const int lo = row_valid ? (a.window > 0 ? qi / a.window * a.window : 0) : 1;
    const int hi = row_valid ? qi : 0;
    const uint32_t ts = tmem_base + (static_cast<uint32_t>(quad * 32) << 16) + ui * 128;
    const uint32_t to = ts + 256;
    const float sink_l2 = a.sink != nullptr ? a.sink[w.h] * 1.4426950408889634f : -INFINITY;
    float m_ref = -INFINITY, l = 0.f;
    bool ok = true;
    for (int j = w.jb; j < w.je; ++j) {
      const int n = j - w.jb;
      if (!__all_sync(0xffffffffu, mbar_wait(&s_full[ui], static_cast<uint32_t>(n) & 1u, abort_flag, a.status, 920))) { ok = false; break; }
      tc_fence_after_sync();
      const int k0 = kb + j * WP_BN;
      const bool need_mask = k0 + WP_BN - 1 > w.p0 || k0 < w.last_lo || w.p_last - w.p0 < WP_BM - 1;
      // scale > 0, so the largest score is the scaled largest product
      WpRow row;
      wp_load_row(ts, row);
      if (need_mask) wp_mask_row(row, k0, lo, hi);
      const float tmax = wp_max_row(row) * a.scale_log2;
      if (n == 0) {
        m_ref = fmaxf(tmax, sink_l2);
        if (sink_l2 != -INFINITY) l = exp2f(sink_l2 - m_ref);
      } else {
        const bool need = tmax > m_ref + WP_RESCALE;
        if (__any_sync(0xffffffffu, need)) {
          const float alpha = need ? exp2f(m_ref - tmax) : 1.f;
          if (need) { m_ref = tmax; l *= alpha; }
#pragma unroll 1
          for (int c = 0; c < HDT / 32; ++c) {
            uint32_t v[32];
            tmem_ld_32x32(to + c * 32, v);
            tmem_wait_ld();
#pragma unroll
            for (int i = 0; i < 32; ++i) v[i] = __float_as_uint(__uint_as_float(v[i]) * alpha);
            tmem_st_32x32(to + c * 32, v);
          }
        }
      }
      // a row that has seen no key yet and has no sink: every weight of this tile is masked to zero
      const float m_use = m_ref == -INFINITY ? 0.f : m_ref;
      l += wp_exp_row(row, ts, a.scale_log2, m_use, &p_half[ui]);
      tmem_wait_st();
      tc_fence_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(&p_full[ui]);
    }
    if (ok && w.je > w.jb && __all_sync(0xffffffffu, mbar_wait(&o_full[ui], 0, abort_flag, a.status, 922))) {
      tc_fence_after_sync();
      const float inv_l = l > 0.f ? 1.f / l : 0.f;
      __nv_bfloat16* orow = a.out + static_cast<size_t>(tok0 + w.q0 + r) * a.ldo + w.h * a.dp;
#pragma unroll 1
      for (int c = 0; c < HDT / 32; ++c) {
        uint32_t v[32];
        tmem_ld_32x32(to + c * 32, v);
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
  const int rows_per_cta = a.pair_heads ? WP_BM : 2 * WP_BM;
  const dim3 grid((max_len + rows_per_cta - 1) / rows_per_cta, a.pair_heads ? a.H / 2 : a.H, B);
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
                  (H / Hkv) % 2 == 0 ? 1 : 0, scale * 1.4426950408889634f, status};
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  return dp <= 64 ? launch_window_prefill<64>(tq, tk, tv, a, B, max_len, st) : launch_window_prefill<128>(tq, tk, tv, a, B, max_len, st);
}
