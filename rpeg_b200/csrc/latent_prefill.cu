// Prompt attention of latent layers on the tensor cores (bf16), over keys and values that were formed from the cached rows:
//
//   O_h = softmax((q_h . k_h + q'_h . k') * scale  [visible keys], sink) v_h
//
// k_h, v_h come from one GEMM over the rows the requests see (latent_gather); the rotated key part k' lies in those rows and is shared by
// all heads, so it is never copied per head: the key tile of a head is built in shared memory from both matrices. Row i of a request's
// portion stands at position p = (cached tokens) + i and sees the last `window` positions up to p (0: all). Whole prompts, portions
// and batches of unequal portions are the same launch.
//
// Like the chunked kernel (window_prefill.cu) one CTA works on two 128-row query tiles ("units") of one head over the same key tiles, and while
// the softmax warps of one unit turn its scores into weights the tensor cores multiply for the other. Roles: a TMA warp, an MMA
// warp, four softmax warps per unit (thread = query row); weights replace the scores in place as two bf16 parts. What differs:
//   * A query / key row is KA atoms of 64 columns (unrotated ones, then rotated ones), a value row VA atoms. The TMA unit pads narrower ones.
//   * Key and value atoms (128 rows x 128 bytes) share one ring, freed atom by atom: with 192-wide keys and 128-wide values two key
//     tiles and a value tile are in flight.
//   * A value atom is a matrix product of its own (64 output columns), so atoms need not be neighbours in the ring.
#include "prefill_softmax.cuh"
#include "rpeg_kernels.h"

namespace rpeg {

constexpr int LP_BM = 128, LP_BN = 128, LP_THREADS = 320, LP_ATOM = 128 * 128;

template <int KA, int VA>
struct LatentPrefillCfg {
  static constexpr int Q_BYTES = 2 * KA * LP_ATOM;
  static constexpr int RAW = (227 * 1024 - 1536 - Q_BYTES) / LP_ATOM;
  static constexpr int SLOTS = RAW > 10 ? 10 : RAW;
  static constexpr int SMEM = Q_BYTES + SLOTS * LP_ATOM + 1536;
  static_assert(SLOTS >= KA + VA, "a key tile and a value tile must fit");
};

struct LatentPrefill {
  const int* cu; const int* pos;
  const int* off; const int* lo;            // rows of what a request sees, first position of it
  const float* sink;
  __nv_bfloat16* out; int ldo;
  int vdim_p, nope_atoms, nope_steps, rot_steps, window;   // k16 steps of the last unrotated / rotated atom
  float scale_log2;
  int* status;
};

struct LatentUnit {
  int q0, p0, p_last, last_lo, jb, je;      // its rows' positions and the key tiles [jb, je) any of them sees (je = jb: absent)
};

template <int KA, int VA>
__global__ void __launch_bounds__(LP_THREADS, 1)
latent_prefill_kernel(const __grid_constant__ CUtensorMap tmap_qn, const __grid_constant__ CUtensorMap tmap_qr, const __grid_constant__ CUtensorMap tmap_kn,
                      const __grid_constant__ CUtensorMap tmap_kr, const __grid_constant__ CUtensorMap tmap_v, const LatentPrefill a) {
  using Cfg = LatentPrefillCfg<KA, VA>;
  constexpr int SLOTS = Cfg::SLOTS, TA = KA + VA;
  const int b = blockIdx.z, h = blockIdx.y;
  const int bx = gridDim.x - 1 - blockIdx.x;                // late tiles have the most keys: first
  const int tok0 = a.cu[b], L = a.cu[b + 1] - tok0;
  const int q_first = bx * 2 * LP_BM;
  if (q_first >= L) return;
  const int start = a.pos[tok0];
  auto first_key = [&](int p) { return a.window > 0 ? max(0, p - a.window + 1) : 0; };
  const int kb = first_key(start + q_first);
  auto unit = [&](int u) -> LatentUnit {
    LatentUnit w;
    w.q0 = q_first + u * LP_BM;
    w.p0 = start + w.q0;
    w.p_last = w.p0 + min(LP_BM, L - w.q0) - 1;
    w.last_lo = first_key(w.p_last);
    w.jb = (first_key(w.p0) - kb) / LP_BN;
    w.je = w.q0 < L ? (w.p_last - kb) / LP_BN + 1 : w.jb;
    return w;
  };
  const LatentUnit u0 = unit(0), u1 = unit(1);
  const bool has1 = u1.je > u1.jb;
  const int n_tiles = has1 ? max(u0.je, u1.je) : u0.je;

  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint8_t* q_sm = smem;                                      // [2][KA] atoms
  uint8_t* ring = smem + Cfg::Q_BYTES;
  uint64_t* bars = reinterpret_cast<uint64_t*>(ring + SLOTS * LP_ATOM);
  uint64_t* q_full = bars;
  uint64_t* full = bars + 1;                // [SLOTS]
  uint64_t* empty = full + SLOTS;           // [SLOTS]
  uint64_t* s_full = empty + SLOTS;         // [2], per unit: S of its next tile is complete (and its P V before that)
  uint64_t* p_half = s_full + 2;            // [2], per unit: its weights for the first 64 keys are in place
  uint64_t* p_full = p_half + 2;            // [2], per unit: and for the others
  uint64_t* o_full = p_full + 2;            // [2], per unit: O is final
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(o_full + 2);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int s = 0; s < SLOTS; ++s) { mbar_init(&full[s], 1); mbar_init(&empty[s], 1); }
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
  // atom number i of the CTA's sequence K(0) V(0) K(1) V(1) ...: its slot, and the parity of the phase in which it is complete
  auto slot_of = [](int i) { return i % SLOTS; };
  auto parity_of = [](int i) { return static_cast<uint32_t>(i / SLOTS) & 1u; };

  if (warp == 0) {
    if (lane == 0) {
      const int row0 = a.off[b] + kb - a.lo[b];
      mbar_expect_tx(q_full, (has1 ? 2 : 1) * KA * LP_ATOM);
      for (int u = 0; u < (has1 ? 2 : 1); ++u)
#pragma unroll
        for (int c = 0; c < KA; ++c) {
          const bool rot = c >= a.nope_atoms;
          tma_load_3d(q_sm + (u * KA + c) * LP_ATOM, rot ? &tmap_qr : &tmap_qn, q_full, (rot ? c - a.nope_atoms : c) * 64, h,
                      tok0 + (u ? u1.q0 : u0.q0));
        }
      bool ok = true;
      for (int j = 0; j < n_tiles && ok; ++j) {
        const int y = row0 + j * LP_BN;
        for (int c = 0; c < TA; ++c) {
          const int i = j * TA + c, s = slot_of(i);
          ok = mbar_wait(&empty[s], parity_of(i) ^ 1u, abort_flag, a.status, 1200);
          if (!ok) break;
          mbar_expect_tx(&full[s], LP_ATOM);
          if (c >= KA) tma_load_3d(ring + s * LP_ATOM, &tmap_v, &full[s], (c - KA) * 64, h, y);
          else if (c >= a.nope_atoms) tma_load_2d(ring + s * LP_ATOM, &tmap_kr, &full[s], (c - a.nope_atoms) * 64, y);
          else tma_load_3d(ring + s * LP_ATOM, &tmap_kn, &full[s], c * 64, h, y);
        }
      }
    }
  } else if (warp == 1) {
    if (lane == 0) {
      constexpr uint32_t idesc_qk = make_idesc_bf16(128, 128, 0, 0);
      constexpr uint32_t idesc_pv = make_idesc_bf16(128, 64, 0, 1);
      auto active = [&](int u, int j) -> bool { return u == 0 ? j >= u0.jb && j < u0.je : has1 && j >= u1.jb && j < u1.je; };
      auto wait_atoms = [&](int i0, int n) -> bool {
        for (int i = i0; i < i0 + n; ++i)
          if (!mbar_wait(&full[slot_of(i)], parity_of(i), abort_flag, a.status, 1210)) return false;
        tc_fence_after_sync();
        return true;
      };
      // Q K^T of unit u over tile j; the tile's key atoms are free again once the last unit has used them
      auto issue_qk = [&](int u, int j) {
        if (active(u, j)) {
          uint32_t acc = 0u;
#pragma unroll
          for (int c = 0; c < KA; ++c) {
            const uint32_t qa = smem_u32(q_sm + (u * KA + c) * LP_ATOM), ka = smem_u32(ring + slot_of(j * TA + c) * LP_ATOM);
            const int steps = c == a.nope_atoms - 1 ? a.nope_steps : (c == KA - 1 ? a.rot_steps : 4);
#pragma unroll
            for (int k = 0; k < 4; ++k)
              if (k < steps) {
                umma_bf16_ss(tmem_base + u * 128, make_smem_desc_sw128(qa + k * 32, 16, 1024), make_smem_desc_sw128(ka + k * 32, 16, 1024), idesc_qk, acc);
                acc = 1u;
              }
          }
          umma_commit(&s_full[u]);
        }
        if (u == 1)
#pragma unroll
          for (int c = 0; c < KA; ++c) umma_commit(&empty[slot_of(j * TA + c)]);
      };
      bool ok = mbar_wait(q_full, 0, abort_flag, a.status, 1211) && wait_atoms(0, KA);
      if (ok) {
        issue_qk(0, 0);
        issue_qk(1, 0);
        for (int j = 0; j < n_tiles && ok; ++j) {
          if (!wait_atoms(j * TA + KA, VA)) break;
          if (j + 1 < n_tiles && !wait_atoms((j + 1) * TA, KA)) break;
#pragma unroll
          for (int u = 0; u < 2; ++u) {
            if (active(u, j)) {
              const int n = j - (u ? u1.jb : u0.jb);         // tiles of this unit before this one
              const uint32_t tp = tmem_base + u * 128, to = tmem_base + 256 + u * 128;
#pragma unroll
              for (int half = 0; half < 2 && ok; ++half) {   // the first keys are multiplied while the last ones are exponentiated
                ok = mbar_wait(half ? &p_full[u] : &p_half[u], static_cast<uint32_t>(n) & 1u, abort_flag, a.status, 1213 + half);
                if (!ok) break;
                tc_fence_after_sync();
#pragma unroll
                for (int va = 0; va < VA; ++va) {
                  const uint32_t v_addr = smem_u32(ring + slot_of(j * TA + KA + va) * LP_ATOM);
#pragma unroll
                  for (int part = 0; part < 2; ++part)
#pragma unroll
                    for (int k = half * 4; k < half * 4 + 4; ++k)   // 16 keys: 8 packed columns of P, 16 rows (2 KiB) of the value atom
                      umma_bf16_ts(to + va * 64, tp + (k >> 1) * 32 + part * 16 + (k & 1) * 8, make_smem_desc_sw128(v_addr + k * 2048, LP_ATOM, 1024),
                                   idesc_pv, (n | half | part | (k & 3)) != 0 ? 1u : 0u);
                }
              }
              if (!ok) break;
              if (j + 1 == (u ? u1.je : u0.je)) umma_commit(&o_full[u]);
            }
            if (u == 1)
#pragma unroll
              for (int va = 0; va < VA; ++va) umma_commit(&empty[slot_of(j * TA + KA + va)]);
            tc_fence_after_sync();
            if (j + 1 < n_tiles) issue_qk(u, j + 1);
          }
        }
      }
    }
  } else {
    const int ui = (warp - 2) >> 2;
    const LatentUnit w = ui ? u1 : u0;
    const int quad = warp & 3;
    const int r = quad * 32 + lane;
    const bool row_valid = w.q0 + r < L;
    const int qi = w.p0 + r;
    const int lo = row_valid ? first_key(qi) : 1, hi = row_valid ? qi : 0;     // an absent row sees nothing
    const uint32_t ts = tmem_base + (static_cast<uint32_t>(quad * 32) << 16) + ui * 128;
    const uint32_t to = ts + 256;
    const float sink_l2 = a.sink != nullptr ? a.sink[h] * 1.4426950408889634f : -INFINITY;
    float m_ref = -INFINITY, l = 0.f;
    bool ok = true;
    for (int j = w.jb; j < w.je; ++j) {
      const int n = j - w.jb;
      if (!__all_sync(0xffffffffu, mbar_wait(&s_full[ui], static_cast<uint32_t>(n) & 1u, abort_flag, a.status, 1220))) { ok = false; break; }
      tc_fence_after_sync();
      const int k0 = kb + j * LP_BN;
      const bool need_mask = k0 + LP_BN - 1 > w.p0 || k0 < w.last_lo || w.p_last - w.p0 < LP_BM - 1;
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
          // a row that has seen no key yet (its window starts in a later tile) has nothing to rescale
          const float alpha = need ? (m_ref == -INFINITY ? 0.f : exp2f(m_ref - tmax)) : 1.f;
          if (need) { m_ref = tmax; l *= alpha; }
#pragma unroll 1
          for (int c = 0; c < VA * 2; ++c) {
            uint32_t v[32];
            tmem_ld_32x32(to + c * 32, v);
            tmem_wait_ld();
#pragma unroll
            for (int i = 0; i < 32; ++i) v[i] = __float_as_uint(__uint_as_float(v[i]) * alpha);
            tmem_st_32x32(to + c * 32, v);
          }
        }
      }
      const float m_use = m_ref == -INFINITY ? 0.f : m_ref;
      l += wp_exp_row(row, ts, a.scale_log2, m_use, &p_half[ui]);
      tmem_wait_st();
      tc_fence_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(&p_full[ui]);
    }
    if (ok && w.je > w.jb && __all_sync(0xffffffffu, mbar_wait(&o_full[ui], 0, abort_flag, a.status, 1222))) {
      tc_fence_after_sync();
      const float inv_l = l > 0.f ? 1.f / l : 0.f;
      __nv_bfloat16* orow = a.out + static_cast<size_t>(tok0 + w.q0 + r) * a.ldo + h * a.vdim_p;
#pragma unroll 1
      for (int c = 0; c < VA * 2; ++c) {
        uint32_t v[32];
        tmem_ld_32x32(to + c * 32, v);
        tmem_wait_ld();
        if (row_valid) {
#pragma unroll
          for (int i = 0; i < 4; ++i) {
            if (c * 32 + i * 8 < a.vdim_p) {
              uint32_t o[4];
#pragma unroll
              for (int e = 0; e < 4; ++e)
                o[e] = pack_bf16x2(__uint_as_float(v[i * 8 + 2 * e]) * inv_l, __uint_as_float(v[i * 8 + 2 * e + 1]) * inv_l);
              *reinterpret_cast<uint4*>(orow + c * 32 + i * 8) = make_uint4(o[0], o[1], o[2], o[3]);
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

template <int KA, int VA>
static int launch_latent_prefill(const CUtensorMap* t, const LatentPrefill& a, int H, int B, int max_len, cudaStream_t stream) {
  using Cfg = LatentPrefillCfg<KA, VA>;
  auto kern = latent_prefill_kernel<KA, VA>;
  static bool configured = false;
  if (!configured) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, Cfg::SMEM) != cudaSuccess) return -20;
    configured = true;
  }
  kern<<<dim3((max_len + 2 * LP_BM - 1) / (2 * LP_BM), H, B), LP_THREADS, Cfg::SMEM, stream>>>(t[0], t[1], t[2], t[3], t[4], a);
  return cudaGetLastError() == cudaSuccess ? 0 : -21;
}

}  // namespace rpeg

using namespace rpeg;

// Whether these (padded) sizes are covered.
extern "C" int rpeg_latent_prefill_fits(int dim_p, int rot_p, int vdim_p) {
  return dim_p >= 8 && vdim_p >= 8 && (dim_p + 63) / 64 + (rot_p + 63) / 64 <= 3 && (vdim_p + 63) / 64 <= 2;
}

// q: T rows of `ldq` elements, head h at h * hsq: [dim_p | rot_p]; kv [n_rows, H * dim_p + H * vdim_p] (keys of all heads, then values);
// rows [n_rows, W] the gathered cache rows (rotated part from column rank_p on); out [T, ldo], head h at h * vdim_p.
extern "C" int rpeg_latent_prefill(const void* q, int ldq, int hsq, const void* kv, const void* rows, long long n_rows, int W, int rank_p, const int* cu,
                                   const int* pos, const int* off, const int* lo, const float* sink, void* out, int ldo, int T, int B, int max_len,
                                   int H, int dim_p, int rot_p, int vdim_p, int window, float scale, int* status, void* stream) {
  if (T <= 0 || B <= 0 || max_len <= 0) return 0;
  if (((dim_p | rot_p | vdim_p | ldq | hsq | ldo | W | rank_p) & 7) || H < 1 || window < 0 || !(scale > 0.f) || B > 65535 || H > 65535) return -2;
  if (!rpeg_latent_prefill_fits(dim_p, rot_p, vdim_p)) return -3;
  if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(kv) | reinterpret_cast<uintptr_t>(rows) | reinterpret_cast<uintptr_t>(out)) & 15)
    return -1;
  const int na = (dim_p + 63) / 64, ra = (rot_p + 63) / 64, va = (vdim_p + 63) / 64;
  const __nv_bfloat16 *qb = static_cast<const __nv_bfloat16*>(q), *kvb = static_cast<const __nv_bfloat16*>(kv), *rb = static_cast<const __nv_bfloat16*>(rows);
  const uint64_t ldkv = static_cast<uint64_t>(H) * (dim_p + vdim_p);
  CUtensorMap t[5];
  int rc = make_tmap_bf16_3d(&t[0], qb, dim_p, H, T, hsq, ldq, 64, 1, LP_BM);
  if (rc) return rc;
  rc = make_tmap_bf16_3d(&t[2], kvb, dim_p, H, n_rows, dim_p, ldkv, 64, 1, LP_BN);
  if (rc) return rc - 100;
  rc = make_tmap_bf16_3d(&t[4], kvb + static_cast<size_t>(H) * dim_p, vdim_p, H, n_rows, vdim_p, ldkv, 64, 1, LP_BN);
  if (rc) return rc - 200;
  t[1] = t[0];
  t[3] = t[2];
  if (ra > 0) {
    rc = make_tmap_bf16_3d(&t[1], qb + dim_p, rot_p, H, T, hsq, ldq, 64, 1, LP_BM);
    if (rc) return rc - 300;
    rc = make_tmap_bf16_2d(&t[3], rb + rank_p, rot_p, n_rows, W, 64, LP_BN);
    if (rc) return rc - 400;
  }
  auto last_steps = [](int width) { return width > 0 ? ((width - 1) % 64) / 16 + 1 : 4; };
  const LatentPrefill a{cu, pos, off, lo, sink, static_cast<__nv_bfloat16*>(out), ldo, vdim_p, na, last_steps(dim_p), last_steps(rot_p), window,
                        scale * 1.4426950408889634f, status};
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  switch ((na + ra) * 10 + va) {
    case 11: return launch_latent_prefill<1, 1>(t, a, H, B, max_len, st);
    case 12: return launch_latent_prefill<1, 2>(t, a, H, B, max_len, st);
    case 21: return launch_latent_prefill<2, 1>(t, a, H, B, max_len, st);
    case 22: return launch_latent_prefill<2, 2>(t, a, H, B, max_len, st);
    case 31: return launch_latent_prefill<3, 1>(t, a, H, B, max_len, st);
    case 32: return launch_latent_prefill<3, 2>(t, a, H, B, max_len, st);
    default: return -3;
  }
}
