// Latent attention of single query rows on the tensor cores (bf16): up to 32 heads of one row against the cached rows themselves.
//
//   S^T[key, head]  = row_key . q_h            q_h [W] = (query through the key map | rotated part), row [W] = (latent | rotated part)
//   P^T             = softmax over the keys (S^T * scale  [visible keys], sink)
//   O^T[d, head]    = sum_key row_key[d] P^T[key, head]      for the latent's dimensions d < rank
//
// A cached row is read from memory once, for the scores of all heads and for their averages: the tile of 64 keys (one cache page) that
// TMA brings to shared memory is operand A of both products, K-major in the first (64 x W), MN-major along its other axis in the second
// (128 latent dimensions x 64 keys at a time). Roles: a TMA warp, an MMA warp, four warps that turn scores into weights and later
// rescale and store the accumulator.
//   * The 64-row scores lie in the first 16 TMEM lanes of each warp's quadrant: a warp sees 16 keys of all 32 heads. The heads are
//     dealt to the two half warps, so a lane works on one key and 16 heads.
//   * A weight goes to the tensor cores as the sum of two bf16 numbers (16 bits), so that rounding the operands does not show: columns
//     0..31 of operand P are the leading parts, 32..63 the remainders, and the two halves of the accumulator are added in the end.
//     Both parts cost one pass.
//   * The maximum a head's weights refer to is set by the first tile and changed (and the accumulator rescaled) only when some score
//     exceeds it by more than 8 (log2); a barrier that also takes the vote is all the warps exchange otherwise.
//   * Scores are double buffered in TMEM, weights in shared memory: the product for the next page runs under the softmax of this one.
// Splits of a row's pages leave unnormalised partial sums; latent_merge adds them up.
#include "act_io.cuh"
#include "rpeg_kernels.h"

namespace rpeg {

constexpr int LD_PAGE = RPEG_KV_PAGE, LD_HEADS = 32, LD_THREADS = 192;
constexpr int LD_ATOM = LD_PAGE * 128;             // 64 keys x 64 columns, 128-byte swizzled
constexpr int LD_Q_ATOM = LD_HEADS * 128;
constexpr int LD_P_BYTES = LD_PAGE * 128;          // 64 keys x [leading parts; remainders] of 32 heads
constexpr int LD_MAX_ATOMS = 9, LD_MAX_BLOCKS = 4; // rows of up to 576 elements, latents of up to 512
constexpr float LD_RESCALE = 8.0f;

struct LatentDecode {
  const int* page_table; int max_pages;
  const int* slot; const int* pos; const int* lens;
  const float* sink;
  __nv_bfloat16* out;                              // [rows, H, rank_p]
  float* partial;                                  // [rows, H, nsplit, rank_p], then (max, sum) [rows, H, nsplit]
  long long ml_offset;
  int H, rank_p, atoms, stage_atoms, blocks, window, nsplit, stages, tmem_cols;
  float scale_log2;
  int* status;
};

// Barrier of the four softmax warps; returns whether any of their threads votes yes.
__device__ __forceinline__ bool softmax_vote(bool yes) {
  uint32_t any;
  asm volatile(
      "{\n\t.reg .pred p, q;\n\t"
      "setp.ne.u32 q, %1, 0;\n\t"
      "barrier.cta.red.or.pred p, 1, 128, q;\n\t"
      "selp.u32 %0, 1, 0, p;\n\t}"
      : "=r"(any)
      : "r"(yes ? 1u : 0u)
      : "memory");
  return any != 0;
}
__device__ __forceinline__ void softmax_sync() { asm volatile("barrier.cta.sync 1, 128;" ::: "memory"); }

// v[i] of 16 lanes -> in lane c of the 16: the maximum (or sum) of their v[c].
template <bool MAX>
__device__ __forceinline__ float half_warp_transpose(float (&v)[16], int lane) {
#pragma unroll
  for (int n = 8; n >= 1; n >>= 1) {
    const bool up = lane & n;
#pragma unroll
    for (int i = 0; i < 8; ++i)
      if (i < n) {
        const float send = up ? v[i] : v[i + n], keep = up ? v[i + n] : v[i];
        const float got = __shfl_xor_sync(0xffffffffu, send, n);
        v[i] = MAX ? fmaxf(keep, got) : keep + got;
      }
  }
  return v[0];
}

__global__ void __launch_bounds__(LD_THREADS, 2)
latent_decode_kernel(const __grid_constant__ CUtensorMap tmap_q, const __grid_constant__ CUtensorMap tmap_c, const LatentDecode a) {
  extern __shared__ uint8_t smem_raw[];
  __shared__ float warp_part[4][LD_HEADS], alpha_sm[LD_HEADS];
  __shared__ int failed[4];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  const int stage_bytes = a.stage_atoms * LD_ATOM;
  uint8_t* q_sm = smem;
  uint8_t* c_sm = q_sm + a.atoms * LD_Q_ATOM;
  uint8_t* p_sm = c_sm + a.stages * stage_bytes;
  uint64_t* bars = reinterpret_cast<uint64_t*>(p_sm + 2 * LD_P_BYTES);
  uint64_t* q_full = bars;
  uint64_t* s_full = bars + 1;              // [2] scores of a tile are complete
  uint64_t* p_full = s_full + 2;            // [2] weights of a tile are in shared memory (and its scores have been read)
  uint64_t* pv_done = p_full + 2;           // [2] the accumulator holds a tile, its weights' buffer is free
  uint64_t* full = pv_done + 2;             // [stages]
  uint64_t* empty = full + a.stages;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(empty + a.stages);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

  const int row = blockIdx.x, h0 = blockIdx.y * LD_HEADS, split = blockIdx.z;
  const int nh = min(LD_HEADS, a.H - h0);
  const int warp = uniform_warp(), lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    tma_prefetch_desc(&tmap_q);
    tma_prefetch_desc(&tmap_c);
    mbar_init(q_full, 1);
    for (int i = 0; i < 2; ++i) { mbar_init(&s_full[i], 1); mbar_init(&p_full[i], 4); mbar_init(&pv_done[i], 1); }
    for (int s = 0; s < a.stages; ++s) { mbar_init(&full[s], 1); mbar_init(&empty[s], 1); }
    *abort_flag = 0;
    fence_mbar_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, a.tmem_cols);
    tmem_relinquish();
  }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem = *tmem_slot;
  griddep_launch();
  griddep_wait();
  const int L = a.lens != nullptr ? a.lens[row] : a.pos[row] + 1;
  const int key0 = a.window > 0 ? max(0, L - a.window) : 0;
  const int pg0 = key0 / LD_PAGE, pg1 = L > 0 ? (L + LD_PAGE - 1) / LD_PAGE : pg0;
  const int per = (pg1 - pg0 + a.nsplit - 1) / a.nsplit;
  const int pa = min(pg1, pg0 + split * per);
  const int n_tiles = __shfl_sync(0xffffffffu, min(pg1, pa + per) - pa, 0);
  auto parity2 = [](int j) { return static_cast<uint32_t>(j >> 1) & 1u; };      // of the phase tile j completes on a pair of barriers
  constexpr int O_COL = 2 * LD_HEADS;                                            // TMEM: two score buffers, then the accumulator

  if (warp == 0) {
    if (lane == 0 && n_tiles > 0) {
      const int* pt = a.page_table + static_cast<size_t>(a.slot[row]) * a.max_pages;
      mbar_expect_tx(q_full, a.atoms * LD_Q_ATOM);
      for (int c = 0; c < a.atoms; ++c) tma_load_2d(q_sm + c * LD_Q_ATOM, &tmap_q, q_full, c * 64, row * a.H + h0);
      int st = 0;
      uint32_t phase = 1u;
      int page = pt[pa];
      for (int j = 0; j < n_tiles; ++j) {
        const int y = page * LD_PAGE;
        if (j + 1 < n_tiles) page = pt[pa + j + 1];              // the next page's number arrives under this page's copies
        if (!mbar_wait(&empty[st], phase, abort_flag, a.status, 1100)) break;
        mbar_expect_tx(&full[st], a.atoms * LD_ATOM);
        uint8_t* dst = c_sm + st * stage_bytes;
        for (int c = 0; c < a.atoms; ++c) tma_load_2d(dst + c * LD_ATOM, &tmap_c, &full[st], c * 64, y);
        if (++st == a.stages) { st = 0; phase ^= 1u; }
      }
    }
  } else if (warp == 1) {
    if (n_tiles > 0) {                               // all lanes, converged; one of them issues
      const bool leader = elect_one();
      constexpr uint32_t idesc_s = make_idesc_bf16(LD_PAGE, LD_HEADS, 0, 0);
      constexpr uint32_t idesc_o = make_idesc_bf16(128, 2 * LD_HEADS, 1, 1);
      const uint64_t q_desc = make_smem_desc_sw128(smem_u32(q_sm), 16, 1024);
      const uint64_t ck_desc = make_smem_desc_sw128(smem_u32(c_sm), 16, 1024);            // keys as rows of the first product
      const uint64_t cv_desc = make_smem_desc_sw128(smem_u32(c_sm), LD_ATOM, 1024);       // the same keys along their other axis
      const uint64_t p_desc = make_smem_desc_sw128(smem_u32(p_sm), LD_P_BYTES, 1024);
      int qs = 0, ps = 0;                   // stages of the next score and the next average
      uint32_t q_phase = 0u;
      auto scores = [&](int j) {
        tc_fence_after_sync();
        const uint32_t ts = tmem + (j & 1) * LD_HEADS;
        uint64_t qd = q_desc, cd = smem_desc_at(ck_desc, qs * stage_bytes);
        for (int c = 0; c < a.atoms; ++c) {                       // columns past the row's end are zeros in both operands
#pragma unroll
          for (int k = 0; k < 4; ++k)
            if (leader) umma_bf16_ss(ts, smem_desc_at(cd, k * 32), smem_desc_at(qd, k * 32), idesc_s, (c | k) != 0 ? 1u : 0u);
          qd = smem_desc_at(qd, LD_Q_ATOM);
          cd = smem_desc_at(cd, LD_ATOM);
        }
        if (leader) umma_commit(&s_full[j & 1]);
        if (++qs == a.stages) { qs = 0; q_phase ^= 1u; }
      };
      auto averages = [&](int j) {
        tc_fence_after_sync();
        const uint64_t pd = smem_desc_at(p_desc, (j & 1) * LD_P_BYTES);
        uint64_t cd = smem_desc_at(cv_desc, ps * stage_bytes);
        uint32_t to = tmem + O_COL;
        for (int blk = 0; blk < a.blocks; ++blk) {
#pragma unroll
          for (int k = 0; k < LD_PAGE / 16; ++k)                  // 16 keys: 16 rows (2 KiB) of both operands' atoms
            if (leader) umma_bf16_ss(to, smem_desc_at(cd, k * 2048), smem_desc_at(pd, k * 2048), idesc_o, (j | k) != 0 ? 1u : 0u);
          cd = smem_desc_at(cd, 2 * LD_ATOM);
          to += 2 * LD_HEADS;
        }
        if (leader) {
          umma_commit(&pv_done[j & 1]);
          umma_commit(&empty[ps]);
        }
        if (++ps == a.stages) ps = 0;
      };
      // Whatever is ready next: averages (they free a stage), else scores of a tile that has arrived, one tile ahead of the weights at
      // most. With two stages in flight a fixed order would make one of them wait for the other's copy.
      auto wait = [&](uint64_t* bar, uint32_t parity, int where) -> bool {
        return __all_sync(0xffffffffu, mbar_wait(bar, parity, abort_flag, a.status, where));
      };
      auto arrived = [&](uint64_t* bar, uint32_t parity) -> bool { return __all_sync(0xffffffffu, mbar_test_wait(bar, parity)); };
      bool ok = wait(q_full, 0, 1111);
      int jq = 0, jp = 0;
      while (ok && jp < n_tiles) {
        const bool can_q = jq < n_tiles && jq <= jp + 1, can_p = jp < jq;
        if (can_q && can_p) {
          uint64_t t0 = 0;
          for (uint32_t spin = 1;; ++spin) {
            if (arrived(&p_full[jp & 1], parity2(jp))) { averages(jp++); break; }
            if (arrived(&full[qs], q_phase)) { scores(jq++); break; }
            if ((spin & 1023u) == 0u) {
              if (t0 == 0) t0 = global_timer_ns();
              if (__any_sync(0xffffffffu, *abort_flag || global_timer_ns() - t0 > RPEG_WAIT_LIMIT_NS)) {
                *abort_flag = 1;
                if (leader) record_error(a.status, RPEG_ERR_MBAR_TIMEOUT, 1112, jp);
                ok = false;
                break;
              }
            }
          }
        } else if (can_q) {
          ok = wait(&full[qs], q_phase, 1110);
          if (ok) scores(jq++);
        } else {
          ok = wait(&p_full[jp & 1], parity2(jp), 1113);
          if (ok) averages(jp++);
        }
      }
    }
  } else {
    const int quad = warp & 3;
    const uint32_t lanes = tmem + (static_cast<uint32_t>(quad * 32) << 16);
    const uint32_t to = lanes + O_COL;
    const int key = quad * 16 + (lane & 15);         // of the tile; this lane's heads: (lane >> 4) * 16 + i
    const float scale = a.scale_log2;
    float m_ref = -INFINITY;                         // of head `lane`, the same in all four warps
    float shift[16], l[16];                          // of the lane's 16 heads: what m_ref is, sum of the weights of this lane's keys
#pragma unroll
    for (int i = 0; i < 16; ++i) { shift[i] = 0.f; l[i] = 0.f; }
    bool alive = true;
    for (int n = 0; n < n_tiles && alive; ++n) {
      const bool ok = __all_sync(0xffffffffu, mbar_wait(&s_full[n & 1], parity2(n), abort_flag, a.status, 1120));
      float x[16];
      {
        uint32_t s[32];
        tc_fence_after_sync();
        tmem_ld_32x32(lanes + (n & 1) * LD_HEADS, s);
        tmem_wait_ld();
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          const float other = __shfl_sync(0xffffffffu, __uint_as_float(s[16 + i]), lane & 15);
          x[i] = lane < 16 ? __uint_as_float(s[i]) : other;
        }
      }
      const int k0 = (pa + n) * LD_PAGE;
      if (k0 + key < key0 || k0 + key >= L) {
#pragma unroll
        for (int i = 0; i < 16; ++i) x[i] = -INFINITY;
      }
      float over = -INFINITY;
#pragma unroll
      for (int i = 0; i < 16; ++i) over = fmaxf(over, fmaf(x[i], scale, -shift[i]));
      if (softmax_vote(n == 0 || !ok || over > LD_RESCALE)) {
        // rare: every head's maximum over the tile, new references, and the accumulator under them
        if (lane == 0) failed[quad] = ok ? 0 : 1;
        float t[16];
#pragma unroll
        for (int i = 0; i < 16; ++i) t[i] = x[i];
        warp_part[quad][lane] = half_warp_transpose<true>(t, lane);        // (scale > 0)
        softmax_sync();
        if (failed[0] | failed[1] | failed[2] | failed[3]) { alive = false; break; }
        const float tmax = fmaxf(fmaxf(warp_part[0][lane], warp_part[1][lane]), fmaxf(warp_part[2][lane], warp_part[3][lane])) * scale;
        float al = 1.f;
        if (n == 0) {
          m_ref = tmax;
        } else if (tmax > m_ref + LD_RESCALE) {
          al = exp2f(m_ref - tmax);
          m_ref = tmax;
        }
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          shift[i] = __shfl_sync(0xffffffffu, m_ref, (lane & 16) + i);
          l[i] *= __shfl_sync(0xffffffffu, al, (lane & 16) + i);
        }
        if (n > 0) {
          if (quad == 0) alpha_sm[lane] = al;
          softmax_sync();
          if (__all_sync(0xffffffffu, mbar_wait(&pv_done[(n - 1) & 1], parity2(n - 1), abort_flag, a.status, 1121))) {
            tc_fence_after_sync();
#pragma unroll 1
            for (int c = 0; c < 2 * a.blocks; ++c) {
              uint32_t v[32];
              tmem_ld_32x32(to + c * 32, v);
              tmem_wait_ld();
#pragma unroll
              for (int i = 0; i < 32; ++i) v[i] = __float_as_uint(__uint_as_float(v[i]) * alpha_sm[i]);
              tmem_st_32x32(to + c * 32, v);
            }
            tmem_wait_st();
          }
        }
        softmax_sync();                               // the exchange buffers may be written again
      }
      // the buffer of this tile's weights is free once the tile before the last has been multiplied
      if (n >= 2) mbar_wait(&pv_done[n & 1], parity2(n - 2), abort_flag, a.status, 1122);
      uint8_t* prow = p_sm + (n & 1) * LD_P_BYTES + key * 128;
      const int chunk0 = lane >> 4 << 1, sw = key & 7;
#pragma unroll
      for (int c = 0; c < 2; ++c) {                   // 8 heads: 16 bytes of leading parts, 16 of remainders
        uint32_t head[4], rest[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          const int i = c * 8 + 2 * e;
          const float p0 = exp2f(fmaf(x[i], scale, -shift[i])), p1 = exp2f(fmaf(x[i + 1], scale, -shift[i + 1]));
          l[i] += p0;
          l[i + 1] += p1;
          // leading part: the upper 16 bits as they are; the remainder is exact in fp32 and rounded to bf16
          const uint32_t w0 = __float_as_uint(p0), w1 = __float_as_uint(p1);
          head[e] = __byte_perm(w0, w1, 0x7632);
          rest[e] = pack_bf16x2(p0 - __uint_as_float(w0 & 0xffff0000u), p1 - __uint_as_float(w1 & 0xffff0000u));
        }
        *reinterpret_cast<uint4*>(prow + (((chunk0 + c) ^ sw) << 4)) = make_uint4(head[0], head[1], head[2], head[3]);
        *reinterpret_cast<uint4*>(prow + (((4 + chunk0 + c) ^ sw) << 4)) = make_uint4(rest[0], rest[1], rest[2], rest[3]);
      }
      fence_proxy_async_smem();
      tc_fence_before_sync();
      __syncwarp();
      if (lane == 0) mbar_arrive(&p_full[n & 1]);
    }
    // sums of all keys, and every head's factor (or what the merge needs)
    warp_part[quad][lane] = half_warp_transpose<false>(l, lane);
    softmax_sync();
    if (quad == 0) {
      const float sum = (warp_part[0][lane] + warp_part[1][lane]) + (warp_part[2][lane] + warp_part[3][lane]);
      float f = 1.f;
      if (a.nsplit == 1) {
        const float sl = a.sink != nullptr && lane < nh ? a.sink[h0 + lane] * 1.4426950408889634f : -INFINITY;
        const float nm = fmaxf(m_ref, sl);
        const float w = m_ref == -INFINITY ? 0.f : exp2f(m_ref - nm);
        const float gl = sum * w + (sl == -INFINITY ? 0.f : exp2f(sl - nm));
        f = gl > 0.f ? w / gl : 0.f;
      } else if (lane < nh) {
        float2* ml = reinterpret_cast<float2*>(a.partial + a.ml_offset);
        ml[(static_cast<size_t>(row) * a.H + h0 + lane) * a.nsplit + split] = make_float2(m_ref, sum);
      }
      alpha_sm[lane] = f;
    }
    softmax_sync();
    const int last = n_tiles - 1;
    const bool have = n_tiles > 0 && __all_sync(0xffffffffu, mbar_wait(&pv_done[last & 1], parity2(last), abort_flag, a.status, 1123));
    tc_fence_after_sync();
    if (have || (n_tiles <= 0 && a.nsplit == 1)) {
      const size_t at = static_cast<size_t>(row) * a.H + h0;
      const size_t pitch = static_cast<size_t>(a.nsplit) * a.rank_p;           // partial sums: head to head
#pragma unroll 1
      for (int blk = 0; blk < a.blocks; ++blk) {
        uint32_t v[32], u[32];
        if (have) {
          tmem_ld_32x32(to + blk * (2 * LD_HEADS), v);
          tmem_ld_32x32(to + blk * (2 * LD_HEADS) + LD_HEADS, u);
          tmem_wait_ld();
        }
        const int d = blk * 128 + quad * 32 + lane;
        if (d >= a.rank_p) continue;
        if (a.nsplit == 1) {
          __nv_bfloat16* o = a.out + at * a.rank_p + d;
#pragma unroll
          for (int h = 0; h < LD_HEADS; ++h)
            if (h < nh) o[h * a.rank_p] = __float2bfloat16(have ? (__uint_as_float(v[h]) + __uint_as_float(u[h])) * alpha_sm[h] : 0.f);
        } else {
          float* o = a.partial + at * pitch + static_cast<size_t>(split) * a.rank_p + d;
#pragma unroll
          for (int h = 0; h < LD_HEADS; ++h) {
            if (h < nh) *o = __uint_as_float(v[h]) + __uint_as_float(u[h]);
            o += pitch;
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
    tmem_dealloc(tmem, a.tmem_cols);
  }
}

// One CTA per (row, head): adds up the splits. A split without keys left its sums unwritten; its maximum says so.
__global__ void __launch_bounds__(128)
latent_merge_kernel(const float* __restrict__ partial, const float2* __restrict__ ml, const float* __restrict__ sink, __nv_bfloat16* __restrict__ out,
                    int H, int rank_p, int nsplit) {
  griddep_launch();
  griddep_wait();
  const size_t at = blockIdx.x;
  const float sl = sink != nullptr ? sink[blockIdx.x % H] * 1.4426950408889634f : -INFINITY;
  const float2* w = ml + at * nsplit;
  float gm = sl;
  for (int s = 0; s < nsplit; ++s) gm = fmaxf(gm, w[s].x);
  float gl = sl == -INFINITY ? 0.f : exp2f(sl - gm);
  for (int s = 0; s < nsplit; ++s) gl += w[s].x == -INFINITY ? 0.f : w[s].y * exp2f(w[s].x - gm);
  const float inv = gl > 0.f ? 1.f / gl : 0.f;
  for (int d = threadIdx.x * 4; d < rank_p; d += 512) {
    float4 r = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
    for (int s = 0; s < nsplit; ++s) {
      const float2 m = w[s];
      if (m.x == -INFINITY) continue;
      const float f = exp2f(m.x - gm) * inv;
      const float4 v = load4(partial + (at * nsplit + s) * rank_p + d);
      r.x = fmaf(v.x, f, r.x); r.y = fmaf(v.y, f, r.y); r.z = fmaf(v.z, f, r.z); r.w = fmaf(v.w, f, r.w);
    }
    store4(out + at * rank_p + d, r);
  }
}

int make_tmap_bf16_2d(CUtensorMap* out, const void* ptr, uint64_t inner, uint64_t outer, uint64_t ld, uint32_t box_inner,
                      uint32_t box_outer);

// Shape of a launch for latents of `rank_p` and rows of `W` elements.
struct LatentShape {
  int atoms, blocks, stage_atoms, stages, tmem_cols, smem, ctas_per_sm;
};

static bool latent_shape(int rank_p, int W, LatentShape* s) {
  s->atoms = (W + 63) / 64;
  s->blocks = (rank_p + 127) / 128;
  if (s->atoms > LD_MAX_ATOMS || s->blocks > LD_MAX_BLOCKS) return false;
  s->stage_atoms = s->atoms > 2 * s->blocks ? s->atoms : 2 * s->blocks;      // the second product reads whole blocks of 128 dimensions
  const int fixed = s->atoms * LD_Q_ATOM + 2 * LD_P_BYTES + 1024 + 256;
  const int stage = s->stage_atoms * LD_ATOM;
  int st = (112 * 1024 - fixed) / stage;                                      // two CTAs per SM if two stages fit that way
  s->ctas_per_sm = st >= 2 ? 2 : 1;
  if (st < 2) st = (226 * 1024 - fixed) / stage;
  if (st < 2) return false;
  s->stages = st > 4 ? 4 : st;
  s->tmem_cols = 128;
  while (s->tmem_cols < 2 * LD_HEADS + s->blocks * 2 * LD_HEADS) s->tmem_cols *= 2;
  if (s->tmem_cols == 512) s->ctas_per_sm = 1;
  s->smem = fixed + s->stages * stage;
  return true;
}

}  // namespace rpeg

using namespace rpeg;

// CTAs that share an SM, 0 if these sizes are not covered.
extern "C" int rpeg_latent_decode_ctas(int rank_p, int W) {
  LatentShape s;
  return latent_shape(rank_p, W, &s) ? s.ctas_per_sm : 0;
}

// floats of scratch for `rows` rows of H heads split `nsplit` ways
extern "C" long long rpeg_latent_decode_scratch(int rows, int H, int rank_p, int nsplit) {
  return nsplit > 1 ? static_cast<long long>(rows) * H * nsplit * (rank_p + 2) : 0;
}

extern "C" int rpeg_latent_decode(const void* q, const void* cache, long long num_pages, const int* page_table, int max_pages, const int* slot,
                                  const int* pos, const int* lens, const float* sink, void* out, float* scratch, int rows, int H, int rank_p,
                                  int W, int window, int nsplit, float scale, int* status, void* stream) {
  if (rows <= 0) return 0;
  if (((rank_p | W) & 7) || rank_p < 8 || W < rank_p || H < 1 || window < 0 || nsplit < 1 || nsplit > 64 || !(scale > 0.f)) return -2;
  LatentShape s;
  if (!latent_shape(rank_p, W, &s)) return -3;
  if (nsplit > 1 && scratch == nullptr) return -6;
  if (static_cast<long long>(rows) * H > 0x7fffffffll) return -2;
  if ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(cache) | reinterpret_cast<uintptr_t>(out) | reinterpret_cast<uintptr_t>(scratch)) & 15)
    return -1;
  CUtensorMap tq, tc;
  int rc = make_tmap_bf16_2d(&tq, q, W, static_cast<uint64_t>(rows) * H, W, 64, LD_HEADS);
  if (rc) return rc;
  rc = make_tmap_bf16_2d(&tc, cache, W, static_cast<uint64_t>(num_pages) * LD_PAGE, W, 64, LD_PAGE);
  if (rc) return rc - 100;
  static int configured = 0;
  if (s.smem > configured) {
    if (cudaFuncSetAttribute(latent_decode_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, s.smem) != cudaSuccess) return -20;
    configured = s.smem;
  }
  const long long ml = static_cast<long long>(rows) * H * nsplit * rank_p;
  const LatentDecode a{page_table, max_pages, slot, pos, lens, sink, static_cast<__nv_bfloat16*>(out), scratch, ml, H, rank_p, s.atoms,
                       s.stage_atoms, s.blocks, window, nsplit, s.stages, s.tmem_cols, scale * 1.4426950408889634f, status};
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  if (launch_pdl(latent_decode_kernel, dim3(rows, (H + LD_HEADS - 1) / LD_HEADS, nsplit), dim3(LD_THREADS), static_cast<size_t>(s.smem), st, tq, tc,
                 a) != cudaSuccess)
    return -21;
  if (nsplit == 1) return 0;
  return launch_pdl(latent_merge_kernel, dim3(static_cast<unsigned>(rows) * H), dim3(128), 0, st, static_cast<const float*>(scratch),
                    reinterpret_cast<const float2*>(scratch + ml), sink, static_cast<__nv_bfloat16*>(out), H, rank_p, nsplit) == cudaSuccess ? 0 : -22;
}
