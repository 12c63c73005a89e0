// Latent attention of single query rows on the tensor cores (bf16): up to 32 heads of one row against the cached rows themselves.
//
//   S[head, key]  = q_h . row_key              q_h [W] = (query through the key map | rotated part), row [W] = (latent | rotated part)
//   P             = softmax(S * scale  [visible keys], sink)
//   O^T[d, head]  = sum_key row_key[d] P[head, key]       for the latent's dimensions d < rank
//
// A cached row is read from memory once, for the scores of all heads and for their averages: the tile of 64 keys (one cache page) that
// TMA brings to shared memory is the K-major operand B of the first product and, read along its other axis, the MN-major operand A
// of the second. Roles: a TMA warp, an MMA warp, four warps of which one turns scores into weights (its lanes are the heads) while all
// four rescale and store the accumulator (their lanes are latent dimensions).
//   * Operand A of the first product is 128 rows high and holds 32 heads; the rows below read whatever lies there, and what they give is
//     in TMEM lanes nobody reads.
//   * A weight goes to the tensor cores as the sum of two bf16 numbers (16 bits), so that rounding the operands does not show: rows 0..31
//     of the 64-row operand P are the leading parts, rows 32..63 the remainders, and the two halves of the accumulator are added in the
//     end. Both parts cost one pass.
//   * Scores are double buffered in TMEM, weights in shared memory: the product for the next page runs under the softmax of this one.
//   * The accumulator is rescaled only when some head's maximum grew by more than 8 (log2).
// Splits of a row's pages leave unnormalised partial sums; latent_merge adds them up.
#include "act_io.cuh"
#include "rpeg_kernels.h"

namespace rpeg {

constexpr int LD_PAGE = RPEG_KV_PAGE, LD_HEADS = 32, LD_THREADS = 192;
constexpr int LD_ATOM = LD_PAGE * 128;             // 64 keys x 64 columns, 128-byte swizzled
constexpr int LD_Q_ATOM = LD_HEADS * 128;
constexpr int LD_P_BYTES = 2 * LD_HEADS * 128;     // [leading parts; remainders] x 64 keys
constexpr int LD_MAX_ATOMS = 9, LD_MAX_BLOCKS = 4; // rows of up to 576 elements, latents of up to 512
constexpr float LD_RESCALE = 8.0f;

struct LatentDecode {
  const int* page_table; int max_pages;
  const int* slot; const int* pos; const int* lens;
  const float* sink;
  __nv_bfloat16* out;                              // [rows, H, rank_p]
  float* partial;                                  // [rows, H, nsplit, rank_p], then (max, sum) [rows, H, nsplit]
  long long ml_offset;
  int H, rank_p, ksteps, atoms, stage_atoms, blocks, window, nsplit, stages, tmem_cols;
  float scale_log2;
  int* status;
};

__device__ __forceinline__ void bar_sync_softmax() { asm volatile("bar.sync 1, 128;" ::: "memory"); }

__global__ void __launch_bounds__(LD_THREADS, 2)
latent_decode_kernel(const __grid_constant__ CUtensorMap tmap_q, const __grid_constant__ CUtensorMap tmap_c, const LatentDecode a) {
  extern __shared__ uint8_t smem_raw[];
  __shared__ float alpha_sm[2][LD_HEADS], fac_sm[LD_HEADS];
  __shared__ int flag_sm[2];
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
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    mbar_init(q_full, 1);
    for (int i = 0; i < 2; ++i) { mbar_init(&s_full[i], 1); mbar_init(&p_full[i], 1); mbar_init(&pv_done[i], 1); }
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
  const int pa = min(pg1, pg0 + split * per), n_tiles = min(pg1, pa + per) - pa;

  if (warp == 0) {
    if (lane == 0 && n_tiles > 0) {
      const int* pt = a.page_table + static_cast<size_t>(a.slot[row]) * a.max_pages;
      mbar_expect_tx(q_full, a.atoms * LD_Q_ATOM);
      for (int c = 0; c < a.atoms; ++c) tma_load_2d(q_sm + c * LD_Q_ATOM, &tmap_q, q_full, c * 64, row * a.H + h0);
      for (int j = 0; j < n_tiles; ++j) {
        const int st = j % a.stages;
        if (!mbar_wait(&empty[st], (static_cast<uint32_t>(j / a.stages) & 1u) ^ 1u, abort_flag, a.status, 1100)) break;
        mbar_expect_tx(&full[st], a.atoms * LD_ATOM);
        const int y = pt[pa + j] * LD_PAGE;
        for (int c = 0; c < a.atoms; ++c) tma_load_2d(c_sm + st * stage_bytes + c * LD_ATOM, &tmap_c, &full[st], c * 64, y);
      }
    }
  } else if (warp == 1) {
    if (lane == 0 && n_tiles > 0) {
      constexpr uint32_t idesc_s = make_idesc_bf16(128, LD_PAGE, 0, 0);
      constexpr uint32_t idesc_o = make_idesc_bf16(128, 2 * LD_HEADS, 1, 0);
      auto scores = [&](int j) -> bool {
        const int st = j % a.stages;
        if (!mbar_wait(&full[st], static_cast<uint32_t>(j / a.stages) & 1u, abort_flag, a.status, 1110)) return false;
        tc_fence_after_sync();
        const uint32_t q_addr = smem_u32(q_sm), c_addr = smem_u32(c_sm + st * stage_bytes), ts = tmem + (j & 1) * LD_PAGE;
#pragma unroll 4
        for (int k = 0; k < a.ksteps; ++k) {
          const uint32_t in = static_cast<uint32_t>(k & 3) * 32;
          umma_bf16_ss(ts, make_smem_desc_sw128(q_addr + (k >> 2) * LD_Q_ATOM + in, 16, 1024),
                       make_smem_desc_sw128(c_addr + (k >> 2) * LD_ATOM + in, 16, 1024), idesc_s, k != 0 ? 1u : 0u);
        }
        umma_commit(&s_full[j & 1]);
        return true;
      };
      bool ok = mbar_wait(q_full, 0, abort_flag, a.status, 1111);
      if (ok) ok = scores(0);
      for (int j = 0; j < n_tiles && ok; ++j) {
        if (j + 1 < n_tiles && !scores(j + 1)) break;
        if (!mbar_wait(&p_full[j & 1], static_cast<uint32_t>(j >> 1) & 1u, abort_flag, a.status, 1112)) break;
        tc_fence_after_sync();
        const int st = j % a.stages;
        const uint32_t c_addr = smem_u32(c_sm + st * stage_bytes), p_addr = smem_u32(p_sm + (j & 1) * LD_P_BYTES);
        for (int blk = 0; blk < a.blocks; ++blk)
#pragma unroll
          for (int k = 0; k < LD_PAGE / 16; ++k)       // 16 keys: 16 rows (2 KiB) of every 64-column atom
            umma_bf16_ss(tmem + 2 * LD_PAGE + blk * (2 * LD_HEADS), make_smem_desc_sw128(c_addr + 2 * blk * LD_ATOM + k * 2048, LD_ATOM, 1024),
                         make_smem_desc_sw128(p_addr + k * 32, 16, 1024), idesc_o, (j | k) != 0 ? 1u : 0u);
        umma_commit(&pv_done[j & 1]);
        umma_commit(&empty[st]);
      }
    }
  } else {
    const int quad = warp & 3;
    const bool leader = quad == 0;                  // this warp's TMEM lanes are the heads of S
    const uint32_t lanes = static_cast<uint32_t>(quad * 32) << 16;
    const uint32_t to = tmem + lanes + 2 * LD_PAGE;
    float m_ref = -INFINITY, l = 0.f;
    for (int n = 0; n < n_tiles; ++n) {
      uint32_t s[2][32];
      if (leader) {
        int flag = 0;
        const bool ok = __all_sync(0xffffffffu, mbar_wait(&s_full[n & 1], static_cast<uint32_t>(n >> 1) & 1u, abort_flag, a.status, 1120));
        if (ok) {
          tc_fence_after_sync();
          tmem_ld_32x32(tmem + (n & 1) * LD_PAGE, s[0]);
          tmem_ld_32x32(tmem + (n & 1) * LD_PAGE + 32, s[1]);
          tmem_wait_ld();
          const int k0 = (pa + n) * LD_PAGE;
          const bool edge = k0 < key0 || k0 + LD_PAGE > L;           // uniform
          float mx[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
          for (int i = 0; i < 64; ++i) {
            float v = __uint_as_float(s[i >> 5][i & 31]) * a.scale_log2;
            if (edge && (k0 + i < key0 || k0 + i >= L)) v = -INFINITY;
            s[i >> 5][i & 31] = __float_as_uint(v);
            mx[i & 3] = fmaxf(mx[i & 3], v);
          }
          const float tmax = fmaxf(fmaxf(mx[0], mx[1]), fmaxf(mx[2], mx[3]));
          float al = 1.f;
          if (lane < nh) {
            if (n == 0) {
              m_ref = tmax;
            } else if (tmax > m_ref + LD_RESCALE) {
              al = exp2f(m_ref - tmax);
              m_ref = tmax;
              l *= al;
            }
          }
          alpha_sm[n & 1][lane] = al;
          flag = __any_sync(0xffffffffu, al != 1.f) ? 1 : 0;
        } else {
          flag = 2;
        }
        if (lane == 0) flag_sm[n & 1] = flag;
      }
      bar_sync_softmax();
      const int flag = flag_sm[n & 1];
      if (flag == 2) break;
      if (flag == 1) {
        if (__all_sync(0xffffffffu, mbar_wait(&pv_done[(n - 1) & 1], static_cast<uint32_t>((n - 1) >> 1) & 1u, abort_flag, a.status, 1121))) {
          tc_fence_after_sync();
#pragma unroll 1
          for (int c = 0; c < 2 * a.blocks; ++c) {
            uint32_t v[32];
            tmem_ld_32x32(to + c * 32, v);
            tmem_wait_ld();
#pragma unroll
            for (int i = 0; i < 32; ++i) v[i] = __float_as_uint(__uint_as_float(v[i]) * alpha_sm[n & 1][i]);
            tmem_st_32x32(to + c * 32, v);
          }
          tmem_wait_st();
        }
        tc_fence_before_sync();
        bar_sync_softmax();
      }
      if (leader) {
        // the buffer of this tile's weights is free once the tile before the last has been multiplied
        if (n >= 2 && !__all_sync(0xffffffffu, mbar_wait(&pv_done[n & 1], static_cast<uint32_t>((n - 2) >> 1) & 1u, abort_flag, a.status, 1122))) {
          // give the others their way out at the next tile: this one is never handed on, so no wait behind it can end well
          continue;
        }
        uint8_t* prow = p_sm + (n & 1) * LD_P_BYTES + lane * 128;
        float sum[2] = {0.f, 0.f};
#pragma unroll
        for (int c = 0; c < 8; ++c) {
          uint32_t head[4], rest[4];
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const int i = c * 8 + 2 * e;
            float p0 = exp2f(__uint_as_float(s[i >> 5][i & 31]) - m_ref), p1 = exp2f(__uint_as_float(s[i >> 5][(i & 31) + 1]) - m_ref);
            if (lane >= nh) p0 = p1 = 0.f;
            sum[0] += p0;
            sum[1] += p1;
            const uint32_t w0 = __float_as_uint(p0), w1 = __float_as_uint(p1);
            head[e] = __byte_perm(w0, w1, 0x7632);
            rest[e] = pack_bf16x2(p0 - __uint_as_float(w0 & 0xffff0000u), p1 - __uint_as_float(w1 & 0xffff0000u));
          }
          const int at = (c ^ (lane & 7)) << 4;
          *reinterpret_cast<uint4*>(prow + at) = make_uint4(head[0], head[1], head[2], head[3]);
          *reinterpret_cast<uint4*>(prow + LD_HEADS * 128 + at) = make_uint4(rest[0], rest[1], rest[2], rest[3]);
        }
        l += sum[0] + sum[1];
        fence_proxy_async_smem();
        tc_fence_before_sync();
        __syncwarp();
        if (lane == 0) mbar_arrive(&p_full[n & 1]);
      }
    }
    if (leader) {
      float f = 1.f;
      if (a.nsplit == 1) {
        const float sl = a.sink != nullptr && lane < nh ? a.sink[h0 + lane] * 1.4426950408889634f : -INFINITY;
        const float nm = fmaxf(m_ref, sl);
        const float w = m_ref == -INFINITY ? 0.f : exp2f(m_ref - nm);
        const float gl = l * w + (sl == -INFINITY ? 0.f : exp2f(sl - nm));
        f = gl > 0.f ? w / gl : 0.f;
      } else if (lane < nh) {
        float2* ml = reinterpret_cast<float2*>(a.partial + a.ml_offset);
        ml[(static_cast<size_t>(row) * a.H + h0 + lane) * a.nsplit + split] = make_float2(m_ref, l);
      }
      fac_sm[lane] = f;
    }
    bar_sync_softmax();
    const int last = n_tiles - 1;
    const bool have = n_tiles > 0 &&
                      __all_sync(0xffffffffu, mbar_wait(&pv_done[last & 1], static_cast<uint32_t>(last >> 1) & 1u, abort_flag, a.status, 1123));
    tc_fence_after_sync();
    if (have || (n_tiles <= 0 && a.nsplit == 1)) {
#pragma unroll 1
      for (int blk = 0; blk < a.blocks; ++blk) {
        uint32_t v[32], u[32];
        if (have) {
          tmem_ld_32x32(to + blk * (2 * LD_HEADS), v);
          tmem_ld_32x32(to + blk * (2 * LD_HEADS) + LD_HEADS, u);
          tmem_wait_ld();
        }
        const int d = blk * 128 + quad * 32 + lane;
        if (d < a.rank_p) {
#pragma unroll
          for (int h = 0; h < LD_HEADS; ++h) {
            if (h >= nh) break;
            const float o = have ? __uint_as_float(v[h]) + __uint_as_float(u[h]) : 0.f;
            const size_t at = static_cast<size_t>(row) * a.H + h0 + h;
            if (a.nsplit == 1) a.out[at * a.rank_p + d] = __float2bfloat16(o * fac_sm[h]);
            else a.partial[(at * a.nsplit + split) * a.rank_p + d] = o;
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
  s->tmem_cols = 2 * LD_PAGE + s->blocks * 2 * LD_HEADS <= 256 ? 256 : 512;
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
  if (((rank_p | W) & 7) || rank_p < 8 || W < rank_p || H < 1 || window < 0 || nsplit < 1 || nsplit > 64) return -2;
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
  const LatentDecode a{page_table, max_pages, slot, pos, lens, sink, static_cast<__nv_bfloat16*>(out), scratch, ml, H, rank_p, (W + 15) / 16, s.atoms,
                       s.stage_atoms, s.blocks, window, nsplit, s.stages, s.tmem_cols, scale * 1.4426950408889634f, status};
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  if (launch_pdl(latent_decode_kernel, dim3(rows, (H + LD_HEADS - 1) / LD_HEADS, nsplit), dim3(LD_THREADS), static_cast<size_t>(s.smem), st, tq, tc,
                 a) != cudaSuccess)
    return -21;
  if (nsplit == 1) return 0;
  return launch_pdl(latent_merge_kernel, dim3(static_cast<unsigned>(rows) * H), dim3(128), 0, st, static_cast<const float*>(scratch),
                    reinterpret_cast<const float2*>(scratch + ml), sink, static_cast<__nv_bfloat16*>(out), H, rank_p, nsplit) == cudaSuccess ? 0 : -22;
}
