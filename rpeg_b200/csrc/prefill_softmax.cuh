// The softmax side of the tensor-core prompt attention kernels: a thread owns one query row, whose 128 scores of a key tile lie in TMEM.
#pragma once
#include "act_io.cuh"

namespace rpeg {

constexpr float WP_RESCALE = 8.0f;       // log2: how far a row's maximum may grow before its accumulator is rescaled

// A row's 128 scores of one tile, in registers from the maximum to the weights: S is read from TMEM once.
struct WpRow {
  uint32_t s[4][32];
};

__device__ __forceinline__ void wp_load_row(uint32_t ts, WpRow& row) {
#pragma unroll
  for (int c = 0; c < 4; ++c) tmem_ld_32x32(ts + c * 32, row.s[c]);
  tmem_wait_ld();
}

// Keys outside [lo, hi] of the tile that starts at k0 get no weight, whatever their (finite or not) score is.
__device__ __forceinline__ void wp_mask_row(WpRow& row, int k0, int lo, int hi) {
#pragma unroll
  for (int c = 0; c < 4; ++c)
#pragma unroll
    for (int i = 0; i < 32; ++i) {
      const int kj = k0 + c * 32 + i;
      if (kj < lo || kj > hi) row.s[c][i] = 0xff800000u;
    }
}

__device__ __forceinline__ float wp_max_row(const WpRow& row) {
  float m[4];
#pragma unroll
  for (int c = 0; c < 4; ++c) {
    m[c] = __uint_as_float(row.s[c][0]);
#pragma unroll
    for (int i = 1; i < 32; ++i) m[c] = fmaxf(m[c], __uint_as_float(row.s[c][i]));
  }
  return fmaxf(fmaxf(m[0], m[1]), fmaxf(m[2], m[3]));
}

// P = exp2(s * scale - m_ref) over S in place (columns 32 c .. + 15: leading parts of chunk c, + 16 .. + 31: remainders);
// returns its row sum. `half_bar` gets this warp's arrival once the first 64 keys are in place.
__device__ __forceinline__ float wp_exp_row(const WpRow& row, uint32_t ts, float scale_log2, float m_ref, uint64_t* half_bar) {
  const uint64_t scale2 = pack2(scale_log2, scale_log2), shift2 = pack2(-m_ref, -m_ref), minus2 = pack2(-1.f, -1.f);
  uint64_t sum2[2] = {0ull, 0ull};
#pragma unroll
  for (int c = 0; c < 4; ++c) {
    uint32_t head[16], rest[16];
#pragma unroll
    for (int i = 0; i < 16; ++i) {
      const float2 t = unpack2(fma2(pack2(__uint_as_float(row.s[c][2 * i]), __uint_as_float(row.s[c][2 * i + 1])), scale2, shift2));
      const float p0 = exp2f(t.x), p1 = exp2f(t.y);
      const uint64_t p = pack2(p0, p1);
      sum2[i & 1] = add2(sum2[i & 1], p);
      // leading part: the upper 16 bits as they are; the remainder is exact in fp32 and rounded to bf16
      const uint32_t w0 = __float_as_uint(p0), w1 = __float_as_uint(p1);
      head[i] = __byte_perm(w0, w1, 0x7632);
      const float2 r = unpack2(fma2(pack2(__uint_as_float(w0 & 0xffff0000u), __uint_as_float(w1 & 0xffff0000u)), minus2, p));
      rest[i] = pack_bf16x2(r.x, r.y);
    }
    tmem_st_32x16(ts + c * 32, head);
    tmem_st_32x16(ts + c * 32 + 16, rest);
    if (c == 1) {
      tmem_wait_st();
      tc_fence_before_sync();
      __syncwarp();
      if ((threadIdx.x & 31) == 0) mbar_arrive(half_bar);
    }
  }
  const float2 s0 = unpack2(sum2[0]), s1 = unpack2(sum2[1]);
  return (s0.x + s0.y) + (s1.x + s1.y);
}

}  // namespace rpeg
