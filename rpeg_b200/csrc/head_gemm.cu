// The same product for every head, each head with its own weight matrix (bf16, fp32 accumulation on tcgen05):
//
//   C[r, h, 0..N) = A[r, h, 0..K) * B_h          A, C: row pitch and head pitch are arguments
//
// B_h is stored [N, K] or (b_kn) [K, N]; the latter reads a matrix that the forward direction stores as [out, in] through its
// transpose, so a query goes back through the very key map the prompt's keys came from.
// One CTA per (column tile x 128-row tile, head): a TMA warp, an MMA warp, four epilogue warps. The maps are 3-D, so columns
// past K or N and rows of another head are never mixed in (out-of-bounds elements read as zero).
#include "common.cuh"
#include "rpeg_kernels.h"

namespace rpeg {

constexpr int HG_BM = 128, HG_BK = 64, HG_THREADS = 192;

template <int BN>
struct HeadGemmCfg {
  static constexpr int A_BYTES = HG_BM * HG_BK * 2;
  static constexpr int B_BYTES = BN * HG_BK * 2;
  static constexpr int STAGE_BYTES = A_BYTES + B_BYTES;
  static constexpr int MAX_STAGES = BN == 64 ? 8 : 6;     // as many as K has blocks, up to this: short ones leave room for more CTAs per SM
  static constexpr int smem_bytes(int stages) { return stages * STAGE_BYTES + 1024 + 256; }
};

template <int BN, bool B_KN>
__global__ void __launch_bounds__(HG_THREADS)
head_gemm_kernel(const __grid_constant__ CUtensorMap tmap_a, const __grid_constant__ CUtensorMap tmap_b, __nv_bfloat16* __restrict__ C, int M,
                 int N, int K, int ldc, int hsc, int a_rows, int stages, int* status) {
  using Cfg = HeadGemmCfg<BN>;
  extern __shared__ uint8_t smem_raw[];
  uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~uintptr_t(1023));
  uint64_t* full_bar = reinterpret_cast<uint64_t*>(smem + stages * Cfg::STAGE_BYTES);
  uint64_t* empty_bar = full_bar + stages;
  uint64_t* done_bar = empty_bar + stages;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(done_bar + 1);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  const int warp = uniform_warp(), lane = threadIdx.x & 31;
  const int n_tiles = (N + BN - 1) / BN;
  const int n0 = (blockIdx.x % n_tiles) * BN, m0 = (blockIdx.x / n_tiles) * HG_BM, h = blockIdx.y;
  const int num_kb = (K + HG_BK - 1) / HG_BK;
  if (threadIdx.x == 0) {
    for (int s = 0; s < stages; ++s) { mbar_init(&full_bar[s], 1); mbar_init(&empty_bar[s], 1); }
    mbar_init(done_bar, 1);
    *abort_flag = 0;
    fence_mbar_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, BN);
    tmem_relinquish();
  }
  tc_fence_before_sync();
  __syncthreads();
  tc_fence_after_sync();
  const uint32_t tmem = *tmem_slot;
  griddep_launch();
  if (warp == 0) {
    if (lane == 0) {
      auto load_b = [&](int kb, int st) {
        uint8_t* sb = smem + st * Cfg::STAGE_BYTES + Cfg::A_BYTES;
        mbar_expect_tx(&full_bar[st], static_cast<uint32_t>(Cfg::B_BYTES + a_rows * HG_BK * 2));
        if constexpr (B_KN) {
#pragma unroll
          for (int c = 0; c < BN / 64; ++c) tma_load_3d(sb + c * (64 * HG_BK * 2), &tmap_b, &full_bar[st], n0 + c * 64, kb * HG_BK, h);
        } else {
          tma_load_3d(sb, &tmap_b, &full_bar[st], kb * HG_BK, n0, h);
        }
      };
      for (int kb = 0; kb < stages; ++kb) load_b(kb, kb);      // weights do not depend on the kernel before
      griddep_wait();
      for (int kb = 0; kb < stages; ++kb) tma_load_3d(smem + kb * Cfg::STAGE_BYTES, &tmap_a, &full_bar[kb], kb * HG_BK, h, m0);
      int st = 0;
      uint32_t phase = 0u;
      for (int kb = stages; kb < num_kb; ++kb) {
        if (!mbar_wait(&empty_bar[st], phase, abort_flag, status, 1000)) break;
        load_b(kb, st);
        tma_load_3d(smem + st * Cfg::STAGE_BYTES, &tmap_a, &full_bar[st], kb * HG_BK, h, m0);
        if (++st == stages) { st = 0; phase ^= 1u; }
      }
    }
  } else if (warp == 1) {
    const bool leader = elect_one();               // all lanes run the loop, one issues
    constexpr uint32_t idesc = make_idesc_bf16(HG_BM, BN, 0, B_KN ? 1 : 0);
    bool ok = true;
    int st = 0;
    uint32_t phase = 0u;
    for (int kb = 0; kb < num_kb; ++kb) {
      if (!__all_sync(0xffffffffu, mbar_wait(&full_bar[st], phase, abort_flag, status, 1010))) { ok = false; break; }
      tc_fence_after_sync();
      const uint32_t sa = smem_u32(smem + st * Cfg::STAGE_BYTES), sb = sa + Cfg::A_BYTES;
#pragma unroll
      for (int k = 0; k < HG_BK / 16; ++k)
        if (leader)
          umma_bf16_ss(tmem, make_smem_desc_sw128(sa + k * 32, 16, 1024),
                       B_KN ? make_smem_desc_sw128(sb + k * 2048, 64 * HG_BK * 2, 1024) : make_smem_desc_sw128(sb + k * 32, 16, 1024), idesc,
                       (kb | k) != 0 ? 1u : 0u);
      if (leader) umma_commit(&empty_bar[st]);
      if (++st == stages) { st = 0; phase ^= 1u; }
    }
    if (ok && leader) umma_commit(done_bar);
  } else {
    const int quad = warp & 3, r = m0 + quad * 32 + lane;
    if (__all_sync(0xffffffffu, mbar_wait(done_bar, 0, abort_flag, status, 1020)) && m0 + quad * 32 < M) {
      tc_fence_after_sync();
      // the buffer may still be read by the kernel before the one this launch depends on: write only behind the wait
      griddep_wait();
      __nv_bfloat16* crow = C + static_cast<size_t>(r) * ldc + static_cast<size_t>(h) * hsc;
#pragma unroll 1
      for (int c = 0; c < BN / 32; ++c) {
        const int col0 = n0 + c * 32;
        if (col0 >= N) break;
        uint32_t v[32];
        tmem_ld_32x32(tmem + (static_cast<uint32_t>(quad * 32) << 16) + c * 32, v);
        tmem_wait_ld();
        if (r < M) {
#pragma unroll
          for (int q = 0; q < 4; ++q)
            if (col0 + q * 8 < N) {
              uint32_t o[4];
#pragma unroll
              for (int e = 0; e < 4; ++e) o[e] = pack_bf16x2(__uint_as_float(v[q * 8 + 2 * e]), __uint_as_float(v[q * 8 + 2 * e + 1]));
              *reinterpret_cast<uint4*>(crow + col0 + q * 8) = make_uint4(o[0], o[1], o[2], o[3]);
            }
        }
      }
    }
  }
  __syncwarp();
  if (*abort_flag) __nanosleep(200000);
  griddep_wait();
  tc_fence_before_sync();
  __syncthreads();
  if (warp == 1) {
    tc_fence_after_sync();
    tmem_dealloc(tmem, BN);
  }
}

int make_tmap_bf16_3d(CUtensorMap* out, const void* ptr, uint64_t d0, uint64_t d1, uint64_t d2, uint64_t ld1, uint64_t ld2, uint32_t b0,
                      uint32_t b1, uint32_t b2);

template <int BN, bool B_KN>
static int launch_head_gemm(const CUtensorMap& ta, const CUtensorMap& tb, void* C, int M, int N, int K, int H, int ldc, int hsc, int a_rows,
                            int* status, cudaStream_t stream) {
  auto kern = head_gemm_kernel<BN, B_KN>;
  using Cfg = HeadGemmCfg<BN>;
  static bool configured = false;
  if (!configured) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, Cfg::smem_bytes(Cfg::MAX_STAGES)) != cudaSuccess) return -20;
    configured = true;
  }
  const long long tiles = static_cast<long long>((N + BN - 1) / BN) * ((M + HG_BM - 1) / HG_BM);
  if (tiles > 0x7fffffffll) return -2;
  const int num_kb = (K + HG_BK - 1) / HG_BK, stages = num_kb < Cfg::MAX_STAGES ? num_kb : Cfg::MAX_STAGES;
  return launch_pdl(kern, dim3(static_cast<unsigned>(tiles), H), dim3(HG_THREADS), static_cast<size_t>(Cfg::smem_bytes(stages)), stream, ta, tb,
                    static_cast<__nv_bfloat16*>(C), M, N, K, ldc, hsc, a_rows, stages, status) == cudaSuccess ? 0 : -21;
}

}  // namespace rpeg

using namespace rpeg;

// A: M rows of `lda` elements, head h at h * hsa; B: H matrices of N x K (b_kn: K x N), contiguous; C like A with ldc, hsc.
extern "C" int rpeg_head_gemm(const void* A, const void* B, void* C, int M, int N, int K, int H, int lda, int hsa, int ldc, int hsc, int b_kn,
                              int* status, void* stream) {
  if (M <= 0 || N <= 0 || K <= 0 || H <= 0) return 0;
  if ((reinterpret_cast<uintptr_t>(A) | reinterpret_cast<uintptr_t>(B) | reinterpret_cast<uintptr_t>(C)) & 15) return -1;
  if (((lda | hsa | ldc | hsc | N | K) & 7) || H > 65535) return -2;
  static int num_sms = 0;
  if (num_sms == 0) {
    int dev = 0;
    cudaGetDevice(&dev);
    cudaDeviceGetAttribute(&num_sms, cudaDevAttrMultiProcessorCount, dev);
  }
  const bool wide = N >= 128 && static_cast<long long>((N + 127) / 128) * ((M + HG_BM - 1) / HG_BM) * H >= num_sms;
  const int a_rows = M <= 32 ? 32 : (M <= 64 ? 64 : HG_BM);
  const int bn = wide ? 128 : 64;
  CUtensorMap ta, tb;
  int rc = make_tmap_bf16_3d(&ta, A, K, H, M, hsa, lda, HG_BK, 1, a_rows);
  if (rc) return rc;
  rc = b_kn ? make_tmap_bf16_3d(&tb, B, N, K, H, N, static_cast<uint64_t>(N) * K, 64, HG_BK, 1)
            : make_tmap_bf16_3d(&tb, B, K, N, H, K, static_cast<uint64_t>(N) * K, HG_BK, bn, 1);
  if (rc) return rc - 100;
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  if (wide) return b_kn ? launch_head_gemm<128, true>(ta, tb, C, M, N, K, H, ldc, hsc, a_rows, status, st)
                        : launch_head_gemm<128, false>(ta, tb, C, M, N, K, H, ldc, hsc, a_rows, status, st);
  return b_kn ? launch_head_gemm<64, true>(ta, tb, C, M, N, K, H, ldc, hsc, a_rows, status, st)
              : launch_head_gemm<64, false>(ta, tb, C, M, N, K, H, ldc, hsc, a_rows, status, st);
}
