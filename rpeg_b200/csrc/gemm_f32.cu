// fp32 matrix products on the CUDA cores (no reduced-precision matrix mode), for models that run in true fp32:
//   C[M,N] = A[M,K] * B[N,K]^T
// plain; grouped: rows of A and C form segments, segment s is multiplied by rows [s * N, s * N + N) of B (the experts of a
// mixture, see moe.cu for the segment layout and the activations); or batched: the same product for every head, at fixed
// strides, with B either [N, K] or [K, N].
// 64 x 64 tile per CTA, 16-deep K slices in shared memory, 4 x 4 outputs per thread.
#include "act_io.cuh"
#include "moe_segments.cuh"
#include "rpeg_kernels.h"

namespace rpeg {

constexpr int SG_T = 64, SG_K = 16;

struct GemmF32 {
  const float *A, *X, *B;
  float* C;
  int M, N, K, lda, ldb, ldc;
  const int* seg_off;                               // grouped
  int n_routed, seg_rows, act;
  long long a_stride, b_stride, c_stride;           // batched: elements between batch members
};

enum { SG_PLAIN = 0, SG_GROUPED = 1, SG_GATED = 2, SG_BATCHED = 3, SG_BATCHED_KN = 4 };   // KN: B is stored [K, N]

template <int MODE>
__global__ void __launch_bounds__(256)
gemm_f32_kernel(const GemmF32 p) {
  constexpr bool GATED = MODE == SG_GATED;
  __shared__ float as[SG_K][SG_T + 4], bs[GATED ? 2 : 1][SG_K][SG_T + 4];
  int M = p.M;
  const float *a = p.A, *B = p.B;
  float* C = p.C;
  if constexpr (MODE == SG_GROUPED || GATED) {
    const MoeSegment sg = moe_segment(p.seg_off, p.n_routed, p.seg_rows, blockIdx.z);
    M = sg.rows;
    B += static_cast<size_t>(blockIdx.z) * p.N * (GATED ? 2 : 1) * p.ldb;
    a = p.X != nullptr && static_cast<int>(blockIdx.z) >= p.n_routed ? p.X : p.A + static_cast<size_t>(sg.row0) * p.lda;
    C += static_cast<size_t>(sg.row0) * p.ldc;
  }
  if constexpr (MODE == SG_BATCHED || MODE == SG_BATCHED_KN) {
    a += blockIdx.z * p.a_stride;
    B += blockIdx.z * p.b_stride;
    C += blockIdx.z * p.c_stride;
  }
  const int m0 = blockIdx.y * SG_T, n0 = blockIdx.x * SG_T;
  if (m0 >= M) return;
  const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  float acc[GATED ? 2 : 1][4][4] = {};
  for (int k0 = 0; k0 < p.K; k0 += SG_K) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int e = tid + i * 256, k = e & 15, r = e >> 4;
      as[k][r] = (m0 + r < M && k0 + k < p.K) ? a[static_cast<size_t>(m0 + r) * p.lda + k0 + k] : 0.f;
      if constexpr (MODE == SG_BATCHED_KN) {
        const int n = e & 63, kk = e >> 6;
        bs[0][kk][n] = (n0 + n < p.N && k0 + kk < p.K) ? B[static_cast<size_t>(k0 + kk) * p.ldb + n0 + n] : 0.f;
      } else {
#pragma unroll
        for (int g = 0; g < (GATED ? 2 : 1); ++g)
          bs[g][k][r] = (n0 + r < p.N && k0 + k < p.K) ? B[(static_cast<size_t>(g) * p.N + n0 + r) * p.ldb + k0 + k] : 0.f;
      }
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < SG_K; ++k) {
      float x[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) x[i] = as[k][ty * 4 + i];
#pragma unroll
      for (int g = 0; g < (GATED ? 2 : 1); ++g) {
        float y[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) y[j] = bs[g][k][tx * 4 + j];
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
          for (int j = 0; j < 4; ++j) acc[g][i][j] = fmaf(x[i], y[j], acc[g][i][j]);
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + ty * 4 + i;
    if (m >= M) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx * 4 + j;
      if (n >= p.N) continue;
      float v = acc[0][i][j];
      if constexpr (GATED) v = silu_mul(v, acc[1][i][j]);
      if constexpr (MODE == SG_GROUPED) v = p.act == FF_GELU ? ff_act<FF_GELU>(v) : (p.act == FF_RELU2 ? ff_act<FF_RELU2>(v) : v);
      C[static_cast<size_t>(m) * p.ldc + n] = v;
    }
  }
}

template <int MODE>
static int launch_gemm_f32(const GemmF32& p, int rows, int batch, void* stream) {
  const dim3 grid((p.N + SG_T - 1) / SG_T, (rows + SG_T - 1) / SG_T, batch);
  if (grid.y > 65535u || grid.z > 65535u) return -2;
  gemm_f32_kernel<MODE><<<grid, 256, 0, reinterpret_cast<cudaStream_t>(stream)>>>(p);
  return cudaGetLastError() == cudaSuccess ? 0 : -21;
}

}  // namespace rpeg

using namespace rpeg;

extern "C" int rpeg_gemm_f32(const float* A, const float* B, float* C, int M, int N, int K, int lda, int ldb, int ldc, void* stream) {
  if (M <= 0 || N <= 0 || K <= 0) return 0;
  return launch_gemm_f32<SG_PLAIN>({A, nullptr, B, C, M, N, K, lda, ldb, ldc, nullptr, 0, 0, FF_NONE, 0, 0, 0}, M, 1, stream);
}

extern "C" int rpeg_moe_gemm_f32(const float* A, const float* X, const float* B, float* C, const int* seg_off, int n_routed, int n_shared,
                                 int seg_rows, int N, int K, int lda, int ldb, int ldc, int act, void* stream) {
  if (seg_rows <= 0 || N <= 0 || K <= 0 || n_routed + n_shared <= 0) return 0;
  if (act < FF_NONE || act > FF_RELU2) return -4;
  const GemmF32 p{A, X, B, C, 0, N, K, lda, ldb, ldc, seg_off, n_routed, seg_rows, act, 0, 0, 0};
  return act == FF_SWIGLU ? launch_gemm_f32<SG_GATED>(p, seg_rows, n_routed + n_shared, stream)
                          : launch_gemm_f32<SG_GROUPED>(p, seg_rows, n_routed + n_shared, stream);
}

// C_h[M, N] = A_h[M, K] * B_h for h = 0 .. batch - 1, each operand `stride` elements after the one before; B_h is [N, K] or (b_kn) [K, N].
extern "C" int rpeg_gemm_f32_batched(const float* A, const float* B, float* C, int M, int N, int K, int lda, int ldb, int ldc, long long a_stride,
                                     long long b_stride, long long c_stride, int batch, int b_kn, void* stream) {
  if (M <= 0 || N <= 0 || K <= 0 || batch <= 0) return 0;
  const GemmF32 p{A, nullptr, B, C, M, N, K, lda, ldb, ldc, nullptr, 0, 0, FF_NONE, a_stride, b_stride, c_stride};
  return b_kn ? launch_gemm_f32<SG_BATCHED_KN>(p, M, batch, stream) : launch_gemm_f32<SG_BATCHED>(p, M, batch, stream);
}
