// fp32 matrix products on the CUDA cores (no reduced-precision matrix mode), for models that run in true fp32:
//   C[M,N] = A[M,K] * B[N,K]^T
// plain, or grouped: rows of A and C form segments, segment s is multiplied by rows [s * N, s * N + N) of B (the
// experts of a mixture, see moe.cu for the segment layout), optionally followed by gelu.
// 64 x 64 tile per CTA, 16-deep K slices in shared memory, 4 x 4 outputs per thread.
#include "act_io.cuh"
#include "moe_segments.cuh"
#include "rpeg_kernels.h"

namespace rpeg {

constexpr int SG_T = 64, SG_K = 16;

template <bool GROUPED>
__global__ void __launch_bounds__(256)
gemm_f32_kernel(const float* __restrict__ A, const float* __restrict__ X, const float* __restrict__ B, float* __restrict__ C, int M, int N,
                int K, int lda, int ldb, int ldc, int gelu, const int* __restrict__ seg_off, int n_routed, int seg_rows) {
  __shared__ float as[SG_K][SG_T + 4], bs[SG_K][SG_T + 4];
  long long row0 = 0;
  const float* a = A;
  long long a_row0 = 0;
  if constexpr (GROUPED) {
    const MoeSegment sg = moe_segment(seg_off, n_routed, seg_rows, blockIdx.z);
    M = sg.rows;
    row0 = a_row0 = sg.row0;
    B += static_cast<size_t>(blockIdx.z) * N * ldb;
    if (X != nullptr && static_cast<int>(blockIdx.z) >= n_routed) { a = X; a_row0 = 0; }
  }
  const int m0 = blockIdx.y * SG_T, n0 = blockIdx.x * SG_T;
  if (m0 >= M) return;
  const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < K; k0 += SG_K) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int e = tid + i * 256, k = e & 15, r = e >> 4;
      as[k][r] = (m0 + r < M && k0 + k < K) ? a[static_cast<size_t>(a_row0 + m0 + r) * lda + k0 + k] : 0.f;
      bs[k][r] = (n0 + r < N && k0 + k < K) ? B[static_cast<size_t>(n0 + r) * ldb + k0 + k] : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < SG_K; ++k) {
      float x[4], y[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) { x[i] = as[k][ty * 4 + i]; y[i] = bs[k][tx * 4 + i]; }
#pragma unroll
      for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(x[i], y[j], acc[i][j]);
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
      if (n < N) C[static_cast<size_t>(row0 + m) * ldc + n] = gelu ? gelu_erf(acc[i][j]) : acc[i][j];
    }
  }
}

}  // namespace rpeg

using namespace rpeg;

extern "C" int rpeg_gemm_f32(const float* A, const float* B, float* C, int M, int N, int K, int lda, int ldb, int ldc, void* stream) {
  if (M <= 0 || N <= 0 || K <= 0) return 0;
  const dim3 grid((N + SG_T - 1) / SG_T, (M + SG_T - 1) / SG_T, 1);
  if (grid.y > 65535u) return -2;
  gemm_f32_kernel<false><<<grid, 256, 0, reinterpret_cast<cudaStream_t>(stream)>>>(A, nullptr, B, C, M, N, K, lda, ldb, ldc, 0, nullptr, 0, 0);
  return cudaGetLastError() == cudaSuccess ? 0 : -21;
}

extern "C" int rpeg_moe_gemm_f32(const float* A, const float* X, const float* B, float* C, const int* seg_off, int n_routed, int n_shared,
                                 int seg_rows, int N, int K, int lda, int ldb, int ldc, int gelu, void* stream) {
  if (seg_rows <= 0 || N <= 0 || K <= 0 || n_routed + n_shared <= 0) return 0;
  const dim3 grid((N + SG_T - 1) / SG_T, (seg_rows + SG_T - 1) / SG_T, n_routed + n_shared);
  if (grid.y > 65535u || grid.z > 65535u) return -2;
  gemm_f32_kernel<true><<<grid, 256, 0, reinterpret_cast<cudaStream_t>(stream)>>>(A, X, B, C, 0, N, K, lda, ldb, ldc, gelu, seg_off,
                                                                                n_routed, seg_rows);
  return cudaGetLastError() == cudaSuccess ? 0 : -21;
}
