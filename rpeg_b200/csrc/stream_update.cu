// The residual stream of decoders whose sublayers run side by side on one normalised input and whose norm is elementwise:
//
//   x += mixer output + feed-forward output            (fp32 stream; or x = embedding row)
//   y  = tanh(alpha * x) * w + b                       (the next layer's operand, or the logits')
//
// in one launch per layer. Each of the two outputs comes as an activation, as split-K partials or as the rows of a mixture of experts
// and is summed here. Nothing is reduced over a row, so a row is spread over as many CTAs as it has runs of 4 * SU_THREADS columns.
// Rows are padded to a multiple of 8 columns; the padding of every source, of w and of b is zero, so that of x and y is.
#include "stream_source.cuh"
#include "rpeg_kernels.h"

namespace rpeg {

constexpr int SU_THREADS = 128;
enum { SU_NONE = -1 };

template <typename T, int SRC_A, int SRC_B>
__global__ void __launch_bounds__(SU_THREADS)
stream_update_kernel(const NormSource a, const NormSource b, const float* __restrict__ alpha, const T* __restrict__ w,
                     const T* __restrict__ bias, float* __restrict__ x, T* __restrict__ y, int rows, int dp) {
  griddep_launch();
  extern __shared__ int choice_row[];
  float* choice_w = reinterpret_cast<float*>(choice_row + b.top + b.n_shared);
  const int row = blockIdx.x, c = (blockIdx.y * SU_THREADS + threadIdx.x) * 4;
  const bool live = c < dp;
  const float s = *alpha;                          // weights do not depend on the kernel before
  const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
  const float4 g = live ? load4(w + c) : zero, o = live ? load4(bias + c) : zero;
  griddep_wait();
  if constexpr (SRC_B == NSRC_MOE) {
    for (int k = threadIdx.x; k < b.top + b.n_shared; k += SU_THREADS) {
      const bool routed = k < b.top;
      choice_row[k] = routed ? b.idx[static_cast<size_t>(row) * b.top + k]
                             : static_cast<int>(b.shared_row0 + static_cast<long long>(k - b.top) * rows + row);
      choice_w[k] = routed && b.wts != nullptr ? b.wts[static_cast<size_t>(row) * b.top + k] : 1.f;
    }
    __syncthreads();
  }
  if (!live) return;
  float* xr = x + static_cast<size_t>(row) * dp + c;
  float4 v = norm_source<T, SRC_A>(a, nullptr, nullptr, row, rows, c);
  if constexpr (SRC_B != SU_NONE) v = add4(v, norm_source<T, SRC_B>(b, choice_row, choice_w, row, rows, c));
  if constexpr (SRC_A != NSRC_EMBED) v = add4(load4(xr), v);
  store4(xr, v);
  store4(y + static_cast<size_t>(row) * dp + c,
         make_float4(fmaf(tanh_f32(s * v.x), g.x, o.x), fmaf(tanh_f32(s * v.y), g.y, o.y), fmaf(tanh_f32(s * v.z), g.z, o.z),
                     fmaf(tanh_f32(s * v.w), g.w, o.w)));
}

template <typename T, int SRC_A, int SRC_B>
static int launch_stream_update(const NormSource& a, const NormSource& b, const float* alpha, const void* w, const void* bias, float* x, void* y,
                                int rows, int dp, cudaStream_t stream) {
  const dim3 grid(rows, (dp / 4 + SU_THREADS - 1) / SU_THREADS);
  const size_t smem = static_cast<size_t>(b.top + b.n_shared) * 8;
  if (grid.y > 65535u || smem > 48 * 1024) return -2;
  return launch_pdl(stream_update_kernel<T, SRC_A, SRC_B>, grid, dim3(SU_THREADS), smem, stream, a, b, alpha, static_cast<const T*>(w),
                    static_cast<const T*>(bias), x, static_cast<T*>(y), rows, dp) == cudaSuccess ? 0 : -21;
}

}  // namespace rpeg

using namespace rpeg;

// Source kinds as in stream_source.cuh; kind_b -1: one source only. `splits`, `stride` and `ld` are the sources' own.
extern "C" int rpeg_stream_update(int kind_a, const void* a, int splits_a, long long stride_a, int ld_a, const int* ids, int kind_b,
                                  const void* b, int splits_b, long long stride_b, int ld_b, const int* row_of, const float* wts, int top,
                                  int n_shared, long long shared_row0, const float* alpha, const void* w, const void* bias, float* x, void* y,
                                  int rows, int dp, int f32, void* stream) {
  if (rows <= 0) return 0;
  if ((dp & 7) || dp < 8 || (ld_a & 3) || (ld_b & 3) || top < 0 || n_shared < 0) return -2;
  if (kind_b == NSRC_MOE && shared_row0 + static_cast<long long>(n_shared) * rows > 0x7fffffffll) return -2;
  if (x == nullptr || y == nullptr || alpha == nullptr) return -3;
  const NormSource sa{a, splits_a, stride_a, ld_a, ids, nullptr, 0, 0, 0};
  const NormSource sb{b, splits_b, stride_b, ld_b, row_of, wts, top, n_shared, shared_row0};
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
#define RPEG_SU(A_, B_)                                                                                             \
  if (kind_a == A_ && kind_b == B_)                                                                                 \
    return f32 ? launch_stream_update<float, A_, B_>(sa, sb, alpha, w, bias, x, y, rows, dp, st)                    \
               : launch_stream_update<__nv_bfloat16, A_, B_>(sa, sb, alpha, w, bias, x, y, rows, dp, st);
  RPEG_SU(NSRC_EMBED, SU_NONE)
  RPEG_SU(NSRC_ACT, SU_NONE)
  RPEG_SU(NSRC_ACT, NSRC_ACT)
  RPEG_SU(NSRC_ACT, NSRC_MOE)
  RPEG_SU(NSRC_PARTIALS, SU_NONE)
  RPEG_SU(NSRC_PARTIALS, NSRC_PARTIALS)
  RPEG_SU(NSRC_PARTIALS, NSRC_MOE)
#undef RPEG_SU
  return -4;
}
