// RMS norms around a residual stream that is kept in fp32.
//
// One kernel covers the places where such a decoder touches the stream, so each is a single launch:
//   embedding    x  = norm(table[id])
//   after a sublayer (norm on the sublayer's OUTPUT)
//                x += norm(sublayer output)
//   before the logits
//                y  = norm(x)
// and the last one can ride on the layer before it (`w2`). The value that is normalised comes from one of five sources:
// a bf16 / fp32 activation, the split-K partials of the GEMM that produced it (summed here), the rows of a mixture of
// experts (weighted and summed here, see moe.cu), an embedding table, or the stream itself. Every sum and every norm
// is fp32; the stream is written back in fp32 together with its bf16 copy, the next GEMM's operand.
//
// Weights are stored either as they are applied or as the difference from one (`w_add` is 0 or 1).
// One CTA per row; the row lives in shared memory between the passes. Rows are padded to a multiple of 8 columns
// (`dp`); the padding holds zeros and stays zero, the mean is over the true width `d`.
#include "act_io.cuh"
#include "rpeg_kernels.h"

namespace rpeg {

enum { NSRC_ACT = 0, NSRC_PARTIALS = 1, NSRC_MOE = 2, NSRC_EMBED = 3, NSRC_STREAM = 4 };

struct NormSource {
  const void* p;            // activation / partials / expert rows / table / stream
  int splits;               // partials: how many, `stride` floats apart
  long long stride;
  int ld;                   // row pitch in elements
  const int* idx;           // token ids, or the expert-output row of every (token, choice)
  const float* wts;         // weight of every (token, choice)
  int top, n_shared;        // choices per token; always-on experts: rows shared_row0 + s * rows + t, weight 1
  long long shared_row0;
};

template <typename T, int SRC>
__device__ __forceinline__ float4 norm_source(const NormSource& s, int row, int rows, int c) {
  if constexpr (SRC == NSRC_PARTIALS) {
    const float* p = static_cast<const float*>(s.p) + static_cast<size_t>(row) * s.ld + c;
    float4 v = load4(p);
#pragma unroll 4
    for (int k = 1; k < s.splits; ++k) v = add4(v, load4(p + k * s.stride));
    return v;
  } else if constexpr (SRC == NSRC_MOE) {
    const T* y = static_cast<const T*>(s.p) + c;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 4
    for (int k = 0; k < s.top; ++k) {
      const float w = s.wts[static_cast<size_t>(row) * s.top + k];
      const float4 e = load4(y + static_cast<size_t>(s.idx[static_cast<size_t>(row) * s.top + k]) * s.ld);
      v.x = fmaf(w, e.x, v.x); v.y = fmaf(w, e.y, v.y); v.z = fmaf(w, e.z, v.z); v.w = fmaf(w, e.w, v.w);
    }
    for (int k = 0; k < s.n_shared; ++k)
      v = add4(v, load4(y + static_cast<size_t>(s.shared_row0 + static_cast<long long>(k) * rows + row) * s.ld));
    return v;
  } else if constexpr (SRC == NSRC_EMBED) {
    return load4(static_cast<const T*>(s.p) + static_cast<size_t>(s.idx[row]) * s.ld + c);
  } else if constexpr (SRC == NSRC_STREAM) {
    return load4(static_cast<const float*>(s.p) + static_cast<size_t>(row) * s.ld + c);
  } else {
    return load4(static_cast<const T*>(s.p) + static_cast<size_t>(row) * s.ld + c);
  }
}

__device__ __forceinline__ float block_sum(float v, float* part) {
  v = warp_sum(v);
  const int nw = (blockDim.x + 31) >> 5;
  if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = v;
  __syncthreads();
  float t = 0.f;
  for (int i = 0; i < nw; ++i) t += part[i];
  return t;
}

template <typename T, int SRC>
__global__ void __launch_bounds__(256)
residual_norm_kernel(const NormSource src, const T* __restrict__ w, const T* __restrict__ w2, float* x, T* __restrict__ y,
                     int rows, int d, int dp, float eps, float w_add, int add) {
  griddep_launch();
  griddep_wait();   // may have been scheduled under the previous kernel's tail: nothing is read or written before this
  extern __shared__ float rowbuf[];
  __shared__ float part[2][8];
  const int row = blockIdx.x;
  float ss = 0.f;
  for (int c = threadIdx.x * 4; c < dp; c += blockDim.x * 4) {
    const float4 v = norm_source<T, SRC>(src, row, rows, c);
    store4(rowbuf + c, v);
    ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
  }
  const float r = rsqrtf(block_sum(ss, part[0]) / static_cast<float>(d) + eps);
  float ss2 = 0.f;
  float* xr = x == nullptr ? nullptr : x + static_cast<size_t>(row) * dp;
  T* yr = y == nullptr ? nullptr : y + static_cast<size_t>(row) * dp;
  // a thread re-reads only the columns it wrote itself, so no barrier is needed between the passes
  for (int c = threadIdx.x * 4; c < dp; c += blockDim.x * 4) {
    const float4 v = load4(rowbuf + c), g = load4(w + c);
    float4 o = make_float4(v.x * r * (w_add + g.x), v.y * r * (w_add + g.y), v.z * r * (w_add + g.z), v.w * r * (w_add + g.w));
    if (add) o = add4(o, load4(xr + c));
    if (xr != nullptr) store4(xr + c, o);
    if (w2 != nullptr) {
      store4(rowbuf + c, o);
      ss2 += o.x * o.x + o.y * o.y + o.z * o.z + o.w * o.w;
    } else if (yr != nullptr) {
      store4(yr + c, o);
    }
  }
  if (w2 != nullptr) {
    const float r2 = rsqrtf(block_sum(ss2, part[1]) / static_cast<float>(d) + eps);
    for (int c = threadIdx.x * 4; c < dp; c += blockDim.x * 4) {
      const float4 v = load4(rowbuf + c), g = load4(w2 + c);
      store4(yr + c, make_float4(v.x * r2 * (w_add + g.x), v.y * r2 * (w_add + g.y), v.z * r2 * (w_add + g.z), v.w * r2 * (w_add + g.w)));
    }
  }
}

template <typename T>
static int launch_residual_norm(int kind, const NormSource& src, const void* w, const void* w2, float* x, void* y, int rows, int d,
                                int dp, float eps, float w_add, int add, cudaStream_t stream) {
  int threads = (dp / 4 + 31) / 32 * 32;
  if (threads > 256) threads = 256;
  const size_t smem = static_cast<size_t>(dp) * 4;
#define RPEG_NORM_CASE(S)                                                                                                     \
  case S: {                                                                                                                   \
    auto kern = residual_norm_kernel<T, S>;                                                                                   \
    if (smem > 48 * 1024 &&                                                                                                   \
        cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)) != cudaSuccess)       \
      return -20;                                                                                                             \
    const cudaError_t e = launch_pdl(kern, dim3(rows), dim3(threads), smem, stream, src, static_cast<const T*>(w),            \
                                     static_cast<const T*>(w2), x, static_cast<T*>(y), rows, d, dp, eps, w_add, add);         \
    return e == cudaSuccess ? 0 : -21;                                                                                        \
  }
  switch (kind) {
    RPEG_NORM_CASE(NSRC_ACT)
    RPEG_NORM_CASE(NSRC_PARTIALS)
    RPEG_NORM_CASE(NSRC_MOE)
    RPEG_NORM_CASE(NSRC_EMBED)
    RPEG_NORM_CASE(NSRC_STREAM)
    default:
      return -4;
  }
#undef RPEG_NORM_CASE
}

}  // namespace rpeg

using namespace rpeg;

extern "C" int rpeg_residual_norm(int kind, const void* src, int splits, long long stride, int ld, const int* idx, const float* wts,
                                  int top, int n_shared, long long shared_row0, const void* w, const void* w2, float* x, void* y,
                                  int rows, int d, int dp, float eps, float w_add, int add, int f32, void* stream) {
  if (rows <= 0) return 0;
  if ((dp & 7) || d > dp || d < 1 || (ld & 3) || dp > 50000) return -2;
  if ((add && x == nullptr) || (w2 != nullptr && y == nullptr)) return -3;
  const NormSource s{src, splits, stride, ld, idx, wts, top, n_shared, shared_row0};
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  return f32 ? launch_residual_norm<float>(kind, s, w, w2, x, y, rows, d, dp, eps, w_add, add, st)
             : launch_residual_norm<__nv_bfloat16>(kind, s, w, w2, x, y, rows, d, dp, eps, w_add, add, st);
}
