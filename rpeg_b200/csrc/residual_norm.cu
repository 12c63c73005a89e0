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
// One CTA per row, the row in registers between the passes. Rows are padded to a multiple of 8 columns
// (`dp`); the padding holds zeros and stays zero, the mean is over the true width `d`.
#include "stream_source.cuh"
#include "rpeg_kernels.h"

namespace rpeg {

__device__ __forceinline__ float block_sum(float v, float* part) {
  v = warp_sum(v);
  const int nw = (blockDim.x + 31) >> 5, lane = threadIdx.x & 31;
  if (lane == 0) part[threadIdx.x >> 5] = v;
  __syncthreads();
  return warp_sum(lane < nw ? part[lane] : 0.f);
}

__device__ __forceinline__ float dot4(float4 v) { return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; }
__device__ __forceinline__ float4 weigh4(float4 v, float r, float w_add, float4 g) {
  return make_float4(v.x * r * (w_add + g.x), v.y * r * (w_add + g.y), v.z * r * (w_add + g.z), v.w * r * (w_add + g.w));
}

// NV > 0: a thread keeps NV groups of 4 columns in registers, together with their weights and (for an update) the stream's
// old values, all requested before the first sum. NV = 0: rows of any width, held in shared memory.
template <typename T, int SRC, int NV>
__global__ void __launch_bounds__(NV == 4 ? 512 : 1024)
residual_norm_kernel(const NormSource src, const T* __restrict__ w, const T* __restrict__ w2, float* x, T* __restrict__ y,
                     int rows, int d, int dp, float eps, float w_add, int add) {
  griddep_launch();
  extern __shared__ float rowbuf[];
  __shared__ float part[2][32];
  const int row = blockIdx.x;
  constexpr int NR = NV > 0 ? NV : 1;
  float4 g[NR];
  if constexpr (NV > 0) {                          // weights do not depend on the kernel before
#pragma unroll
    for (int j = 0; j < NV; ++j) {
      const int c = (threadIdx.x + j * blockDim.x) * 4;
      g[j] = c < dp ? load4(w + c) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
  }
  griddep_wait();   // may have been scheduled under the previous kernel's tail: nothing it writes is read before this
  int* choice_row = reinterpret_cast<int*>(rowbuf + (NV > 0 ? 0 : dp));
  float* choice_w = reinterpret_cast<float*>(choice_row + src.top + src.n_shared);
  if constexpr (SRC == NSRC_MOE) {
    for (int k = threadIdx.x; k < src.top + src.n_shared; k += blockDim.x) {
      const bool routed = k < src.top;
      choice_row[k] = routed ? src.idx[static_cast<size_t>(row) * src.top + k]
                             : static_cast<int>(src.shared_row0 + static_cast<long long>(k - src.top) * rows + row);
      choice_w[k] = routed && src.wts != nullptr ? src.wts[static_cast<size_t>(row) * src.top + k] : 1.f;
    }
    __syncthreads();
  }
  float* xr = x == nullptr ? nullptr : x + static_cast<size_t>(row) * dp;
  T* yr = y == nullptr ? nullptr : y + static_cast<size_t>(row) * dp;
  if constexpr (NV > 0) {
    float4 v[NV], old[NV];
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < NV; ++j) {
      const int c = (threadIdx.x + j * blockDim.x) * 4;
      v[j] = old[j] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (c < dp) {
        if (add) old[j] = load4(xr + c);
        v[j] = norm_source<T, SRC>(src, choice_row, choice_w, row, rows, c);
      }
      ss += dot4(v[j]);
    }
    const float r = rsqrtf(block_sum(ss, part[0]) / static_cast<float>(d) + eps);
    float ss2 = 0.f;
#pragma unroll
    for (int j = 0; j < NV; ++j) {
      const int c = (threadIdx.x + j * blockDim.x) * 4;
      if (c >= dp) continue;
      v[j] = add4(weigh4(v[j], r, w_add, g[j]), old[j]);
      if (xr != nullptr) store4(xr + c, v[j]);
      if (w2 == nullptr) {
        if (yr != nullptr) store4(yr + c, v[j]);
      } else {
        ss2 += dot4(v[j]);
      }
    }
    if (w2 != nullptr) {
      const float r2 = rsqrtf(block_sum(ss2, part[1]) / static_cast<float>(d) + eps);
#pragma unroll
      for (int j = 0; j < NV; ++j) {
        const int c = (threadIdx.x + j * blockDim.x) * 4;
        if (c < dp) store4(yr + c, weigh4(v[j], r2, w_add, load4(w2 + c)));
      }
    }
  } else {
    float ss = 0.f;
    for (int c = threadIdx.x * 4; c < dp; c += blockDim.x * 4) {
      const float4 v = norm_source<T, SRC>(src, choice_row, choice_w, row, rows, c);
      store4(rowbuf + c, v);
      ss += dot4(v);
    }
    const float r = rsqrtf(block_sum(ss, part[0]) / static_cast<float>(d) + eps);
    float ss2 = 0.f;
    // a thread re-reads only the columns it wrote itself, so no barrier is needed between the passes
    for (int c = threadIdx.x * 4; c < dp; c += blockDim.x * 4) {
      float4 o = weigh4(load4(rowbuf + c), r, w_add, load4(w + c));
      if (add) o = add4(o, load4(xr + c));
      if (xr != nullptr) store4(xr + c, o);
      if (w2 != nullptr) {
        store4(rowbuf + c, o);
        ss2 += dot4(o);
      } else if (yr != nullptr) {
        store4(yr + c, o);
      }
    }
    if (w2 != nullptr) {
      const float r2 = rsqrtf(block_sum(ss2, part[1]) / static_cast<float>(d) + eps);
      for (int c = threadIdx.x * 4; c < dp; c += blockDim.x * 4)
        store4(yr + c, weigh4(load4(rowbuf + c), r2, w_add, load4(w2 + c)));
    }
  }
}

template <typename T, int SRC>
static int launch_residual_norm_src(const NormSource& src, const T* w, const T* w2, float* x, T* y, int rows, int d, int dp, float eps,
                                    float w_add, int add, cudaStream_t stream) {
  const int vecs = dp / 4;
  // Few rows: as many threads per row as there are vectors (the row's latency is all that counts). Many rows are bound by
  // bytes in flight: wide ones run as small CTAs, the gathers of a mixture with the row in registers, plain sources with the
  // row in shared memory (fewer registers, more CTAs per SM).
  int nv, threads;
  if (rows <= 296 || vecs <= 512) {
    nv = vecs <= 1024 ? 1 : (vecs <= 2048 ? 2 : 4);
    threads = (vecs + nv - 1) / nv;
  } else {
    nv = SRC == NSRC_MOE ? 4 : 0;
    threads = nv == 0 ? 256 : (vecs + nv - 1) / nv;
  }
  threads = (threads + 31) / 32 * 32;
  if (threads > (nv == 4 ? 512 : 1024)) { nv = 0; threads = 1024; }
  const size_t smem = (nv == 0 ? static_cast<size_t>(dp) * 4 : 0) + static_cast<size_t>(src.top + src.n_shared) * 8;
  if (smem > 220 * 1024) return -2;
#define RPEG_NORM_NV(NV_)                                                                                                       \
  {                                                                                                                             \
    auto kern = residual_norm_kernel<T, SRC, NV_>;                                                                              \
    if (smem > 48 * 1024 &&                                                                                                     \
        cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)) != cudaSuccess)         \
      return -20;                                                                                                               \
    const cudaError_t e = launch_pdl(kern, dim3(rows), dim3(threads), smem, stream, src, w, w2, x, y, rows, d, dp, eps, w_add, add); \
    return e == cudaSuccess ? 0 : -21;                                                                                          \
  }
  if (nv == 0) RPEG_NORM_NV(0)
  if (nv == 1) RPEG_NORM_NV(1)
  if (nv == 2) RPEG_NORM_NV(2)
  RPEG_NORM_NV(4)
#undef RPEG_NORM_NV
}

template <typename T>
static int launch_residual_norm(int kind, const NormSource& src, const void* w_, const void* w2_, float* x, void* y_, int rows, int d,
                                int dp, float eps, float w_add, int add, cudaStream_t stream) {
  const T *w = static_cast<const T*>(w_), *w2 = static_cast<const T*>(w2_);
  T* y = static_cast<T*>(y_);
  switch (kind) {
    case NSRC_ACT: return launch_residual_norm_src<T, NSRC_ACT>(src, w, w2, x, y, rows, d, dp, eps, w_add, add, stream);
    case NSRC_PARTIALS: return launch_residual_norm_src<T, NSRC_PARTIALS>(src, w, w2, x, y, rows, d, dp, eps, w_add, add, stream);
    case NSRC_MOE: return launch_residual_norm_src<T, NSRC_MOE>(src, w, w2, x, y, rows, d, dp, eps, w_add, add, stream);
    case NSRC_EMBED: return launch_residual_norm_src<T, NSRC_EMBED>(src, w, w2, x, y, rows, d, dp, eps, w_add, add, stream);
    case NSRC_STREAM: return launch_residual_norm_src<T, NSRC_STREAM>(src, w, w2, x, y, rows, d, dp, eps, w_add, add, stream);
    default: return -4;
  }
}

}  // namespace rpeg

using namespace rpeg;

extern "C" int rpeg_residual_norm(int kind, const void* src, int splits, long long stride, int ld, const int* idx, const float* wts,
                                  int top, int n_shared, long long shared_row0, const void* w, const void* w2, float* x, void* y,
                                  int rows, int d, int dp, float eps, float w_add, int add, int f32, void* stream) {
  if (rows <= 0) return 0;
  if ((dp & 7) || d > dp || d < 1 || (ld & 3) || top < 0 || n_shared < 0) return -2;
  if (kind == NSRC_MOE && shared_row0 + static_cast<long long>(n_shared) * rows > 0x7fffffffll) return -2;
  if ((add && x == nullptr) || (w2 != nullptr && y == nullptr)) return -3;
  const NormSource s{src, splits, stride, ld, idx, wts, top, n_shared, shared_row0};
  cudaStream_t st = reinterpret_cast<cudaStream_t>(stream);
  return f32 ? launch_residual_norm<float>(kind, s, w, w2, x, y, rows, d, dp, eps, w_add, add, st)
             : launch_residual_norm<__nv_bfloat16>(kind, s, w, w2, x, y, rows, d, dp, eps, w_add, add, st);
}
