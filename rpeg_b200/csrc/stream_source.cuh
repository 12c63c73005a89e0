// Where the kernels that update the residual stream take a sublayer's output from.
#pragma once
#include "act_io.cuh"

namespace rpeg {

enum { NSRC_ACT = 0, NSRC_PARTIALS = 1, NSRC_MOE = 2, NSRC_EMBED = 3, NSRC_STREAM = 4 };

struct NormSource {
  const void* p;            // activation / partials / expert rows / table / stream
  int splits;               // partials: how many, `stride` floats apart
  long long stride;
  int ld;                   // row pitch in elements
  const int* idx;           // token ids, or the expert-output row of every (token, choice)
  const float* wts;         // weight of every (token, choice); null: one
  int top, n_shared;        // choices per token; always-on experts: rows shared_row0 + s * rows + t, weight 1
  long long shared_row0;
};

// Four columns of one row; `choice_row`, `choice_w`: the row's expert outputs (NSRC_MOE).
template <typename T, int SRC>
__device__ __forceinline__ float4 norm_source(const NormSource& s, const int* choice_row, const float* choice_w, int row, int rows, int c) {
  if constexpr (SRC == NSRC_PARTIALS) {
    const float* p = static_cast<const float*>(s.p) + static_cast<size_t>(row) * s.ld + c;
    float4 v = load4(p);
#pragma unroll 8
    for (int k = 1; k < s.splits; ++k) v = add4(v, load4(p + k * s.stride));
    return v;
  } else if constexpr (SRC == NSRC_MOE) {
    const T* y = static_cast<const T*>(s.p) + c;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
    for (int k = 0; k < s.top + s.n_shared; ++k) {
      const float w = choice_w[k];
      const float4 e = load4(y + static_cast<size_t>(choice_row[k]) * s.ld);
      v.x = fmaf(w, e.x, v.x); v.y = fmaf(w, e.y, v.y); v.z = fmaf(w, e.z, v.z); v.w = fmaf(w, e.w, v.w);
    }
    return v;
  } else if constexpr (SRC == NSRC_EMBED) {
    return load4(static_cast<const T*>(s.p) + static_cast<size_t>(s.idx[row]) * s.ld + c);
  } else if constexpr (SRC == NSRC_STREAM) {
    return load4(static_cast<const float*>(s.p) + static_cast<size_t>(row) * s.ld + c);
  } else {
    return load4(static_cast<const T*>(s.p) + static_cast<size_t>(row) * s.ld + c);
  }
}

}  // namespace rpeg
