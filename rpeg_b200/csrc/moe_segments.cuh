// Row segments of a mixture of experts over `seg_rows` tokens, in the order in which the grouped GEMMs see them:
//   routed expert e      rows [seg_off[e], seg_off[e + 1])          (tokens that chose it; seg_off[n_routed] = tokens x choices)
//   always-on expert s   rows [seg_off[n_routed] + s * seg_rows, + seg_rows), token t at offset t
// A shared feed-forward wider than a routed one is cut along its hidden size into several always-on experts (the hidden
// units of a feed-forward without gate are independent, so the parts add up to the whole).
#pragma once

namespace rpeg {

struct MoeSegment {
  long long row0;
  int rows;
};

__device__ __forceinline__ MoeSegment moe_segment(const int* seg_off, int n_routed, int seg_rows, int s) {
  if (s < n_routed) {
    const int a = seg_off[s];
    return {a, seg_off[s + 1] - a};
  }
  return {seg_off[n_routed] + static_cast<long long>(s - n_routed) * seg_rows, seg_rows};
}

}  // namespace rpeg
