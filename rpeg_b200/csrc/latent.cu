// Latent attention: a token's cache row holds one latent of `rank` numbers, from which every head's key and value are linear maps, and
// one rotated key part that all heads share:
//
//   row = [ norm(c) (rank, padded to rank_p) | rotated part (rot, padded to rot_p) ],   W = rank_p + rot_p
//   key_h = (U_h c, rotated part),  value_h = V_h c
//
// Keys and values need not exist: a query through U_h^T scores the cached rows themselves, and the softmax average of cached
// latents goes through V_h once per query. `rank` and `rot` are padded to multiples of 8 with zeros.
//
//   latent_rows        one launch between the projections and the attention: weight-scaled RMS norm of up to two segments of a
//                      projection (a query latent to a buffer, the key/value latent to the cache), interleaved rotation of the shared
//                      key part (to the cache) and of the queries' rotated parts, and the activation of a feed-forward whose first
//                      product is part of the same projection
//   latent_gather      the cache rows a prompt sees, as one contiguous matrix (the operand of the products that give its keys and values)
//   latent_attn_rows   attention of single query rows over the cache on the CUDA cores, for fp32 and for sizes the tensor-core
//                      kernels (latent_decode.cu, latent_prefill.cu) do not take
#include "act_io.cuh"
#include "rpeg_kernels.h"

namespace rpeg {

constexpr int LPAGE = RPEG_KV_PAGE;

// A projection's output: an activation [rows, ld], or `splits` fp32 partials of it.
struct Projection {
  const void* p;
  int splits;
  long long stride;
  int ld;
};

template <typename T, bool PARTIALS>
__device__ __forceinline__ float4 read_projection(const Projection& s, int t, int col) {
  const size_t off = static_cast<size_t>(t) * s.ld + col;
  if constexpr (PARTIALS) {
    const float* p = static_cast<const float*>(s.p) + off;
    float4 a = load4(p);
#pragma unroll 8
    for (int k = 1; k < s.splits; ++k) a = add4(a, load4(p + k * s.stride));
    return a;
  } else {
    return load4(static_cast<const T*>(s.p) + off);
  }
}

struct LatentRows {
  Projection src;
  int rows;
  const int* pos; const int* slot;
  const float* cos_t; const float* sin_t;          // [positions, rot / 2]
  int rot, rot_p;
  float eps;
  // query latent: src columns [nq_col0, + nq_p), mean over the first nq; -> nq_out [rows, nq_p]; nq = 0: none
  int nq_col0, nq, nq_p;
  const void* nq_w; void* nq_out;
  // key/value latent and its rotated part: src columns [kv_col0, + rank_p + rot_p) -> cache row; rank = 0: none
  int kv_col0, rank, rank_p;
  const void* kv_w; void* cache; const int* page_table; int max_pages;
  // queries: head h at src column q_col0 + h * (dim_p + rot_p): [dim_p | rot_p]; H = 0: none. The rotated part goes to q_rot + t * ld_rot
  // + h * hs_rot, the other one to q_nope + t * ld_nope + h * dim_p (null: it stays where it is)
  int q_col0, H, dim_p;
  void* q_nope; int ld_nope;
  void* q_rot; int ld_rot, hs_rot;
  // feed-forward: squared relu of src columns [ff_col0, + ff_p) -> ff_out [rows, ff_p]; ff_p = 0: none
  int ff_col0, ff_p;
  void* ff_out;
};

__device__ __forceinline__ float4 rotate_pairs(float4 u, const LatentRows& a, int p, int c) {
  const int half = a.rot >> 1, pr = c >> 1;
  const size_t row = static_cast<size_t>(p) * half;
  float2 s0 = make_float2(1.f, 0.f), s1 = make_float2(1.f, 0.f);
  if (pr < half) s0 = make_float2(a.cos_t[row + pr], a.sin_t[row + pr]);
  if (pr + 1 < half) s1 = make_float2(a.cos_t[row + pr + 1], a.sin_t[row + pr + 1]);
  return make_float4(u.x * s0.x - u.y * s0.y, u.y * s0.x + u.x * s0.y, u.z * s1.x - u.w * s1.y, u.w * s1.x + u.z * s1.y);
}

// The first blocks normalise (one per token and segment), the others do what is elementwise (four columns per thread).
template <typename T, bool PARTIALS>
__global__ void __launch_bounds__(512)
latent_rows_kernel(const LatentRows a, int norm_blocks, int items) {
  griddep_launch();
  griddep_wait();
  extern __shared__ float rowbuf[];
  __shared__ float part[16];
  if (static_cast<int>(blockIdx.x) < norm_blocks) {
    const int nseg = (a.nq > 0) + (a.rank > 0);
    const int t = blockIdx.x / nseg;
    const bool kv = a.rank > 0 && blockIdx.x % nseg == nseg - 1;
    const int col0 = kv ? a.kv_col0 : a.nq_col0, n = kv ? a.rank : a.nq, np = kv ? a.rank_p : a.nq_p;
    const T* w = static_cast<const T*>(kv ? a.kv_w : a.nq_w);
    T* out;
    int p = 0;
    if (kv) {
      p = a.pos[t];
      const int page = a.page_table[static_cast<size_t>(a.slot[t]) * a.max_pages + p / LPAGE];
      out = static_cast<T*>(a.cache) + (static_cast<size_t>(page) * LPAGE + p % LPAGE) * (a.rank_p + a.rot_p);
    } else {
      out = static_cast<T*>(a.nq_out) + static_cast<size_t>(t) * a.nq_p;
    }
    float ss = 0.f;
    const int all = np + (kv ? a.rot_p : 0), step = blockDim.x * 4;
    for (int c = threadIdx.x * 4; c < all; c += step) {
      const float4 v = read_projection<T, PARTIALS>(a.src, t, col0 + c);
      if (c < np) {
        store4(rowbuf + c, v);
        ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
      } else {
        store4(out + c, rotate_pairs(v, a, p, c - np));
      }
    }
    ss = warp_sum(ss);
    if ((threadIdx.x & 31) == 0) part[threadIdx.x >> 5] = ss;
    __syncthreads();
    ss = warp_sum((threadIdx.x & 31) < (blockDim.x >> 5) ? part[threadIdx.x & 31] : 0.f);
    const float r = rsqrtf(ss / static_cast<float>(n) + a.eps);
    for (int c = threadIdx.x * 4; c < np; c += step) {                // a thread reads back only what it wrote
      const float4 v = load4(rowbuf + c), g = load4(w + c);
      store4(out + c, make_float4(v.x * r * g.x, v.y * r * g.y, v.z * r * g.z, v.w * r * g.w));
    }
    return;
  }
  const long long item = static_cast<long long>(blockIdx.x - norm_blocks) * blockDim.x + threadIdx.x;
  const int t = static_cast<int>(item / items);
  if (t >= a.rows) return;
  const int e = static_cast<int>(item - static_cast<long long>(t) * items);
  const int nr = a.rot_p >> 2, rot_items = a.H * nr, hw = a.dim_p + a.rot_p;
  if (e < rot_items) {
    const int h = e / nr, c = (e - h * nr) * 4;
    const float4 v = rotate_pairs(read_projection<T, PARTIALS>(a.src, t, a.q_col0 + h * hw + a.dim_p + c), a, a.pos[t], c);
    store4(static_cast<T*>(a.q_rot) + static_cast<size_t>(t) * a.ld_rot + h * a.hs_rot + c, v);
    return;
  }
  const int nd = a.dim_p >> 2, nope_items = a.q_nope != nullptr ? a.H * nd : 0;
  if (e < rot_items + nope_items) {
    const int f = e - rot_items, h = f / nd, c = (f - h * nd) * 4;
    store4(static_cast<T*>(a.q_nope) + static_cast<size_t>(t) * a.ld_nope + h * a.dim_p + c,
           read_projection<T, PARTIALS>(a.src, t, a.q_col0 + h * hw + c));
    return;
  }
  const int c = (e - rot_items - nope_items) * 4;
  const float4 v = read_projection<T, PARTIALS>(a.src, t, a.ff_col0 + c);
  store4(static_cast<T*>(a.ff_out) + static_cast<size_t>(t) * a.ff_p + c,
         make_float4(ff_act<FF_RELU2>(v.x), ff_act<FF_RELU2>(v.y), ff_act<FF_RELU2>(v.z), ff_act<FF_RELU2>(v.w)));
}

// One warp per visible row: row r of request b (off[b] <= r < off[b + 1]) is position lo[b] + r - off[b] of page-table row slot[cu[b]].
__global__ void __launch_bounds__(256)
latent_gather_kernel(const uint4* __restrict__ cache, int vecs, const int* __restrict__ page_table, int max_pages, const int* __restrict__ slot,
                     const int* __restrict__ cu, const int* __restrict__ off, const int* __restrict__ lo, int B, int rows, uint4* __restrict__ out) {
  const int r = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (r >= rows) return;
  int b = 0, hi = B;
  while (hi - b > 1) {
    const int mid = (b + hi) >> 1;
    if (off[mid] <= r) b = mid; else hi = mid;
  }
  const int p = lo[b] + r - off[b];
  const int page = page_table[static_cast<size_t>(slot[cu[b]]) * max_pages + p / LPAGE];
  const uint4* src = cache + (static_cast<size_t>(page) * LPAGE + p % LPAGE) * vecs;
  uint4* dst = out + static_cast<size_t>(r) * vecs;
  for (int i0 = lane; i0 < vecs; i0 += 96) {                          // three loads in flight per lane
    uint4 v[3];
#pragma unroll
    for (int k = 0; k < 3; ++k)
      if (i0 + 32 * k < vecs) v[k] = src[i0 + 32 * k];
#pragma unroll
    for (int k = 0; k < 3; ++k)
      if (i0 + 32 * k < vecs) dst[i0 + 32 * k] = v[k];
  }
}

// ---------------------------------------------------------------------------------- attention on the CUDA cores
constexpr int LA_THREADS = 256, LA_HEADS = 8, LA_VALS = 4;        // rank up to LA_THREADS * LA_VALS

struct LatentAttn {
  const void* q;                                                  // [rows, H, W]
  const void* cache;
  const int* page_table; int max_pages;
  const int* slot; const int* pos; const int* lens;               // lens null: pos + 1 keys
  const float* sink;
  void* out;                                                      // [rows, H, rank_p]
  int H, rank_p, W, window, tile;
  float scale;
};

// One CTA per (row, up to 8 heads). A tile of keys lies in shared memory as fp32 (rows one word apart from a bank conflict): a thread takes
// (key, head) pairs of the scores, then a warp per head runs the online softmax, then a thread owns latent dimensions of all heads.
template <typename T>
__global__ void __launch_bounds__(LA_THREADS)
latent_attn_rows_kernel(const LatentAttn a) {
  griddep_launch();
  griddep_wait();
  extern __shared__ float la_sm[];
  const int row = blockIdx.x, h0 = blockIdx.y * LA_HEADS, nh = min(LA_HEADS, a.H - h0), W = a.W, tile = a.tile;
  float* qs = la_sm;                               // [LA_HEADS][W]
  float* ks = qs + LA_HEADS * W;                   // [tile][W + 1]
  float* sc = ks + tile * (W + 1);                 // [LA_HEADS][tile]
  __shared__ float alpha[LA_HEADS], total[LA_HEADS];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int L = a.lens != nullptr ? a.lens[row] : a.pos[row] + 1;
  const int key0 = a.window > 0 ? max(0, L - a.window) : 0;
  const T* q = static_cast<const T*>(a.q) + (static_cast<size_t>(row) * a.H + h0) * W;
  for (int i = threadIdx.x; i < nh * W; i += LA_THREADS) qs[i] = load1(q + i) * a.scale;
  const int* pt = a.page_table + static_cast<size_t>(a.slot[row]) * a.max_pages;
  float acc[LA_HEADS][LA_VALS];
#pragma unroll
  for (int h = 0; h < LA_HEADS; ++h)
#pragma unroll
    for (int j = 0; j < LA_VALS; ++j) acc[h][j] = 0.f;
  float m = -INFINITY, l = 0.f;                    // warp h: the running softmax of head h
  if (a.sink != nullptr && warp < nh) { m = a.sink[h0 + warp]; l = 1.f; }
  for (int k0 = key0; k0 < L; k0 += tile) {
    const int nk = min(tile, L - k0);
    __syncthreads();
    for (int k = warp; k < nk; k += LA_THREADS / 32) {
      const int p = k0 + k;
      const T* src = static_cast<const T*>(a.cache) + (static_cast<size_t>(pt[p / LPAGE]) * LPAGE + p % LPAGE) * W;
      for (int d = lane * 4; d < W; d += 128) {
        const float4 v = load4(src + d);
        float* dst = ks + k * (W + 1) + d;
        dst[0] = v.x; dst[1] = v.y; dst[2] = v.z; dst[3] = v.w;
      }
    }
    __syncthreads();
    for (int i = threadIdx.x; i < nh * tile; i += LA_THREADS) {
      const int h = i / tile, k = i % tile;
      float s = -INFINITY;
      if (k < nk) {
        const float *x = qs + h * W, *y = ks + k * (W + 1);
        float s4[4] = {0.f, 0.f, 0.f, 0.f};
        for (int d = 0; d < W; d += 4)
#pragma unroll
          for (int e = 0; e < 4; ++e) s4[e] = fmaf(x[d + e], y[d + e], s4[e]);
        s = (s4[0] + s4[1]) + (s4[2] + s4[3]);
      }
      sc[i] = s;
    }
    __syncthreads();
    if (warp < nh) {
      float b = -INFINITY;
      for (int k = lane; k < nk; k += 32) b = fmaxf(b, sc[warp * tile + k]);
      const float nm = fmaxf(m, warp_max(b)), al = m == -INFINITY ? 0.f : __expf(m - nm);
      float s = 0.f;
      for (int k = lane; k < nk; k += 32) {
        const float p = __expf(sc[warp * tile + k] - nm);
        sc[warp * tile + k] = p;
        s += p;
      }
      l = l * al + warp_sum(s);
      m = nm;
      if (lane == 0) alpha[warp] = al;
    }
    __syncthreads();
#pragma unroll
    for (int j = 0; j < LA_VALS; ++j) {
      const int d = threadIdx.x + j * LA_THREADS;
      if (d >= a.rank_p) continue;
#pragma unroll
      for (int h = 0; h < LA_HEADS; ++h) acc[h][j] *= h < nh ? alpha[h] : 0.f;
      for (int k = 0; k < nk; ++k) {
        const float v = ks[k * (W + 1) + d];
#pragma unroll
        for (int h = 0; h < LA_HEADS; ++h)
          if (h < nh) acc[h][j] = fmaf(sc[h * tile + k], v, acc[h][j]);
      }
    }
  }
  if (warp < nh && lane == 0) total[warp] = l;
  __syncthreads();
  T* out = static_cast<T*>(a.out) + (static_cast<size_t>(row) * a.H + h0) * a.rank_p;
#pragma unroll
  for (int j = 0; j < LA_VALS; ++j) {
    const int d = threadIdx.x + j * LA_THREADS;
    if (d >= a.rank_p) continue;
#pragma unroll
    for (int h = 0; h < LA_HEADS; ++h)
      if (h < nh) {
        const float r = L > 0 && total[h] > 0.f ? acc[h][j] / total[h] : 0.f;
        if constexpr (sizeof(T) == 2) out[h * a.rank_p + d] = __float2bfloat16(r); else out[h * a.rank_p + d] = r;
      }
  }
}

template <typename T>
static int launch_latent_attn_rows(LatentAttn a, int rows, cudaStream_t stream) {
  a.tile = 64;
  auto bytes = [&](int tile) { return static_cast<size_t>(LA_HEADS * a.W + tile * (a.W + 1) + LA_HEADS * tile) * 4; };
  while (a.tile > 4 && bytes(a.tile) > 220 * 1024) a.tile >>= 1;
  const size_t smem = bytes(a.tile);
  if (smem > 220 * 1024) return -3;
  auto kern = latent_attn_rows_kernel<T>;
  static size_t configured = 48 * 1024;
  if (smem > configured) {
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem)) != cudaSuccess) return -20;
    configured = smem;
  }
  return launch_pdl(kern, dim3(rows, (a.H + LA_HEADS - 1) / LA_HEADS), dim3(LA_THREADS), smem, stream, a) == cudaSuccess ? 0 : -21;
}

}  // namespace rpeg

using namespace rpeg;
#define STREAM(s) reinterpret_cast<cudaStream_t>(s)

extern "C" int rpeg_latent_rows(const void* src, int splits, long long stride, int ld, int rows, const int* pos, const int* slot,
                                const float* cos_t, const float* sin_t, int rot, int rot_p, float eps, int nq_col0, int nq, int nq_p,
                                const void* nq_w, void* nq_out, int kv_col0, int rank, int rank_p, const void* kv_w, void* cache,
                                const int* page_table, int max_pages, int q_col0, int H, int dim_p, void* q_nope, int ld_nope, void* q_rot,
                                int ld_rot, int hs_rot, int ff_col0, int ff_p, void* ff_out, int f32, void* stream) {
  if (rows <= 0) return 0;
  if ((ff_p & 7) || (ff_col0 & 3) || ff_p < 0 || (ff_p > 0 && ff_out == nullptr)) return -2;
  if ((rot_p | nq_p | rank_p | dim_p | ld_nope | ld_rot | hs_rot) & 7 || ((ld | nq_col0 | kv_col0 | q_col0) & 3)) return -2;
  if (rot < 0 || rot > rot_p || (rot & 1) || nq > nq_p || rank > rank_p || H < 0) return -2;
  if ((nq > 0 && (nq_w == nullptr || nq_out == nullptr)) || (rank > 0 && (kv_w == nullptr || cache == nullptr || page_table == nullptr)) ||
      (H > 0 && rot_p > 0 && q_rot == nullptr))
    return -3;
  const LatentRows a{{src, splits, stride, ld}, rows, pos, slot, cos_t, sin_t, rot, rot_p, eps, nq_col0, nq, nq_p, nq_w, nq_out, kv_col0, rank,
                     rank_p, kv_w, cache, page_table, max_pages, q_col0, H, dim_p, q_nope, ld_nope, q_rot, ld_rot, hs_rot, ff_col0, ff_p, ff_out};
  const long long norm_blocks = static_cast<long long>(rows) * ((nq > 0) + (rank > 0));
  const int items = H * ((rot_p >> 2) + (q_nope != nullptr ? dim_p >> 2 : 0)) + (ff_p >> 2);
  // few tokens: a normalised row in one step of its block (its latency is all that counts); many: small blocks
  const int widest = norm_blocks && rows <= 1024 ? (nq_p > rank_p + rot_p ? nq_p : rank_p + rot_p) : 0;
  int threads = 128;
  while (threads < 512 && threads * 4 < widest) threads *= 2;
  const long long blocks = norm_blocks + (static_cast<long long>(rows) * items + threads - 1) / threads;
  if (blocks <= 0) return 0;
  const size_t smem = static_cast<size_t>(norm_blocks ? (nq_p > rank_p ? nq_p : rank_p) : 0) * 4;
  if (blocks > 0x7fffffffll || smem > 48 * 1024) return -2;
#define RPEG_LR(T_, P_)                                                                                                                      \
  return launch_pdl(latent_rows_kernel<T_, P_>, dim3(static_cast<unsigned>(blocks)), dim3(threads), smem, STREAM(stream), a,                 \
                    static_cast<int>(norm_blocks), items) == cudaSuccess ? 0 : -21;
  if (f32) { RPEG_LR(float, false) }
  if (splits > 0) { RPEG_LR(__nv_bfloat16, true) }
  RPEG_LR(__nv_bfloat16, false)
#undef RPEG_LR
}

// `row_bytes` = W elements of the cache's type; cu [B + 1] rows of the requests' portions, off [B + 1] rows and lo [B] first positions of what each sees.
extern "C" int rpeg_latent_gather(const void* cache, int row_bytes, const int* page_table, int max_pages, const int* slot, const int* cu,
                                  const int* off, const int* lo, int B, int rows, void* out, void* stream) {
  if (rows <= 0 || B <= 0) return 0;
  if (row_bytes & 15) return -2;
  latent_gather_kernel<<<(rows + 7) / 8, 256, 0, STREAM(stream)>>>(static_cast<const uint4*>(cache), row_bytes / 16, page_table, max_pages, slot,
                                                                   cu, off, lo, B, rows, static_cast<uint4*>(out));
  return cudaGetLastError() == cudaSuccess ? 0 : -21;
}

extern "C" int rpeg_latent_attn_rows(const void* q, const void* cache, const int* page_table, int max_pages, const int* slot, const int* pos,
                                     const int* lens, const float* sink, void* out, int rows, int H, int rank_p, int W, int window, float scale,
                                     int f32, void* stream) {
  if (rows <= 0) return 0;
  if (((rank_p | W) & 7) || rank_p < 8 || rank_p > LA_THREADS * LA_VALS || W < rank_p || H < 1 || window < 0) return -2;
  const LatentAttn a{q, cache, page_table, max_pages, slot, pos, lens, sink, out, H, rank_p, W, window, 0, scale};
  return f32 ? launch_latent_attn_rows<float>(a, rows, STREAM(stream)) : launch_latent_attn_rows<__nv_bfloat16>(a, rows, STREAM(stream));
}
