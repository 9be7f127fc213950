// Mixture of experts: grouped top-k routing over sigmoid scores, and the expert products over the routed rows.
//
// Routing: one warp per token picks the experts from fp32 logits and takes a place in each expert's list; a
// second launch turns the lists into one matrix of rows sorted by expert (a copy of each token's activations
// per chosen expert) plus the tiles the products run over.  Everything stays on the device: the grids are
// sized by the bounds the host knows (rows * top rows, at most experts + rows * top / tile tiles) and a CTA
// beyond the last tile returns.
//
// Products: for every expert  act = f(x . W_gate^T, x . W_up^T)  in one launch (gate, up and the activation),
// then  y = act . W_down^T  in another; the weighted sum over a token's experts is taken by the residual
// kernel that follows (residual_norm.cu).  bf16 runs on tcgen05 with the weights as the M side (moe_umma.cu);
// this file holds the fp32-arithmetic evaluation of every other size and type.
#include <limits.h>
#include <math.h>

#include "moe.cuh"

namespace axb {
namespace {

constexpr int kRouteWarps = 8;

struct RouteParams {
  const float *logits;      // (rows, experts)
  const float *correction;  // (experts), or null
  int32_t *ids;             // (rows, top), in the order of choice
  float *weights;           // (rows, top)
  int32_t *place;           // (rows, top): place in the expert's list
  int32_t *counts;          // (experts), zero on entry
  int rows, experts, groups, keep, top, rows_per_warp;
  float scale;
};

// argmax over lanes, the lowest index among equal values
__device__ __forceinline__ void warp_argmax(float &v, int &i) {
#pragma unroll
  for (int off = 16; off > 0; off >>= 1) {
    const float ov = __shfl_xor_sync(0xffffffffu, v, off);
    const int oi = __shfl_xor_sync(0xffffffffu, i, off);
    if (ov > v || (ov == v && oi < i)) v = ov, i = oi;
  }
}

// choice = sigmoid(logit) + correction.  A group of neighbouring experts is worth the sum of its two largest
// choices; only the `keep` best groups are open, and among their experts the `top` largest choices win.
// Weights are the scores without the correction, times scale.
__global__ void __launch_bounds__(kRouteWarps * 32) moe_route_kernel(const RouteParams p) {
  extern __shared__ float sm[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, row0 = blockIdx.x * kRouteWarps * p.rows_per_warp;
  int *count = reinterpret_cast<int *>(sm);  // rows of this CTA per expert; then the CTA's first place there
  float *score = sm + p.experts + (size_t)warp * (2 * p.experts + p.groups), *choice = score + p.experts, *group = choice + p.experts;
  for (int e = threadIdx.x; e < p.experts; e += kRouteWarps * 32) count[e] = 0;
  grid_dependency_wait();
  grid_dependency_launch();
  __syncthreads();
  const int row_end = min(p.rows, row0 + kRouteWarps * p.rows_per_warp);
#pragma unroll 1
  for (int row = row0 + warp; row < row_end; row += kRouteWarps) {
    for (int e = lane; e < p.experts; e += 32) {
      const float s = 1.0f / (1.0f + expf(-p.logits[(size_t)row * p.experts + e]));
      score[e] = s;
      choice[e] = s + (p.correction ? p.correction[e] : 0.f);
    }
    __syncwarp();
    if (p.keep < p.groups) {
      const int size = p.experts / p.groups;
      for (int g = lane; g < p.groups; g += 32) {
        float a = -INFINITY, b = -INFINITY;  // the two largest
        for (int e = g * size; e < (g + 1) * size; ++e) {
          const float c = choice[e];
          if (c > a)
            b = a, a = c;
          else if (c > b)
            b = c;
        }
        group[g] = size > 1 ? a + b : a;
      }
      __syncwarp();
      // close all but the `keep` best groups: an open group is marked by a NaN-free flag in its score
      for (int k = 0; k < p.keep; ++k) {
        float best = -INFINITY;
        int at = INT_MAX;
        for (int g = lane; g < p.groups; g += 32)
          if (group[g] > best || (group[g] == best && g < at)) best = group[g], at = g;
        warp_argmax(best, at);
        __syncwarp();
        if (lane == 0 && at != INT_MAX) group[at] = -INFINITY;
        __syncwarp();
      }
      for (int e = lane; e < p.experts; e += 32)
        if (group[e / size] != -INFINITY) choice[e] = -INFINITY;
      __syncwarp();
    }
    for (int k = 0; k < p.top; ++k) {
      float best = -INFINITY;
      int at = INT_MAX;
      for (int e = lane; e < p.experts; e += 32)
        if (choice[e] > best) best = choice[e], at = e;
      warp_argmax(best, at);
      if (at == INT_MAX) at = 0;  // only with NaN logits: stay in bounds
      __syncwarp();
      if (lane == 0) {
        choice[at] = -INFINITY;
        const int64_t o = (int64_t)row * p.top + k;
        p.ids[o] = at;
        p.weights[o] = score[at] * p.scale;
        p.place[o] = atomicAdd(&count[at], 1);
      }
      __syncwarp();
    }
  }
  __syncthreads();
  for (int e = threadIdx.x; e < p.experts; e += kRouteWarps * 32) count[e] = count[e] ? atomicAdd(&p.counts[e], count[e]) : 0;
  __syncthreads();
  for (int64_t o = (int64_t)row0 * p.top + threadIdx.x; o < (int64_t)row_end * p.top; o += kRouteWarps * 32)
    p.place[o] += count[p.ids[o]];
}

// offsets[e] = start of expert e's rows in the sorted order; tiles of up to tile_rows rows in expert order.
// Every CTA forms the offsets for itself (a scan over the experts in shared memory) and copies its tokens'
// rows to their places; CTA 0 also stores offsets and tiles.
constexpr int kSortThreads = 256;
__global__ void __launch_bounds__(kSortThreads)
moe_sort_kernel(const uint8_t *x, uint8_t *sorted, const int32_t *ids, const int32_t *place, const int32_t *counts,
                int32_t *row_of, int32_t *offsets, int4 *tiles, int32_t *n_tiles, int rows, int experts, int top,
                int tile_rows, int row_bytes, int unit) {
  extern __shared__ int offs[];  // (experts + 1) offsets, then (experts + 1) tile offsets
  int *toffs = offs + experts + 1;
  grid_dependency_wait();
  grid_dependency_launch();
  for (int e = threadIdx.x; e < experts; e += kSortThreads) offs[e + 1] = counts[e];
  __syncthreads();
  if (threadIdx.x < 32) {
    // inclusive scans of the counts and of the tile counts, 32 experts at a time
    int base = 0, tbase = 0;
    for (int e0 = 0; e0 < experts; e0 += 32) {
      const int e = e0 + threadIdx.x;
      int c = e < experts ? offs[e + 1] : 0, t = (c + tile_rows - 1) / tile_rows;
#pragma unroll
      for (int d = 1; d < 32; d <<= 1) {
        const int oc = __shfl_up_sync(0xffffffffu, c, d), ot = __shfl_up_sync(0xffffffffu, t, d);
        if ((int)threadIdx.x >= d) c += oc, t += ot;
      }
      if (e < experts) offs[e + 1] = base + c, toffs[e + 1] = tbase + t;
      base += __shfl_sync(0xffffffffu, c, 31);
      tbase += __shfl_sync(0xffffffffu, t, 31);
    }
    if (threadIdx.x == 0) offs[0] = toffs[0] = 0;
  }
  __syncthreads();
  if (blockIdx.x == 0) {
    for (int e = threadIdx.x; e <= experts; e += kSortThreads) offsets[e] = offs[e];
    for (int e = threadIdx.x; e < experts; e += kSortThreads)
      for (int t = toffs[e]; t < toffs[e + 1]; ++t) {
        const int r0 = offs[e] + (t - toffs[e]) * tile_rows;
        tiles[t] = make_int4(e, r0, min(tile_rows, offs[e + 1] - r0), 0);
      }
    if (threadIdx.x == 0) *n_tiles = toffs[experts];
  }
  for (int item = blockIdx.x; item < rows * top; item += gridDim.x) {
    const int e = ids[item], dst = offs[e] + place[item];
    if (threadIdx.x == 0) row_of[item] = dst;
    const uint8_t *s = x + (size_t)(item / top) * row_bytes;
    uint8_t *d = sorted + (size_t)dst * row_bytes;
    if (unit == 16)
      for (int i = threadIdx.x; i < row_bytes / 16; i += kSortThreads)
        reinterpret_cast<uint4 *>(d)[i] = reinterpret_cast<const uint4 *>(s)[i];
    else
      for (int i = threadIdx.x; i < row_bytes / 2; i += kSortThreads)
        reinterpret_cast<uint16_t *>(d)[i] = reinterpret_cast<const uint16_t *>(s)[i];
  }
}

// ---- any size and type: 32 rows x 32 features per CTA, fp32 arithmetic ---------------------------------
constexpr int kGenRows = 32, kGenCols = 32, kGenK = 32, kGenThreads = 256;

template <typename T, bool kGateUp>
__global__ void __launch_bounds__(kGenThreads) moe_product_generic_kernel(const MoeProduct p) {
  __shared__ float xs[kGenRows][kGenK + 1], ws[kGateUp ? 2 : 1][kGenCols][kGenK + 1];
  grid_dependency_wait();
  grid_dependency_launch();
  int4 tile;
  if (!moe_tile(p, blockIdx.y, kGenRows, tile)) return;
  const int c0 = blockIdx.x * kGenCols;
  const T *x = static_cast<const T *>(p.x) + (size_t)tile.y * p.in;
  const T *w = static_cast<const T *>(p.w) + (size_t)tile.x * (kGateUp ? 2 : 1) * p.out * p.in;
  const int col = threadIdx.x & 31, r0 = threadIdx.x >> 5;  // rows r0, r0 + 8, r0 + 16, r0 + 24
  float acc[kGateUp ? 2 : 1][4] = {};
  for (int k0 = 0; k0 < p.in; k0 += kGenK) {
    __syncthreads();
    for (int i = threadIdx.x; i < kGenRows * kGenK; i += kGenThreads) {
      const int r = i / kGenK, k = i % kGenK;
      xs[r][k] = r < tile.z && k0 + k < p.in ? ldf(x + (size_t)r * p.in + k0 + k) : 0.f;
    }
    for (int i = threadIdx.x; i < kGenCols * kGenK; i += kGenThreads) {
      const int c = i / kGenK, k = i % kGenK;
      const bool in = c0 + c < p.out && k0 + k < p.in;
      ws[0][c][k] = in ? ldf(w + (size_t)(c0 + c) * p.in + k0 + k) : 0.f;
      if (kGateUp) ws[1][c][k] = in ? ldf(w + (size_t)(p.out + c0 + c) * p.in + k0 + k) : 0.f;
    }
    __syncthreads();
#pragma unroll 8
    for (int k = 0; k < kGenK; ++k) {
#pragma unroll
      for (int g = 0; g < (kGateUp ? 2 : 1); ++g) {
        const float wv = ws[g][col][k];
#pragma unroll
        for (int i = 0; i < 4; ++i) acc[g][i] = fmaf(xs[r0 + 8 * i][k], wv, acc[g][i]);
      }
    }
  }
  if (c0 + col >= p.out) return;
  T *y = static_cast<T *>(p.y) + (size_t)tile.y * p.out + c0 + col;
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int r = r0 + 8 * i;
    if (r >= tile.z) continue;
    float v = acc[0][i];
    if (kGateUp) v = clamped_gate<sizeof(T) == 4>(acc[0][i], acc[kGateUp ? 1 : 0][i], p.act);
    stf(y + (size_t)r * p.out, v);
  }
}

template <typename T>
int launch_generic(const MoeProduct &p, bool gate_up, cudaStream_t st) {
  const dim3 grid((p.out + kGenCols - 1) / kGenCols, p.max_tiles);
  return gate_up ? launch_dependent(moe_product_generic_kernel<T, true>, grid, dim3(kGenThreads), 0, st, p)
                 : launch_dependent(moe_product_generic_kernel<T, false>, grid, dim3(kGenThreads), 0, st, p);
}

// The grid bound of a product, in tiles; < 0: invalid.
int check_product(MoeProduct &p) {
  if (!p.x || !p.w || !p.y || (p.tiles && !p.n_tiles)) return -AXB200_INVALID_PTR;
  if (p.rows <= 0 || p.experts <= 0 || p.in <= 0 || p.out <= 0 || p.tile_rows <= 0 || (!p.tiles && p.experts != 1))
    return -AXB200_INVALID_ARGUMENT;
  const int64_t bound = p.tiles ? (int64_t)p.rows / p.tile_rows + (p.experts < p.rows ? p.experts : p.rows)
                                : ((int64_t)p.rows + p.tile_rows - 1) / p.tile_rows;
  if (bound > 65535) return -AXB200_INVALID_ARGUMENT;
  p.max_tiles = (int)bound;
  p.wait_ns = wait_limit_ns();
  return AXB200_OK;
}

int products(MoeProduct routed, MoeProduct shared, bool gate_up, int dtype, void *stream) {
  if (dtype != AXB200_FLOAT32 && dtype != AXB200_BFLOAT16) return AXB200_UNSUPPORTED_TYPE;
  if (routed.rows == 0 && shared.rows == 0) return AXB200_OK;
  int rc = check_product(routed);
  if (rc == AXB200_OK && shared.rows > 0) rc = check_product(shared);
  if (rc != AXB200_OK) return -rc;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const bool umma = dtype == AXB200_BFLOAT16 && moe_umma_supported(routed, gate_up);
  if (umma && (shared.rows == 0 || moe_umma_supported(shared, gate_up))) return moe_umma(routed, shared, gate_up, st);
  if (umma) {
    rc = moe_umma(routed, MoeProduct{}, gate_up, st);
  } else {
    if (routed.tile_rows > kGenRows) return AXB200_INVALID_ARGUMENT;
    rc = dtype == AXB200_FLOAT32 ? launch_generic<float>(routed, gate_up, st) : launch_generic<__nv_bfloat16>(routed, gate_up, st);
  }
  if (rc != AXB200_OK || shared.rows == 0) return rc;
  shared.tile_rows = kGenRows;
  rc = check_product(shared);
  if (rc != AXB200_OK) return -rc;
  return dtype == AXB200_FLOAT32 ? launch_generic<float>(shared, gate_up, st) : launch_generic<__nv_bfloat16>(shared, gate_up, st);
}

}  // namespace
}  // namespace axb

extern "C" {

int axb200_moe_route(const float *logits, const float *correction, int32_t *ids, float *weights, int32_t *place,
                     int32_t *counts, int64_t rows, int experts, int groups, int keep, int top, float scale, void *stream) {
  if (!logits || !ids || !weights || !place || !counts) return AXB200_INVALID_PTR;
  if (rows < 0 || rows > 0x7fffffff || experts <= 0 || experts > 2048 || groups <= 0 || experts % groups != 0 || keep <= 0 ||
      keep > groups || top <= 0 || top > keep * (experts / groups) || rows * top > 0x7fffffff)
    return AXB200_INVALID_ARGUMENT;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (cudaMemsetAsync(counts, 0, (size_t)experts * sizeof(int32_t), st) != cudaSuccess) return AXB200_DEVICE_ERROR;
  if (rows == 0) return AXB200_OK;
  // enough rows per CTA that its experts' places come in one round of global atomics, and enough CTAs
  const int per_warp = rows >= 148 * 2 * axb::kRouteWarps * 4 ? 4 : rows >= 148 * axb::kRouteWarps * 2 ? 2 : 1;
  axb::RouteParams p{logits, correction, ids, weights, place, counts, (int)rows, experts, groups, keep, top, per_warp, scale};
  const size_t smem = ((size_t)experts + axb::kRouteWarps * (2 * experts + groups)) * sizeof(float);
  if (smem > 48 * 1024 && cudaFuncSetAttribute(axb::moe_route_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                               (int)smem) != cudaSuccess)
    return AXB200_DEVICE_ERROR;
  const int per_cta = axb::kRouteWarps * per_warp;
  return axb::launch_dependent(axb::moe_route_kernel, dim3((unsigned)((rows + per_cta - 1) / per_cta)), dim3(axb::kRouteWarps * 32),
                               smem, st, p);
}

int axb200_moe_tile_rows(int64_t rows, int experts, int width, int ff, int dtype) {
  if (rows <= 0 || experts <= 0 || width <= 0 || ff <= 0) return 0;
  if (dtype == AXB200_BFLOAT16 && axb::moe_umma_takes(width, ff)) return axb::moe_umma_tile_rows(rows, experts);
  return axb::kGenRows;
}

int axb200_moe_sort(const void *x, void *sorted, const int32_t *ids, const int32_t *place, const int32_t *counts,
                    int32_t *row_of, int32_t *offsets, int32_t *tiles, int32_t *n_tiles, int64_t rows, int experts, int top,
                    int tile_rows, int width, int dtype, void *stream) {
  const size_t es = axb::dtype_size(dtype);
  if (es == 0) return AXB200_UNSUPPORTED_TYPE;
  if (!x || !sorted || !ids || !place || !counts || !row_of || !offsets || !tiles || !n_tiles) return AXB200_INVALID_PTR;
  if (rows < 0 || experts <= 0 || experts > 2048 || top <= 0 || rows * top > 0x7fffffff || tile_rows <= 0 || width <= 0)
    return AXB200_INVALID_ARGUMENT;
  if (rows == 0) return AXB200_OK;
  const int row_bytes = (int)(width * es);
  const bool vec = row_bytes % 16 == 0 && ((reinterpret_cast<uintptr_t>(x) | reinterpret_cast<uintptr_t>(sorted)) & 15u) == 0;
  const int64_t items = rows * top;
  const int grid = (int)(items < 148 * 8 ? items : 148 * 8);
  return axb::launch_dependent(axb::moe_sort_kernel, dim3(grid), dim3(axb::kSortThreads), (size_t)2 * (experts + 1) * sizeof(int),
                               static_cast<cudaStream_t>(stream), static_cast<const uint8_t *>(x), static_cast<uint8_t *>(sorted),
                               ids, place, counts, row_of, offsets, reinterpret_cast<int4 *>(tiles), n_tiles, (int)rows, experts,
                               top, tile_rows, row_bytes, vec ? 16 : 2);
}

int axb200_moe_gate_up(const void *x, const void *w, void *act, const int32_t *tiles, const int32_t *n_tiles, int64_t rows,
                       int experts, int ff, float limit, const void *shared_x, const void *shared_w, void *shared_act,
                       int64_t shared_rows, int shared_ff, float shared_limit, int width, int tile_rows, float slope,
                       float offset, int dtype, void *stream) {
  if (rows < 0 || rows > 0x7fffffff || shared_rows < 0 || shared_rows > 0x7fffffff) return AXB200_INVALID_ARGUMENT;
  axb::MoeProduct p{}, s{};
  p.x = x, p.w = w, p.y = act, p.tiles = reinterpret_cast<const int4 *>(tiles), p.n_tiles = n_tiles;
  p.rows = (int)rows, p.experts = experts, p.in = width, p.out = ff, p.tile_rows = tile_rows;
  p.act = {limit, slope, offset};
  s.x = shared_x, s.w = shared_w, s.y = shared_act, s.rows = (int)shared_rows, s.experts = 1, s.in = width, s.out = shared_ff;
  s.tile_rows = tile_rows;
  s.act = {shared_limit, slope, offset};
  return axb::products(p, s, true, dtype, stream);
}

int axb200_moe_down(const void *act, const void *w, void *y, const int32_t *tiles, const int32_t *n_tiles, int64_t rows,
                    int experts, int ff, const void *shared_act, const void *shared_w, void *shared_y, int64_t shared_rows,
                    int shared_ff, int width, int tile_rows, int dtype, void *stream) {
  if (rows < 0 || rows > 0x7fffffff || shared_rows < 0 || shared_rows > 0x7fffffff) return AXB200_INVALID_ARGUMENT;
  axb::MoeProduct p{}, s{};
  p.x = act, p.w = w, p.y = y, p.tiles = reinterpret_cast<const int4 *>(tiles), p.n_tiles = n_tiles;
  p.rows = (int)rows, p.experts = experts, p.in = ff, p.out = width, p.tile_rows = tile_rows;
  s.x = shared_act, s.w = shared_w, s.y = shared_y, s.rows = (int)shared_rows, s.experts = 1, s.in = shared_ff, s.out = width;
  s.tile_rows = tile_rows;
  return axb::products(p, s, false, dtype, stream);
}

}  // extern "C"
