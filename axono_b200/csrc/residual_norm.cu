// The residual stream of a decoder whose mixer and feed-forward both read the same x ("parallel" layers),
// kept in fp32: one launch between two layers adds everything the finished layer contributes - the mixer's
// output, the weighted rows of the chosen experts, the shared expert's output - and writes the one or two
// layer norms that the next layer (or the output projection) reads.  Both norms share the row's mean and
// variance, so the second costs one multiply per element.  Another kernel is the start of the stream: embedding
// gather + layer norm.  The operators of fused.cu are their RMS, fp16 / fp32-storage siblings.
//
// The other kind of stream norms what a sublayer puts out, not what it reads: x += rms_norm(y) * (offset + w), and the
// next sublayer reads x itself (rounded to the activations' type), or after the last one the model's final norm of it.
#include "vec.cuh"

namespace axb {
namespace {

constexpr int kThreads = 256;

struct RowStats {
  float mean, inv;
};

// Mean and 1 / sqrt(mean of squared deviations + eps) of the row in `row` (each thread reads back only the
// elements it wrote).
template <int kVec>
__device__ __forceinline__ RowStats row_stats(const float *row, int width, float sum, float eps, float *scratch) {
  RowStats s;
  s.mean = block_sum(sum, scratch) / (float)width;
  float sq = 0.f;
  for (int c = threadIdx.x * kVec; c < width; c += kThreads * kVec)
#pragma unroll
    for (int i = 0; i < kVec; ++i) {
      const float d = row[c + i] - s.mean;
      sq = fmaf(d, d, sq);
    }
  s.inv = 1.0f / sqrtf(block_sum(sq, scratch) / (float)width + eps);
  return s;
}

template <typename T>
struct ResidualParams {
  float *x;             // (rows, width), updated in place
  const T *a, *b;       // (rows, width) addends, or null
  const T *expert_rows; // (slots, width), or null: sum_k weight[r, k] * expert_rows[slot[r, k]]
  const int32_t *slot;  // (rows, top)
  const float *weight;  // (rows, top)
  int top;
  const T *w1, *w2;  // norm weights; null: no such output
  T *h1, *h2;
  float eps;
  int width;
};

template <typename T, int kVec>
__global__ void __launch_bounds__(kThreads) residual_layer_norm_kernel(const ResidualParams<T> p) {
  extern __shared__ float row[];
  __shared__ float scratch[32];
  const size_t r = blockIdx.x, off = r * p.width;
  grid_dependency_wait();
  grid_dependency_launch();
  const bool adds = p.a || p.b || p.expert_rows;
  float sum = 0.f;
  for (int c = threadIdx.x * kVec; c < p.width; c += kThreads * kVec) {
    float v[kVec], t[kVec];
    load_vec<kVec>(p.x + off + c, v);
    float add[kVec] = {};
    if (p.a) {
      load_vec<kVec>(p.a + off + c, t);
#pragma unroll
      for (int i = 0; i < kVec; ++i) add[i] += t[i];
    }
    if (p.b) {
      load_vec<kVec>(p.b + off + c, t);
#pragma unroll
      for (int i = 0; i < kVec; ++i) add[i] += t[i];
    }
    if (p.expert_rows) {
      for (int k = 0; k < p.top; ++k) {
        const float wt = p.weight[r * p.top + k];
        load_vec<kVec>(p.expert_rows + (size_t)p.slot[r * p.top + k] * p.width + c, t);
#pragma unroll
        for (int i = 0; i < kVec; ++i) add[i] = fmaf(wt, t[i], add[i]);
      }
    }
#pragma unroll
    for (int i = 0; i < kVec; ++i) {
      v[i] += add[i];
      row[c + i] = v[i];
      sum += v[i];
    }
    if (adds) store_vec<kVec>(p.x + off + c, v);
  }
  if (!p.w1 && !p.w2) return;
  const RowStats st = row_stats<kVec>(row, p.width, sum, p.eps, scratch);
  for (int c = threadIdx.x * kVec; c < p.width; c += kThreads * kVec) {
    float n[kVec], w[kVec], o[kVec];
#pragma unroll
    for (int i = 0; i < kVec; ++i) n[i] = (row[c + i] - st.mean) * st.inv;
    if (p.w1) {
      load_vec<kVec>(p.w1 + c, w);
#pragma unroll
      for (int i = 0; i < kVec; ++i) o[i] = n[i] * w[i];
      store_vec<kVec>(p.h1 + off + c, o);
    }
    if (p.w2) {
      load_vec<kVec>(p.w2 + c, w);
#pragma unroll
      for (int i = 0; i < kVec; ++i) o[i] = n[i] * w[i];
      store_vec<kVec>(p.h2 + off + c, o);
    }
  }
}

template <typename T, int kVec>
__global__ void __launch_bounds__(kThreads)
embed_layer_norm_kernel(const int64_t *ids, const T *table, const T *w, float eps, float *x, long long vocab, int width) {
  extern __shared__ float row[];
  __shared__ float scratch[32];
  const size_t off = (size_t)blockIdx.x * width;
  grid_dependency_wait();
  grid_dependency_launch();
  const long long id = ids[blockIdx.x];
  const bool ok = id >= 0 && id < vocab;
  if (!ok && threadIdx.x == 0) atomicOr(&g_error_word, AXB200_ERR_BAD_INDEX);
  const T *src = table + (size_t)(ok ? id : 0) * width;
  float sum = 0.f;
  for (int c = threadIdx.x * kVec; c < width; c += kThreads * kVec) {
    float v[kVec];
    load_vec<kVec>(src + c, v);
#pragma unroll
    for (int i = 0; i < kVec; ++i) {
      row[c + i] = ok ? v[i] : 0.f;
      sum += row[c + i];
    }
  }
  const RowStats st = row_stats<kVec>(row, width, sum, eps, scratch);
  for (int c = threadIdx.x * kVec; c < width; c += kThreads * kVec) {
    float v[kVec];
    load_vec<kVec>(w + c, v);
#pragma unroll
    for (int i = 0; i < kVec; ++i) v[i] *= (row[c + i] - st.mean) * st.inv;
    store_vec<kVec>(x + off + c, v);
  }
}

template <typename T>
struct PostNormParams {
  float *x;      // (rows, width), updated in place
  const T *y;    // (rows, width): the sublayer's output
  const T *w;    // its norm
  const T *w2;   // norm of the new x in h, or null: h is x itself
  T *h;          // or null
  float offset;  // added to the stored weights (1 when they are stored around zero)
  float eps;
  int width;
};

template <typename T, int kVec>
__global__ void __launch_bounds__(kThreads) residual_post_norm_kernel(const PostNormParams<T> p) {
  extern __shared__ float row[];
  __shared__ float scratch[32];
  const size_t off = (size_t)blockIdx.x * p.width;
  grid_dependency_wait();
  grid_dependency_launch();
  float sq = 0.f;
  for (int c = threadIdx.x * kVec; c < p.width; c += kThreads * kVec) {
    float v[kVec];
    load_vec<kVec>(p.y + off + c, v);
#pragma unroll
    for (int i = 0; i < kVec; ++i) {
      row[c + i] = v[i];
      sq = fmaf(v[i], v[i], sq);
    }
  }
  const float inv = 1.0f / sqrtf(block_sum(sq, scratch) / (float)p.width + p.eps);
  sq = 0.f;
  for (int c = threadIdx.x * kVec; c < p.width; c += kThreads * kVec) {  // a thread reads back what it wrote
    float v[kVec], w[kVec];
    load_vec<kVec>(p.x + off + c, v);
    load_vec<kVec>(p.w + c, w);
#pragma unroll
    for (int i = 0; i < kVec; ++i) {
      v[i] += row[c + i] * inv * (p.offset + w[i]);
      row[c + i] = v[i];
      sq = fmaf(v[i], v[i], sq);
    }
    store_vec<kVec>(p.x + off + c, v);
    if (p.h && !p.w2) store_vec<kVec>(p.h + off + c, v);
  }
  if (!p.h || !p.w2) return;
  const float inv2 = 1.0f / sqrtf(block_sum(sq, scratch) / (float)p.width + p.eps);
  for (int c = threadIdx.x * kVec; c < p.width; c += kThreads * kVec) {
    float v[kVec], w[kVec];
    load_vec<kVec>(p.w2 + c, w);
#pragma unroll
    for (int i = 0; i < kVec; ++i) v[i] = row[c + i] * inv2 * (p.offset + w[i]);
    store_vec<kVec>(p.h + off + c, v);
  }
}

template <typename T, int kVec>
__global__ void __launch_bounds__(kThreads)
embed_residual_kernel(const int64_t *ids, const T *table, float *x, T *h, long long vocab, int width) {
  const size_t off = (size_t)blockIdx.x * width;
  grid_dependency_wait();
  grid_dependency_launch();
  const long long id = ids[blockIdx.x];
  const bool ok = id >= 0 && id < vocab;
  if (!ok && threadIdx.x == 0) atomicOr(&g_error_word, AXB200_ERR_BAD_INDEX);
  const T *src = table + (size_t)(ok ? id : 0) * width;
  for (int c = threadIdx.x * kVec; c < width; c += kThreads * kVec) {
    float v[kVec];
    load_vec<kVec>(src + c, v);
#pragma unroll
    for (int i = 0; i < kVec; ++i) v[i] = ok ? v[i] : 0.f;
    store_vec<kVec>(x + off + c, v);
    if (h) store_vec<kVec>(h + off + c, v);
  }
}

bool al16(const void *p) { return (reinterpret_cast<uintptr_t>(p) & 15u) == 0; }

constexpr int kMaxWidth = 49152;  // the row is staged in shared memory as fp32

template <typename T>
int launch_residual(const ResidualParams<T> &p, int64_t rows, cudaStream_t st) {
  const bool vec = p.width % 8 == 0 && al16(p.x) && al16(p.a) && al16(p.b) && al16(p.expert_rows) && al16(p.w1) &&
                   al16(p.w2) && al16(p.h1) && al16(p.h2);
  auto *kernel = vec ? residual_layer_norm_kernel<T, 8> : residual_layer_norm_kernel<T, 1>;
  const size_t smem = (size_t)p.width * sizeof(float);
  if (smem > 48 * 1024 && cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
    return AXB200_DEVICE_ERROR;
  return launch_dependent(kernel, dim3((unsigned)rows), dim3(kThreads), smem, st, p);
}

template <typename T>
int launch_embed(const int64_t *ids, const void *table, const void *w, float eps, float *x, int64_t n, int64_t vocab,
                 int width, cudaStream_t st) {
  const bool vec = width % 8 == 0 && al16(table) && al16(w) && al16(x);
  auto *kernel = vec ? embed_layer_norm_kernel<T, 8> : embed_layer_norm_kernel<T, 1>;
  const size_t smem = (size_t)width * sizeof(float);
  if (smem > 48 * 1024 && cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
    return AXB200_DEVICE_ERROR;
  return launch_dependent(kernel, dim3((unsigned)n), dim3(kThreads), smem, st, ids, static_cast<const T *>(table),
                          static_cast<const T *>(w), eps, x, (long long)vocab, width);
}

template <typename T>
int residual_typed(float *x, const void *a, const void *b, const void *expert_rows, const int32_t *slot, const float *weight,
                   int top, const void *w1, void *h1, const void *w2, void *h2, float eps, int64_t rows, int width,
                   cudaStream_t st) {
  ResidualParams<T> p{x, static_cast<const T *>(a), static_cast<const T *>(b), static_cast<const T *>(expert_rows), slot,
                      weight, top, static_cast<const T *>(w1), static_cast<const T *>(w2), static_cast<T *>(h1),
                      static_cast<T *>(h2), eps, width};
  return launch_residual(p, rows, st);
}

template <typename T>
int launch_post_norm(const PostNormParams<T> &p, int64_t rows, cudaStream_t st) {
  const bool vec = p.width % 8 == 0 && al16(p.x) && al16(p.y) && al16(p.w) && al16(p.w2) && al16(p.h);
  auto *kernel = vec ? residual_post_norm_kernel<T, 8> : residual_post_norm_kernel<T, 1>;
  const size_t smem = (size_t)p.width * sizeof(float);
  if (smem > 48 * 1024 && cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
    return AXB200_DEVICE_ERROR;
  return launch_dependent(kernel, dim3((unsigned)rows), dim3(kThreads), smem, st, p);
}

template <typename T>
int launch_embed_residual(const int64_t *ids, const void *table, float *x, void *h, int64_t n, int64_t vocab, int width,
                          cudaStream_t st) {
  const bool vec = width % 8 == 0 && al16(table) && al16(x) && al16(h);
  auto *kernel = vec ? embed_residual_kernel<T, 8> : embed_residual_kernel<T, 1>;
  return launch_dependent(kernel, dim3((unsigned)n), dim3(kThreads), 0, st, ids, static_cast<const T *>(table), x,
                          static_cast<T *>(h), (long long)vocab, width);
}

}  // namespace
}  // namespace axb

extern "C" {

int axb200_embed_residual(const int64_t *ids, const void *table, float *x, void *h, int64_t n, int64_t vocab, int width,
                          int dtype, void *stream) {
  if (dtype != AXB200_FLOAT32 && dtype != AXB200_BFLOAT16) return AXB200_UNSUPPORTED_TYPE;
  if (!ids || !table || !x) return AXB200_INVALID_PTR;
  if (n < 0 || n > 0x7fffffff || vocab <= 0 || width <= 0) return AXB200_INVALID_ARGUMENT;
  if (n == 0) return AXB200_OK;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return dtype == AXB200_FLOAT32 ? axb::launch_embed_residual<float>(ids, table, x, h, n, vocab, width, st)
                                 : axb::launch_embed_residual<__nv_bfloat16>(ids, table, x, h, n, vocab, width, st);
}

int axb200_residual_post_norm(float *x, const void *y, const void *w, float offset, float eps, const void *w2, void *h,
                              int64_t rows, int width, int dtype, void *stream) {
  if (dtype != AXB200_FLOAT32 && dtype != AXB200_BFLOAT16) return AXB200_UNSUPPORTED_TYPE;
  if (!x || !y || !w || (w2 && !h)) return AXB200_INVALID_PTR;
  if (rows < 0 || rows > 0x7fffffff || width <= 0 || width > axb::kMaxWidth) return AXB200_INVALID_ARGUMENT;
  if (rows == 0) return AXB200_OK;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  auto go = [&](auto tag) {
    using T = decltype(tag);
    axb::PostNormParams<T> p{x, static_cast<const T *>(y), static_cast<const T *>(w), static_cast<const T *>(w2),
                             static_cast<T *>(h), offset, eps, width};
    return axb::launch_post_norm(p, rows, st);
  };
  return dtype == AXB200_FLOAT32 ? go(float{}) : go(__nv_bfloat16{});
}

int axb200_embed_layer_norm(const int64_t *ids, const void *table, const void *weight, float eps, float *x, int64_t n,
                            int64_t vocab, int width, int dtype, void *stream) {
  if (dtype != AXB200_FLOAT32 && dtype != AXB200_BFLOAT16) return AXB200_UNSUPPORTED_TYPE;
  if (!ids || !table || !weight || !x) return AXB200_INVALID_PTR;
  if (n < 0 || n > 0x7fffffff || vocab <= 0 || width <= 0 || width > axb::kMaxWidth) return AXB200_INVALID_ARGUMENT;
  if (n == 0) return AXB200_OK;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return dtype == AXB200_FLOAT32 ? axb::launch_embed<float>(ids, table, weight, eps, x, n, vocab, width, st)
                                 : axb::launch_embed<__nv_bfloat16>(ids, table, weight, eps, x, n, vocab, width, st);
}

int axb200_residual_layer_norm(float *x, const void *a, const void *b, const void *expert_rows, const int32_t *slot,
                               const float *weight, int top, const void *w1, void *h1, const void *w2, void *h2, float eps,
                               int64_t rows, int width, int dtype, void *stream) {
  if (dtype != AXB200_FLOAT32 && dtype != AXB200_BFLOAT16) return AXB200_UNSUPPORTED_TYPE;
  if (!x || (w1 && !h1) || (w2 && !h2) || (expert_rows && (!slot || !weight))) return AXB200_INVALID_PTR;
  if (rows < 0 || rows > 0x7fffffff || width <= 0 || width > axb::kMaxWidth || (expert_rows && top <= 0))
    return AXB200_INVALID_ARGUMENT;
  if (rows == 0) return AXB200_OK;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return dtype == AXB200_FLOAT32
             ? axb::residual_typed<float>(x, a, b, expert_rows, slot, weight, top, w1, h1, w2, h2, eps, rows, width, st)
             : axb::residual_typed<__nv_bfloat16>(x, a, b, expert_rows, slot, weight, top, w1, h1, w2, h2, eps, rows, width, st);
}

}  // extern "C"
