// Grouped attention whose values are the keys as projected: the cache holds kv_heads rows of dim raw key elements per
// token, head by head within a page, and a page ends with one fp32 factor per token.  The factor, 1 / rms of all the
// token's elements, makes the rows the normed keys.  The key norm's weight is folded into
// the queries, so a score is factor_j * (q' . k_j) and a value is k_j itself: one read of the row serves both, where a
// cache of keys and values would take two.  The attention over these rows is latent_attn.cu / latent_umma.cu; for long
// portions of prompts the rows are gathered into normed keys and raw values for the kernel of latent_prefill.cu.
#include "vec.cuh"

namespace axb {
namespace {

constexpr int kThreads = 256;

template <typename T>
__host__ __device__ constexpr size_t page_elems(int page_tokens, int elems) {
  return (size_t)page_tokens * (elems + sizeof(float) / sizeof(T));
}

template <typename T>
struct SharedKvParams {
  const T *q;  // (rows, q_ld): heads * dim
  int64_t q_ld;
  const T *q_w;  // (heads * dim)
  T *q_out;      // (rows, heads * dim): normed, times q_w and the key norm's weight
  const T *k;    // (rows, k_ld): kv_heads * dim
  int64_t k_ld;
  const T *k_w;  // (kv_heads * dim)
  T *pages;      // per page: (kv_heads, page_tokens, dim) and page_tokens fp32 factors
  const int32_t *block_table, *row_seq, *row_pos;
  int heads, kv_heads, dim, max_blocks, page_tokens, num_pages, max_seqs;
  float eps;
};

// One CTA per row: both norms run over all heads of the row.
template <typename T, int kVec>
__global__ void __launch_bounds__(kThreads) shared_kv_prepare_kernel(const SharedKvParams<T> p) {
  __shared__ float scratch[32];
  const int64_t r = blockIdx.x;
  grid_dependency_wait();
  grid_dependency_launch();
  const int nq = p.heads * p.dim, nk = p.kv_heads * p.dim, group_elems = nq / p.kv_heads;
  const T *q = p.q + r * p.q_ld, *k = p.k + r * p.k_ld;
  float v[kVec], w[kVec], f[kVec], sq = 0.f, sk = 0.f;
  for (int i = threadIdx.x * kVec; i < nq; i += kThreads * kVec) {
    load_vec<kVec>(q + i, v);
#pragma unroll
    for (int e = 0; e < kVec; ++e) sq = fmaf(v[e], v[e], sq);
  }
  for (int i = threadIdx.x * kVec; i < nk; i += kThreads * kVec) {
    load_vec<kVec>(k + i, v);
#pragma unroll
    for (int e = 0; e < kVec; ++e) sk = fmaf(v[e], v[e], sk);
  }
  const float inv_q = 1.0f / sqrtf(block_sum(sq, scratch) / (float)nq + p.eps);
  const float inv_k = 1.0f / sqrtf(block_sum(sk, scratch) / (float)nk + p.eps);
  for (int i = threadIdx.x * kVec; i < nq; i += kThreads * kVec) {
    load_vec<kVec>(q + i, v);
    load_vec<kVec>(p.q_w + i, w);
    load_vec<kVec>(p.k_w + i / group_elems * p.dim + i % p.dim, f);
#pragma unroll
    for (int e = 0; e < kVec; ++e) v[e] = v[e] * inv_q * w[e] * f[e];
    store_vec<kVec>(p.q_out + r * nq + i, v);
  }
  const int seq = p.row_seq[r], pos = p.row_pos[r], blk = pos / p.page_tokens;
  if (seq < 0 || seq >= p.max_seqs || pos < 0 || blk >= p.max_blocks) {
    if (threadIdx.x == 0) atomicOr(&g_error_word, AXB200_ERR_CAPACITY);
    return;
  }
  const int page = p.block_table[(size_t)seq * p.max_blocks + blk];
  if (page < 0 || page >= p.num_pages) {
    if (threadIdx.x == 0) atomicOr(&g_error_word, AXB200_ERR_BAD_PAGE);
    return;
  }
  T *base = p.pages + page * page_elems<T>(p.page_tokens, nk);
  for (int i = threadIdx.x * kVec; i < nk; i += kThreads * kVec) {
    load_vec<kVec>(k + i, v);
    store_vec<kVec>(base + ((size_t)(i / p.dim) * p.page_tokens + pos % p.page_tokens) * p.dim + i % p.dim, v);
  }
  if (threadIdx.x == 0) reinterpret_cast<float *>(base + (size_t)p.page_tokens * nk)[pos % p.page_tokens] = inv_k;
}

// Cached rows first .. first + n - 1 of one sequence as normed keys and raw values, both (n, elems); a warp per row.
template <typename T, int kVec>
__global__ void __launch_bounds__(kThreads)
shared_kv_gather_kernel(const T *pages, const int32_t *table, T *keys, T *values, int first, int n, int elems, int dim, int page_tokens, int max_blocks, int num_pages) {
  grid_dependency_wait();
  grid_dependency_launch();
  const int lane = threadIdx.x & 31;
  for (int r = blockIdx.x * (kThreads / 32) + (threadIdx.x >> 5); r < n; r += gridDim.x * (kThreads / 32)) {
    const int t = first + r, blk = t / page_tokens, page = blk < max_blocks ? table[blk] : -1;
    if (page < 0 || page >= num_pages) {
      if (lane == 0) atomicOr(&g_error_word, AXB200_ERR_BAD_PAGE);
      continue;
    }
    const T *base = pages + page * page_elems<T>(page_tokens, elems);
    const float inv = reinterpret_cast<const float *>(base + (size_t)page_tokens * elems)[t % page_tokens];
    for (int i = lane * kVec; i < elems; i += 32 * kVec) {
      float v[kVec];
      load_vec<kVec>(base + ((size_t)(i / dim) * page_tokens + t % page_tokens) * dim + i % dim, v);
      store_vec<kVec>(values + (size_t)r * elems + i, v);
#pragma unroll
      for (int e = 0; e < kVec; ++e) v[e] *= inv;
      store_vec<kVec>(keys + (size_t)r * elems + i, v);
    }
  }
}

bool al16(const void *p) { return (reinterpret_cast<uintptr_t>(p) & 15u) == 0; }

// the factors are aligned floats
bool page_ok(int kv_heads, int dim, int page_tokens, int dtype) {
  return (int64_t)kv_heads * dim * page_tokens * (int64_t)dtype_size(dtype) % 4 == 0;
}

}  // namespace
}  // namespace axb

extern "C" {

int axb200_shared_kv_prepare(const void *q, int64_t q_ld, const void *q_w, void *q_out, const void *k, int64_t k_ld,
                             const void *k_w, float eps, void *pages, const int32_t *block_table, const int32_t *row_seq,
                             const int32_t *row_pos, int64_t rows, int heads, int kv_heads, int dim, int page_tokens, int max_blocks, int num_pages, int max_seqs, int dtype, void *stream) {
  if (dtype != AXB200_FLOAT32 && dtype != AXB200_BFLOAT16) return AXB200_UNSUPPORTED_TYPE;
  if (!q || !q_w || !q_out || !k || !k_w || !pages || !block_table || !row_seq || !row_pos) return AXB200_INVALID_PTR;
  if (rows < 0 || rows > 0x7fffffff || heads <= 0 || kv_heads <= 0 || heads % kv_heads != 0 || dim <= 0 || page_tokens <= 0 ||
      max_blocks <= 0 || num_pages <= 0 || max_seqs <= 0 || !axb::page_ok(kv_heads, dim, page_tokens, dtype))
    return AXB200_INVALID_ARGUMENT;
  if (q_ld < (int64_t)heads * dim || k_ld < (int64_t)kv_heads * dim) return AXB200_SHAPE_MISMATCH;
  if (rows == 0) return AXB200_OK;
  auto go = [&](auto tag) {
    using T = decltype(tag);
    axb::SharedKvParams<T> p{static_cast<const T *>(q), q_ld, static_cast<const T *>(q_w), static_cast<T *>(q_out),
                             static_cast<const T *>(k), k_ld, static_cast<const T *>(k_w), static_cast<T *>(pages), block_table,
                             row_seq, row_pos, heads, kv_heads, dim, max_blocks, page_tokens, num_pages,
                             max_seqs, eps};
    const bool vec = dim % 8 == 0 && q_ld % 8 == 0 && k_ld % 8 == 0 && page_tokens % 8 == 0 && axb::al16(q) && axb::al16(q_w) &&
                     axb::al16(q_out) && axb::al16(k) && axb::al16(k_w) && axb::al16(pages);
    auto *kernel = vec ? axb::shared_kv_prepare_kernel<T, 8> : axb::shared_kv_prepare_kernel<T, 1>;
    return axb::launch_dependent(kernel, dim3((unsigned)rows), dim3(axb::kThreads), 0, static_cast<cudaStream_t>(stream), p);
  };
  return dtype == AXB200_FLOAT32 ? go(float{}) : go(__nv_bfloat16{});
}

int axb200_shared_kv_gather(const void *pages, const int32_t *block_row, void *keys, void *values, int64_t first, int64_t n,
                            int kv_heads, int dim, int page_tokens, int max_blocks, int num_pages,
                            int dtype, void *stream) {
  if (dtype != AXB200_FLOAT32 && dtype != AXB200_BFLOAT16) return AXB200_UNSUPPORTED_TYPE;
  if (!pages || !block_row || !keys || !values) return AXB200_INVALID_PTR;
  if (n < 0 || first < 0 || first + n > (int64_t)max_blocks * page_tokens || kv_heads <= 0 || dim <= 0 || page_tokens <= 0 ||
      max_blocks <= 0 || num_pages <= 0 || !axb::page_ok(kv_heads, dim, page_tokens, dtype))
    return AXB200_INVALID_ARGUMENT;
  if (n == 0) return AXB200_OK;
  auto go = [&](auto tag) {
    using T = decltype(tag);
    const int elems = kv_heads * dim;
    const bool vec = dim % 8 == 0 && page_tokens % 8 == 0 && axb::al16(pages) && axb::al16(keys) && axb::al16(values);
    auto *kernel = vec ? axb::shared_kv_gather_kernel<T, 8> : axb::shared_kv_gather_kernel<T, 1>;
    const int64_t want = (n + axb::kThreads / 32 - 1) / (axb::kThreads / 32);
    return axb::launch_dependent(kernel, dim3((unsigned)(want < 148 * 8 ? want : 148 * 8)), dim3(axb::kThreads), 0,
                                 static_cast<cudaStream_t>(stream), static_cast<const T *>(pages), block_row,
                                 static_cast<T *>(keys), static_cast<T *>(values), (int)first, (int)n, elems, dim,
                                 page_tokens, max_blocks, num_pages);
  };
  return dtype == AXB200_FLOAT32 ? go(float{}) : go(__nv_bfloat16{});
}

}  // extern "C"
