// Attention over a cache of latents: every token caches one row [c (kv_rank) | rotated key part (rot_dim)] that
// all heads share, and a head's key and value are linear maps of c.  Folding the key map into the query
// (q_lat = q . W_uk) and the value map behind the sum turns it into attention of H queries per token over ONE
// key row of kv_rank + rot_dim elements whose first kv_rank elements are also the value:
//     score = (q_lat . c + q_rot . k_rot) * scale,   out_lat = sum softmax(score) c.
// This file holds the step's norms, rotation and append in one launch; the attention for fp32 and for sizes
// that the tensor-core form (latent_umma.cu) does not take; and the gather that the expanded form
// (latent_prefill.cu) reads from.
//
// Rows are independent: row r belongs to sequence row_seq[r] (its block-table row) and sees the cached tokens
// 0 .. row_pos[r], or the last `window` of them, so one launch serves decode batches, portions of prompts and
// mixtures of both.  A per-head sink may join the denominator.
//
// The same kernels attend plain cached keys that are also the values: kv_heads rows per token, each read by its group of
// query heads, and a factor per token, behind the rows of its page, that turns its keys - not its values - into normed ones (shared_kv.cu).
#include <math.h>

#include "latent_attn.cuh"

namespace axb {
namespace {

// ---- norms, rotation, append -----------------------------------------------------------------------
template <typename T>
struct PrepareParams {
  T *q;  // (rows, q_ld): heads of [dim plain | rot_dim rotated], rotated in place; null: none
  int64_t q_ld;
  int heads, dim;
  const T *dq;  // (rows, dq_ld): query latent to norm into cq (rows, q_rank); null: none
  int64_t dq_ld;
  int q_rank;
  const T *dq_w;
  T *cq;
  const T *dkv;  // (rows, dkv_ld): [kv_rank | rot_dim] to norm, rotate and append; null: none
  int64_t dkv_ld;
  int kv_rank;
  const T *dkv_w;
  T *pages;  // (num_pages, page_tokens, kv_rank + rot_dim)
  const int32_t *block_table, *row_seq, *row_pos;
  const double *inv_freq;  // (rot_pairs)
  int rot_dim, rot_pairs, max_blocks, page_tokens, num_pages, max_seqs;
  float eps;
};

constexpr int kPrepThreads = 256, kMaxRotPairs = 256;

// One CTA per row.  The angle position * frequency is formed and reduced to one turn in double, so that far
// positions lose nothing; its sine and cosine are evaluated in fp32, once per pair for all heads.
template <typename T>
__global__ void __launch_bounds__(kPrepThreads) latent_prepare_kernel(const PrepareParams<T> p) {
  __shared__ float scratch[32], cs[kMaxRotPairs], sn[kMaxRotPairs];
  const int64_t r = blockIdx.x;
  grid_dependency_wait();
  grid_dependency_launch();
  const int pos = p.row_pos[r];
  for (int i = threadIdx.x; i < p.rot_pairs; i += kPrepThreads) {
    const double turns = (double)pos * p.inv_freq[i] * 0.15915494309189533577;  // 1 / (2 pi)
    const float a = (float)((turns - rint(turns)) * 6.28318530717958647692);
    sincosf(a, &sn[i], &cs[i]);
  }
  __syncthreads();
  if (p.q) {
    const int per = p.rot_pairs, n = p.heads * per;
    for (int i = threadIdx.x; i < n; i += kPrepThreads) {
      const int h = i / per, j = i % per;
      T *e = p.q + r * p.q_ld + (int64_t)h * (p.dim + p.rot_dim) + p.dim + 2 * j;
      const float u = ldf(e), v = ldf(e + 1);
      stf(e, u * cs[j] - v * sn[j]);
      stf(e + 1, v * cs[j] + u * sn[j]);
    }
  }
  if (p.dq) {
    const T *src = p.dq + r * p.dq_ld;
    float sq = 0.f;
    for (int i = threadIdx.x; i < p.q_rank; i += kPrepThreads) {
      const float v = ldf(src + i);
      sq = fmaf(v, v, sq);
    }
    const float inv = 1.0f / sqrtf(block_sum(sq, scratch) / (float)p.q_rank + p.eps);
    for (int i = threadIdx.x; i < p.q_rank; i += kPrepThreads)
      stf(p.cq + r * p.q_rank + i, ldf(src + i) * inv * ldf(p.dq_w + i));
  }
  if (p.dkv) {
    const T *src = p.dkv + r * p.dkv_ld;
    float sq = 0.f;
    for (int i = threadIdx.x; i < p.kv_rank; i += kPrepThreads) {
      const float v = ldf(src + i);
      sq = fmaf(v, v, sq);
    }
    const float inv = 1.0f / sqrtf(block_sum(sq, scratch) / (float)p.kv_rank + p.eps);
    const int seq = p.row_seq[r], blk = pos / p.page_tokens;
    if (seq < 0 || seq >= p.max_seqs || pos < 0 || blk >= p.max_blocks) {
      if (threadIdx.x == 0) atomicOr(&g_error_word, AXB200_ERR_CAPACITY);
      return;
    }
    const int page = p.block_table[(size_t)seq * p.max_blocks + blk];
    if (page < 0 || page >= p.num_pages) {
      if (threadIdx.x == 0) atomicOr(&g_error_word, AXB200_ERR_BAD_PAGE);
      return;
    }
    T *dst = p.pages + ((size_t)page * p.page_tokens + pos % p.page_tokens) * (p.kv_rank + p.rot_dim);
    for (int i = threadIdx.x; i < p.kv_rank; i += kPrepThreads) stf(dst + i, ldf(src + i) * inv * ldf(p.dkv_w + i));
    src += p.kv_rank;
    dst += p.kv_rank;
    for (int j = threadIdx.x; j < p.rot_pairs; j += kPrepThreads) {
      const float u = ldf(src + 2 * j), v = ldf(src + 2 * j + 1);
      stf(dst + 2 * j, u * cs[j] - v * sn[j]);
      stf(dst + 2 * j + 1, v * cs[j] + u * sn[j]);
    }
    for (int i = 2 * p.rot_pairs + threadIdx.x; i < p.rot_dim; i += kPrepThreads) stf(dst + i, ldf(src + i));
  }
}

// bf16 with sizes and addresses that allow 16-byte accesses and at most 32 rotated pairs: one CTA per row, its warps
// take turns at the row's jobs - the cached row, the query latent, then 32 chunks of 8 query elements at a time.
// Lane i holds the sine and cosine of pair i; the sums of the norms stay inside a warp.
constexpr int kPrepVecWarps = 4;

struct Bf16x8 {
  uint4 raw;
  __device__ __forceinline__ void get(float (&v)[8]) const {
    const __nv_bfloat16 *e = reinterpret_cast<const __nv_bfloat16 *>(&raw);
#pragma unroll
    for (int i = 0; i < 8; ++i) v[i] = __bfloat162float(e[i]);
  }
  __device__ __forceinline__ void set(const float (&v)[8]) {
    raw = make_uint4(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]), pack_bf16x2(v[4], v[5]), pack_bf16x2(v[6], v[7]));
  }
};

__global__ void __launch_bounds__(kPrepVecWarps * 32, 9) latent_prepare_vec_kernel(const PrepareParams<__nv_bfloat16> p) {
  const int64_t r = blockIdx.x;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  grid_dependency_wait();
  grid_dependency_launch();
  const int pos = p.row_pos[r];
  // what a warp needs first is on its way while the angles are evaluated
  const int rot_chunks = p.rot_dim / 8, q_chunks = p.q ? p.heads * rot_chunks : 0;
  auto q_chunk = [&](int i) {  // address of chunk i of the rotated query parts
    const int h = i / rot_chunks;
    return p.q + r * p.q_ld + (int64_t)h * (p.dim + p.rot_dim) + p.dim + (i - h * rot_chunks) * 8;
  };
  const int first_q = warp < 2 ? warp + kPrepVecWarps : warp;  // the first of this warp's jobs from 2 on
  Bf16x8 ahead;
  ahead.raw = make_uint4(0, 0, 0, 0);
  if ((first_q - 2) * 32 + lane < q_chunks) ahead.raw = *reinterpret_cast<const uint4 *>(q_chunk((first_q - 2) * 32 + lane));
  Bf16x8 ahead_norm[2];  // warp 0: of the row to cache, warp 1: of the query latent
#pragma unroll
  for (int k = 0; k < 2; ++k) {
    const int e = (k * 32 + lane) * 8;
    ahead_norm[k].raw = make_uint4(0, 0, 0, 0);
    if (warp == 0 && p.dkv && e < p.kv_rank) ahead_norm[k].raw = *reinterpret_cast<const uint4 *>(p.dkv + r * p.dkv_ld + e);
    if (warp == 1 && p.dq && e < p.q_rank) ahead_norm[k].raw = *reinterpret_cast<const uint4 *>(p.dq + r * p.dq_ld + e);
  }
  float c = 1.f, s = 0.f;
  if (lane < p.rot_pairs) {
    const double turns = (double)pos * p.inv_freq[lane] * 0.15915494309189533577;  // 1 / (2 pi)
    sincosf((float)((turns - rint(turns)) * 6.28318530717958647692), &s, &c);
  }
  // chunk j of a rotated part: pairs 4j .. 4j + 3 (all lanes take part)
  auto rotate = [&](float (&v)[8], int j) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float ci = __shfl_sync(0xffffffffu, c, (4 * j + i) & 31), si = __shfl_sync(0xffffffffu, s, (4 * j + i) & 31);
      const float u = v[2 * i], w = v[2 * i + 1];
      v[2 * i] = u * ci - w * si;
      v[2 * i + 1] = w * ci + u * si;
    }
  };
  auto norm = [&](const __nv_bfloat16 *src, const __nv_bfloat16 *weight, __nv_bfloat16 *dst, int n) {
    // the first 512 elements are in registers, the rest is read twice, the second time from L1: holding more would
    // cost the registers that keep enough rows in flight
    float v[8], sq = 0.f;
    auto square = [&](const Bf16x8 &x) {
      x.get(v);
#pragma unroll
      for (int i = 0; i < 8; ++i) sq = fmaf(v[i], v[i], sq);
    };
#pragma unroll
    for (int k = 0; k < 2; ++k) square(ahead_norm[k]);  // zeros past the end
    Bf16x8 x;
    for (int e = 512 + lane * 8; e < n; e += 256) {
      x.raw = *reinterpret_cast<const uint4 *>(src + e);
      square(x);
    }
    const float inv = 1.0f / sqrtf(warp_sum(sq) / (float)n + p.eps);
    auto scale_store = [&](Bf16x8 x, int e) {
      Bf16x8 ww;
      float w[8];
      ww.raw = *reinterpret_cast<const uint4 *>(weight + e);
      x.get(v);
      ww.get(w);
#pragma unroll
      for (int i = 0; i < 8; ++i) v[i] = v[i] * inv * w[i];
      x.set(v);
      *reinterpret_cast<uint4 *>(dst + e) = x.raw;
    };
#pragma unroll
    for (int k = 0; k < 2; ++k)
      if ((k * 32 + lane) * 8 < n) scale_store(ahead_norm[k], (k * 32 + lane) * 8);
    for (int e = 512 + lane * 8; e < n; e += 256) {
      x.raw = *reinterpret_cast<const uint4 *>(src + e);
      scale_store(x, e);
    }
  };
  for (int job = warp;; job += kPrepVecWarps) {
    if (job == 0) {
      if (!p.dkv) continue;
      const int seq = p.row_seq[r], blk = pos / p.page_tokens;
      if (seq < 0 || seq >= p.max_seqs || pos < 0 || blk >= p.max_blocks) {
        if (lane == 0) atomicOr(&g_error_word, AXB200_ERR_CAPACITY);
        continue;
      }
      const int page = p.block_table[(size_t)seq * p.max_blocks + blk];
      if (page < 0 || page >= p.num_pages) {
        if (lane == 0) atomicOr(&g_error_word, AXB200_ERR_BAD_PAGE);
        continue;
      }
      const __nv_bfloat16 *src = p.dkv + r * p.dkv_ld;
      __nv_bfloat16 *dst = p.pages + ((size_t)page * p.page_tokens + pos % p.page_tokens) * (p.kv_rank + p.rot_dim);
      norm(src, p.dkv_w, dst, p.kv_rank);
      Bf16x8 x;
      float v[8] = {};
      if (lane < rot_chunks) {
        x.raw = *reinterpret_cast<const uint4 *>(src + p.kv_rank + lane * 8);
        x.get(v);
      }
      rotate(v, lane);
      if (lane < rot_chunks) {
        x.set(v);
        *reinterpret_cast<uint4 *>(dst + p.kv_rank + lane * 8) = x.raw;
      }
    } else if (job == 1) {
      if (p.dq) norm(p.dq + r * p.dq_ld, p.dq_w, p.cq + r * p.q_rank, p.q_rank);
    } else {
      const int i = (job - 2) * 32 + lane;
      if ((job - 2) * 32 >= q_chunks) break;
      Bf16x8 x = ahead;
      if (job != first_q && i < q_chunks) x.raw = *reinterpret_cast<const uint4 *>(q_chunk(i));
      float v[8];
      x.get(v);
      rotate(v, i % rot_chunks);
      if (i < q_chunks) {
        x.set(v);
        *reinterpret_cast<uint4 *>(q_chunk(i)) = x.raw;
      }
    }
  }
}

bool prepare_vec_takes(const PrepareParams<__nv_bfloat16> &p) {
  const auto al = [](const void *q) { return (reinterpret_cast<uintptr_t>(q) & 15u) == 0; };
  return p.rot_pairs <= 32 && p.rot_dim % 8 == 0 && p.rot_pairs * 2 == p.rot_dim &&
         (!p.q || (al(p.q) && p.dim % 8 == 0 && p.q_ld % 8 == 0)) &&
         (!p.dq || (al(p.dq) && al(p.dq_w) && al(p.cq) && p.q_rank % 8 == 0 && p.dq_ld % 8 == 0)) &&
         (!p.dkv || (al(p.dkv) && al(p.dkv_w) && al(p.pages) && p.kv_rank % 8 == 0 && p.dkv_ld % 8 == 0));
}

// ---- attention in latent form -------------------------------------------------------------------------
// Any size, fp32 or bf16: one CTA per (row, head); 64 keys at a time, one warp per key for the scores, one
// thread per latent element for the sum.  fp32 arithmetic throughout.
constexpr int kGenThreads = 256, kGenTile = 64;

template <typename T>
__global__ void __launch_bounds__(kGenThreads) latent_attend_generic_kernel(const AttendParams p) {
  extern __shared__ float sm[];
  __shared__ float scratch[32], score[kGenTile], factor[kGenTile];
  __shared__ const T *key[kGenTile];
  const int part_elems = p.kv_rank + p.rot_dim;
  float *q = sm, *acc = sm + part_elems;
  const int r = blockIdx.x, h = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const size_t part = (size_t)(h / (p.heads / p.kv_heads)) * p.page_tokens;
  grid_dependency_wait();
  grid_dependency_launch();
  const T *ql = static_cast<const T *>(p.q_lat) + ((size_t)r * p.heads + h) * p.kv_rank;
  const T *qr = static_cast<const T *>(p.q) + (size_t)r * p.q_ld + (size_t)h * (p.dim + p.rot_dim) + p.dim;
  for (int i = threadIdx.x; i < part_elems; i += kGenThreads) q[i] = i < p.kv_rank ? ldf(ql + i) : ldf(qr + i - p.kv_rank);
  for (int i = threadIdx.x; i < p.kv_rank; i += kGenThreads) acc[i] = 0.f;
  const int keys = visible_keys(p, r);
  const int32_t *table = p.block_table + (size_t)max(0, min(p.row_seq[r], p.max_seqs - 1)) * p.max_blocks;
  const T *pages = static_cast<const T *>(p.pages);
  float m = p.sink ? p.sink[h] : -INFINITY, l = p.sink ? 1.f : 0.f;
  for (int k0 = first_key(p, r); k0 < keys; k0 += kGenTile) {
    const int n = min(kGenTile, keys - k0);
    __syncthreads();
    if (threadIdx.x < n) {
      const int t = k0 + threadIdx.x;
      int page = table[t / p.page_tokens];
      if (page < 0 || page >= p.num_pages) {
        atomicOr(&g_error_word, AXB200_ERR_BAD_PAGE);
        page = 0;
      }
      const T *base = pages + (size_t)page * p.page_elems;
      key[threadIdx.x] = base + (part + t % p.page_tokens) * p.row_elems;
      factor[threadIdx.x] = p.key_scale ? p.scale * page_factors(base, p)[t % p.page_tokens] : p.scale;
    }
    __syncthreads();
    for (int j = warp; j < n; j += kGenThreads / 32) {
      float s = 0.f;
      for (int i = lane; i < part_elems; i += 32) s = fmaf(q[i], ldf(key[j] + i), s);
      s = warp_sum(s);
      if (lane == 0) score[j] = s * factor[j];
    }
    __syncthreads();
    float mt = m;
    for (int j = 0; j < n; ++j) mt = fmaxf(mt, score[j]);
    const float corr = expf(m - mt);  // 0 at the first tile without a sink
    m = mt;
    __syncthreads();
    if (threadIdx.x < n) score[threadIdx.x] = expf(score[threadIdx.x] - m);
    __syncthreads();
    l = l * corr + block_sum(threadIdx.x < n ? score[threadIdx.x] : 0.f, scratch);
    for (int i = threadIdx.x; i < p.kv_rank; i += kGenThreads) {
      float a = acc[i] * corr;
      for (int j = 0; j < n; ++j) a = fmaf(score[j], ldf(key[j] + i), a);
      acc[i] = a;
    }
  }
  const float inv = l > 0.f ? 1.0f / l : 0.f;
  T *out = static_cast<T *>(p.out) + ((size_t)r * p.heads + h) * p.kv_rank;
  for (int i = threadIdx.x; i < p.kv_rank; i += kGenThreads) stf(out + i, acc[i] * inv);
}

// ---- gather: cached rows first .. first + n - 1 of one sequence, contiguous -----------------------------------------
__global__ void __launch_bounds__(256)
latent_gather_kernel(const uint8_t *pages, const int32_t *table, uint8_t *out, int first, int n, int row_bytes, int page_tokens,
                     int max_blocks, int num_pages, int unit) {
  grid_dependency_wait();
  grid_dependency_launch();
  const int per = row_bytes / unit;
  const int64_t total = (int64_t)n * per;
  for (int64_t i = blockIdx.x * 256ll + threadIdx.x; i < total; i += gridDim.x * 256ll) {
    const int t = first + (int)(i / per), c = (int)(i % per), blk = t / page_tokens;
    const int page = blk < max_blocks ? table[blk] : -1;
    if (page < 0 || page >= num_pages) {
      atomicOr(&g_error_word, AXB200_ERR_BAD_PAGE);
      continue;
    }
    const uint8_t *src = pages + ((size_t)page * page_tokens + t % page_tokens) * row_bytes + (size_t)c * unit;
    uint8_t *dst = out + (size_t)(t - first) * row_bytes + (size_t)c * unit;
    if (unit == 16)
      *reinterpret_cast<uint4 *>(dst) = *reinterpret_cast<const uint4 *>(src);
    else
      *reinterpret_cast<uint16_t *>(dst) = *reinterpret_cast<const uint16_t *>(src);
  }
}

}  // namespace
}  // namespace axb

extern "C" {

int axb200_latent_prepare(void *q, int64_t q_ld, int heads, int dim, const void *dq, int64_t dq_ld, int q_rank,
                          const void *dq_w, void *cq, const void *dkv, int64_t dkv_ld, int kv_rank, const void *dkv_w,
                          float eps, void *pages, const int32_t *block_table, const int32_t *row_seq,
                          const int32_t *row_pos, const double *inv_freq, int rot_dim, int rot_pairs, int64_t rows,
                          int page_tokens, int max_blocks, int num_pages, int max_seqs, int dtype, void *stream) {
  if (dtype != AXB200_FLOAT32 && dtype != AXB200_BFLOAT16) return AXB200_UNSUPPORTED_TYPE;
  if (!row_pos || (rot_pairs > 0 && !inv_freq) || (dq && (!dq_w || !cq)) ||
      (dkv && (!dkv_w || !pages || !block_table || !row_seq)))
    return AXB200_INVALID_PTR;
  if (rows < 0 || rows > 0x7fffffff || rot_pairs < 0 || rot_pairs > axb::kMaxRotPairs || 2 * rot_pairs > rot_dim ||
      (q && (heads <= 0 || dim < 0)) || (dq && q_rank <= 0) ||
      (dkv && (kv_rank <= 0 || page_tokens <= 0 || max_blocks <= 0 || num_pages <= 0 || max_seqs <= 0)))
    return AXB200_INVALID_ARGUMENT;
  if ((q && q_ld < (int64_t)heads * (dim + rot_dim)) || (dq && dq_ld < q_rank) || (dkv && dkv_ld < kv_rank + rot_dim))
    return AXB200_SHAPE_MISMATCH;
  if (rows == 0) return AXB200_OK;
  auto go = [&](auto tag) {
    using T = decltype(tag);
    axb::PrepareParams<T> p{static_cast<T *>(q), q_ld, heads, dim, static_cast<const T *>(dq), dq_ld, q_rank,
                            static_cast<const T *>(dq_w), static_cast<T *>(cq), static_cast<const T *>(dkv), dkv_ld, kv_rank,
                            static_cast<const T *>(dkv_w), static_cast<T *>(pages), block_table, row_seq, row_pos, inv_freq,
                            rot_dim, rot_pairs, max_blocks, page_tokens, num_pages, max_seqs, eps};
    if constexpr (sizeof(T) == 2) {
      if (axb::prepare_vec_takes(p))
        return axb::launch_dependent(axb::latent_prepare_vec_kernel, dim3((unsigned)rows), dim3(axb::kPrepVecWarps * 32), 0,
                                     static_cast<cudaStream_t>(stream), p);
    }
    return axb::launch_dependent(axb::latent_prepare_kernel<T>, dim3((unsigned)rows), dim3(axb::kPrepThreads), 0,
                                 static_cast<cudaStream_t>(stream), p);
  };
  return dtype == AXB200_FLOAT32 ? go(float{}) : go(__nv_bfloat16{});
}

size_t axb200_latent_attend_workspace_bytes(int rows, int heads, int kv_rank, int rot_dim, int64_t max_len, int dtype) {
  if (rows <= 0 || heads <= 0 || kv_rank <= 0 || dtype != AXB200_BFLOAT16) return 0;
  return axb::latent_umma_workspace_bytes(heads, kv_rank, rot_dim);
}

int axb200_latent_attend(const void *q_lat, const void *q, int64_t q_ld, int dim, void *out, const void *pages,
                         const int32_t *block_table, const int32_t *row_seq, const int32_t *row_pos, const float *sink,
                         int rows, int heads, int kv_heads, int kv_rank, int rot_dim, int key_scale, int window,
                         float scale, int page_tokens, int max_blocks, int num_pages, int max_seqs, int64_t max_len, int dtype,
                         void *workspace, size_t workspace_bytes, void *stream) {
  if (dtype != AXB200_FLOAT32 && dtype != AXB200_BFLOAT16) return AXB200_UNSUPPORTED_TYPE;
  if (!q_lat || (!q && rot_dim > 0) || !out || !pages || !block_table || !row_seq || !row_pos) return AXB200_INVALID_PTR;
  if (kv_heads <= 0 || heads % kv_heads != 0 || (kv_heads > 1 && rot_dim > 0) || window < 0) return AXB200_INVALID_ARGUMENT;
  if (rows < 0 || heads <= 0 || heads > 65535 || kv_rank <= 0 || rot_dim < 0 || dim < 0 || page_tokens <= 0 || max_blocks <= 0 ||
      num_pages <= 0 || max_seqs <= 0 || max_len <= 0 || max_len > 0x7fffffff - 4096)
    return AXB200_INVALID_ARGUMENT;
  if (rot_dim > 0 && q_ld < (int64_t)heads * (dim + rot_dim)) return AXB200_SHAPE_MISMATCH;
  if (rows == 0) return AXB200_OK;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  axb::AttendParams p{};
  p.kv_heads = kv_heads;
  p.row_elems = kv_rank + rot_dim;
  p.page_elems = page_tokens * kv_heads * p.row_elems + (key_scale ? page_tokens * (4 / (int)axb::dtype_size(dtype)) : 0);
  p.key_scale = key_scale;
  p.window = window;
  p.sink = sink;
  p.q_lat = q_lat;
  p.q = q;
  p.q_ld = q_ld;
  p.out = out;
  p.pages = pages;
  p.block_table = block_table;
  p.row_seq = row_seq;
  p.row_pos = row_pos;
  p.rows = rows;
  p.heads = heads;
  p.dim = dim;
  p.kv_rank = kv_rank;
  p.rot_dim = rot_dim;
  p.page_tokens = page_tokens;
  p.max_blocks = max_blocks;
  p.num_pages = num_pages;
  p.max_seqs = max_seqs;
  p.max_len = (int)max_len;
  p.scale = scale;
  p.wait_ns = axb::wait_limit_ns();
  if (dtype == AXB200_BFLOAT16 && axb::latent_umma_supported(p)) {
    if (!workspace || workspace_bytes < axb200_latent_attend_workspace_bytes(rows, heads / kv_heads, kv_rank, rot_dim, max_len, dtype))
      return AXB200_OUT_OF_MEMORY;
    if ((reinterpret_cast<uintptr_t>(workspace) & 15u) == 0) return axb::latent_umma(p, workspace, st);
  }
  const size_t smem = (size_t)(2 * kv_rank + rot_dim) * sizeof(float);
  if (smem > 200 * 1024) return AXB200_INVALID_ARGUMENT;
  auto *kernel = dtype == AXB200_FLOAT32 ? axb::latent_attend_generic_kernel<float>
                                         : axb::latent_attend_generic_kernel<__nv_bfloat16>;
  if (smem > 40 * 1024 && cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
    return AXB200_DEVICE_ERROR;
  return axb::launch_dependent(kernel, dim3(rows, heads), dim3(axb::kGenThreads), smem, st, p);
}

int axb200_latent_gather(const void *pages, const int32_t *block_row, void *out, int64_t first, int64_t n, int row_elems, int page_tokens,
                         int max_blocks, int num_pages, int dtype, void *stream) {
  const size_t es = axb::dtype_size(dtype);
  if (es == 0) return AXB200_UNSUPPORTED_TYPE;
  if (!pages || !block_row || !out) return AXB200_INVALID_PTR;
  if (n < 0 || first < 0 || first + n > (int64_t)max_blocks * page_tokens || row_elems <= 0 || page_tokens <= 0 || max_blocks <= 0 || num_pages <= 0)
    return AXB200_INVALID_ARGUMENT;
  if (n == 0) return AXB200_OK;
  const int row_bytes = (int)(row_elems * es);
  const bool vec = row_bytes % 16 == 0 && ((reinterpret_cast<uintptr_t>(pages) | reinterpret_cast<uintptr_t>(out)) & 15u) == 0;
  const int unit = vec ? 16 : 2;
  const int64_t items = n * (row_bytes / unit);
  const int grid = (int)(items / 256 + 1 < 148 * 8 ? items / 256 + 1 : 148 * 8);
  return axb::launch_dependent(axb::latent_gather_kernel, dim3(grid), dim3(256), 0, static_cast<cudaStream_t>(stream),
                               static_cast<const uint8_t *>(pages), block_row, static_cast<uint8_t *>(out), (int)first, (int)n, row_bytes,
                               page_tokens, max_blocks, num_pages, unit);
}

}  // extern "C"
