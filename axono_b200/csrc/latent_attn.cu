// Attention over a cache of latents: every token caches one row [c (kv_rank) | rotated key part (rot_dim)] that
// all heads share, and a head's key and value are linear maps of c.  Folding the key map into the query
// (q_lat = q . W_uk) and the value map behind the sum turns it into attention of H queries per token over ONE
// key row of kv_rank + rot_dim elements whose first kv_rank elements are also the value:
//     score = (q_lat . c + q_rot . k_rot) * scale,   out_lat = sum softmax(score) c.
// This file holds the kernels of that form: the step's norms, rotation and append in one launch; the
// tensor-core split kernel (bf16) with its merge; an evaluation for every other size and for fp32; and the
// gather that the expanded form (latent_prefill.cu) reads from.
//
// Rows are independent: row r belongs to sequence row_seq[r] (its block-table row) and sees the cached tokens
// 0 .. row_pos[r], so one launch serves decode batches, portions of prompts and mixtures of both.
#include <math.h>

#include <mutex>

#include "tcgen05.cuh"

namespace axb {
namespace {

constexpr float kLog2e = 1.4426950408889634f;

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

// ---- attention in latent form -------------------------------------------------------------------------
struct AttendParams {
  const void *q_lat;  // (rows, heads, kv_rank)
  const void *q;      // (rows, q_ld): the rotated part of head h starts at h * (dim + rot_dim) + dim
  int64_t q_ld;
  void *out;  // (rows, heads, kv_rank)
  const void *pages;
  const int32_t *block_table, *row_seq, *row_pos;
  int rows, heads, dim, kv_rank, rot_dim, page_tokens, max_blocks, num_pages, max_seqs, max_len;
  float scale;
  unsigned long long wait_ns;
};

// Keys row r may read: 0 .. row_pos[r], never beyond the block table's reach or the host's bound.
__device__ __forceinline__ int visible_keys(const AttendParams &p, int r) {
  const int seq = p.row_seq[r];
  if (seq < 0 || seq >= p.max_seqs) return 0;
  const int cover = min(p.max_blocks * p.page_tokens, p.max_len);
  return max(0, min(p.row_pos[r] + 1, cover));
}

// Any size, fp32 or bf16: one CTA per (row, head); 64 keys at a time, one warp per key for the scores, one
// thread per latent element for the sum.  fp32 arithmetic throughout.
constexpr int kGenThreads = 256, kGenTile = 64;

template <typename T>
__global__ void __launch_bounds__(kGenThreads) latent_attend_generic_kernel(const AttendParams p) {
  extern __shared__ float sm[];
  __shared__ float scratch[32], score[kGenTile];
  __shared__ const T *key[kGenTile];
  const int row_elems = p.kv_rank + p.rot_dim;
  float *q = sm, *acc = sm + row_elems;
  const int r = blockIdx.x, h = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  grid_dependency_wait();
  grid_dependency_launch();
  const T *ql = static_cast<const T *>(p.q_lat) + ((size_t)r * p.heads + h) * p.kv_rank;
  const T *qr = static_cast<const T *>(p.q) + (size_t)r * p.q_ld + (size_t)h * (p.dim + p.rot_dim) + p.dim;
  for (int i = threadIdx.x; i < row_elems; i += kGenThreads) q[i] = i < p.kv_rank ? ldf(ql + i) : ldf(qr + i - p.kv_rank);
  for (int i = threadIdx.x; i < p.kv_rank; i += kGenThreads) acc[i] = 0.f;
  const int keys = visible_keys(p, r);
  const int32_t *table = p.block_table + (size_t)max(0, min(p.row_seq[r], p.max_seqs - 1)) * p.max_blocks;
  const T *pages = static_cast<const T *>(p.pages);
  float m = -INFINITY, l = 0.f;
  for (int k0 = 0; k0 < keys; k0 += kGenTile) {
    const int n = min(kGenTile, keys - k0);
    __syncthreads();
    if (threadIdx.x < n) {
      const int t = k0 + threadIdx.x;
      int page = table[t / p.page_tokens];
      if (page < 0 || page >= p.num_pages) {
        atomicOr(&g_error_word, AXB200_ERR_BAD_PAGE);
        page = 0;
      }
      key[threadIdx.x] = pages + ((size_t)page * p.page_tokens + t % p.page_tokens) * row_elems;
    }
    __syncthreads();
    for (int j = warp; j < n; j += kGenThreads / 32) {
      float s = 0.f;
      for (int i = lane; i < row_elems; i += 32) s = fmaf(q[i], ldf(key[j] + i), s);
      s = warp_sum(s);
      if (lane == 0) score[j] = s * p.scale;
    }
    __syncthreads();
    float mt = m;
    for (int j = 0; j < n; ++j) mt = fmaxf(mt, score[j]);
    const float corr = expf(m - mt);  // 0 at the first tile
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

// ---- bf16 on tensor cores (mma.sync): one key row serves 16 heads ------------------------------------------
// With few heads the form is bound by reading the cache: 1152 bytes of row against 16 x 1088 products at
// kv_rank 512, rot_dim 64.  The work of a launch - items (row, tile of 16 heads), each of ceil(keys / 64) key
// tiles - is laid end to end and cut into one equal range of key tiles per SM, from the positions in device
// memory, so that a captured graph stays balanced as the cache grows.  A CTA walks its range with one
// continuous ring of TMA stages; an item that lies in one range is finished there, the others leave one
// un-normalised record per range for the merge kernel.
//
// Eight warps (a ninth would cut the registers a thread can have from 255 to 168, and the queries alone are 144).
// Scores: warp w takes keys 8w .. 8w + 7 of the tile, its A operand (the 16 queries) in registers for the
// whole item.  Then the row maxima meet in shared memory, the weights go to shared
// memory as bf16, and for the sum warp w takes the latent elements 8 * kTiles * w ... .  Every stage is read
// twice from shared memory and once from the cache.  Warp 0 refills the stage of the tile before last whenever the
// barrier between the two halves shows that every warp is done with it.
constexpr int kMmaWarps = 8, kMmaThreads = kMmaWarps * 32, kMmaKeys = 64, kMmaHeads = 16, kMaxMmaRows = 1024;
constexpr int kMinTilesPerCta = 2, kPStride = 72;  // P rows of 64 bf16, padded against bank conflicts

// kBoxes: 64-element blocks of a cached row; kTiles: 8-element output tiles per warp (kv_rank <= 64 * kTiles)
template <int kBoxes>
struct MmaShape {
  static constexpr int kStageBytes = kBoxes * kMmaKeys * 128;
  static constexpr int kStages = kBoxes >= 8 ? 3 : 4;
  static constexpr int kOffP = kStages * kStageBytes, kOffMax = kOffP + kMmaHeads * kPStride * 2;
  static constexpr int kOffSum = kOffMax + kMmaWarps * kMmaHeads * 4, kOffBar = kOffSum + kMmaWarps * kMmaHeads * 4;
  static constexpr int kOffStart = kOffBar + 128;  // first key tile of every row, per head tile
  static constexpr int kSmem = kOffStart + (kMaxMmaRows + 1) * 4;
};

struct MmaParams {
  AttendParams a;
  int head_tiles;
  float *part_o;   // (2 * CTAs, 16, kv_rank)
  float2 *part_ml; // (2 * CTAs, 16): maximum (log2 domain), sum
};

__device__ __forceinline__ int tiles_of(const AttendParams &p, int r) { return (visible_keys(p, r) + kMmaKeys - 1) / kMmaKeys; }

// Key tiles one CTA takes when `total` are to be done by `ctas`.
__device__ __forceinline__ int tiles_per_cta(int total, int ctas) { return max(kMinTilesPerCta, (total + ctas - 1) / ctas); }

// start[r] = key tiles of the rows before r (for one head tile), r = 0 .. rows; all threads of the CTA.
__device__ __forceinline__ void scan_tiles(const AttendParams &p, int *start) {
  __shared__ int warp_total[32];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
  int base = 0;
  if (threadIdx.x == 0) start[0] = 0;
  for (int r0 = 0; r0 < p.rows; r0 += blockDim.x) {
    const int r = r0 + threadIdx.x;
    int v = r < p.rows ? tiles_of(p, r) : 0;
#pragma unroll
    for (int d = 1; d < 32; d <<= 1) {
      const int o = __shfl_up_sync(0xffffffffu, v, d);
      if (lane >= d) v += o;
    }
    if (lane == 31) warp_total[warp] = v;
    __syncthreads();
    int before = base, all = base;
    for (int w = 0; w < warps; ++w) {
      if (w < warp) before += warp_total[w];
      all += warp_total[w];
    }
    if (r < p.rows) start[r + 1] = before + v;
    base = all;
    __syncthreads();
  }
}

// Items are ordered row by row, head tiles within a row: item i = r * head_tiles + t covers key tiles
// [head_tiles * start[r] + t * n_r, ... + n_r), n_r = start[r + 1] - start[r].
template <int kBoxes, int kTiles>
__global__ void __launch_bounds__(kMmaThreads, 1)
latent_attend_mma_kernel(const __grid_constant__ CUtensorMap tmPages, const __grid_constant__ MmaParams mp) {
  using S = MmaShape<kBoxes>;
  extern __shared__ __align__(1024) uint8_t smem[];
  const AttendParams &p = mp.a;
  uint64_t *full = reinterpret_cast<uint64_t *>(smem + S::kOffBar);
  volatile int *abort_flag = reinterpret_cast<volatile int *>(full + S::kStages);
  __nv_bfloat16 *ps = reinterpret_cast<__nv_bfloat16 *>(smem + S::kOffP);
  float(*smax)[kMmaHeads] = reinterpret_cast<float(*)[kMmaHeads]>(smem + S::kOffMax);
  float(*ssum)[kMmaHeads] = reinterpret_cast<float(*)[kMmaHeads]>(smem + S::kOffSum);
  int *start = reinterpret_cast<int *>(smem + S::kOffStart);
  if ((smem_u32(smem) & 1023u) != 0) {
    if (threadIdx.x == 0) atomicOr(&g_error_word, AXB200_ERR_WAIT_TIMEOUT);
    return;
  }
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    for (int i = 0; i < S::kStages; ++i) mbar_init(&full[i], 1);
    *abort_flag = 0;
    mbar_fence_init();
  }
  grid_dependency_wait();
  grid_dependency_launch();
  scan_tiles(p, start);
  __syncthreads();
  const int ht = mp.head_tiles, total = ht * start[p.rows], per = tiles_per_cta(total, gridDim.x);
  const int lo = blockIdx.x * per, hi = min(total, lo + per);
  if (lo >= hi) return;
  // the row that holds key tile lo: the last r with ht * start[r] <= lo and at least one tile
  int r_first = 0;
  {
    int a = 0, b = p.rows - 1;
    while (a < b) {
      const int m = (a + b + 1) >> 1;
      if (ht * start[m] <= lo)
        a = m;
      else
        b = m - 1;
    }
    r_first = a;
  }

  // ---- warp 0 as the loader: the next key tile of the range into the next stage ----
  int load_row = r_first, load_at = lo, loaded = 0;
  auto load_next = [&] {
    if (warp != 0 || load_at >= hi) return;
    while (load_at >= ht * start[load_row + 1]) ++load_row;
    const int n = start[load_row + 1] - start[load_row], t0 = (load_at - ht * start[load_row]) % n * kMmaKeys;
    int page = p.block_table[(size_t)p.row_seq[load_row] * p.max_blocks + t0 / p.page_tokens];
    if (page < 0 || page >= p.num_pages) {
      if (lane == 0) atomicOr(&g_error_word, AXB200_ERR_BAD_PAGE);
      page = 0;
    }
    const int s = loaded % S::kStages;
    if (lane == 0) mbar_arrive_expect_tx(&full[s], S::kStageBytes);
    __syncwarp();
    if (lane < kBoxes)
      tma_load_2d(smem + s * S::kStageBytes + lane * (kMmaKeys * 128), &tmPages, &full[s], lane * 64,
                  page * p.page_tokens + t0 % p.page_tokens);
    ++load_at;
    ++loaded;
  };
  if (warp == 0 && lane == 0) tma_prefetch_descriptor(&tmPages);
#pragma unroll 1
  for (int i = 0; i < S::kStages; ++i) load_next();

  const int gr = lane >> 2, gc = (lane & 3) * 2;  // fragment row (and + 8) and first of two columns
  const float scale_log2 = p.scale * kLog2e;
  const uint32_t smem_base = smem_u32(smem), ps_base = smem_u32(ps);
  int step = 0;
  bool gave_up = false;  // the same in every warp
  for (int r = r_first, g = lo; g < hi && !gave_up; ++r) {
    const int n = start[r + 1] - start[r], base = ht * start[r], keys = visible_keys(p, r);
    while (g < hi && g < base + ht * n && !gave_up) {
      // ---- one segment: key tiles [k_first, k_last) of item (r, tile t) ----
      const int t = (g - base) / n, k_first = (g - base) % n, k_last = min(n, k_first + hi - g);
      const int h0 = t * kMmaHeads;
      uint32_t qa[kBoxes * 4][4];
      {
        const __nv_bfloat16 *ql = static_cast<const __nv_bfloat16 *>(p.q_lat) + (size_t)r * p.heads * p.kv_rank;
        const __nv_bfloat16 *qr = static_cast<const __nv_bfloat16 *>(p.q) + (size_t)r * p.q_ld + p.dim;
        const int elems = p.kv_rank + p.rot_dim;
        auto pair = [&](int h, int e) -> uint32_t {
          if (h >= p.heads || e >= elems) return 0u;
          return e < p.kv_rank ? *reinterpret_cast<const uint32_t *>(ql + (size_t)h * p.kv_rank + e)
                               : *reinterpret_cast<const uint32_t *>(qr + (size_t)h * (p.dim + p.rot_dim) + (e - p.kv_rank));
        };
#pragma unroll
        for (int k = 0; k < kBoxes * 4; ++k) {
          qa[k][0] = pair(h0 + gr, k * 16 + gc);
          qa[k][1] = pair(h0 + gr + 8, k * 16 + gc);
          qa[k][2] = pair(h0 + gr, k * 16 + 8 + gc);
          qa[k][3] = pair(h0 + gr + 8, k * 16 + 8 + gc);
        }
      }
      float o[kTiles][4] = {};
      float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};  // rows gr, gr + 8; l over this warp's keys
      for (int k = k_first; k < k_last; ++k, ++step) {
        const int s = step % S::kStages;
        const uint32_t stage = smem_base + s * S::kStageBytes;
        const bool ok = __all_sync(0xffffffffu, mbar_wait_bounded(&full[s], (step / S::kStages) & 1, abort_flag, p.wait_ns));
        const int valid = min(kMmaKeys, keys - k * kMmaKeys);
        if (valid < kMmaKeys) {
          // the last tile: rows past the end are not the sequence's and may hold anything; weight 0 is not enough
          // against a NaN, so they are cleared
          if (ok)
            for (int i = threadIdx.x; i < (kMmaKeys - valid) * kBoxes * 8; i += kMmaWarps * 32) {
              const int c = i & 7, b = (i >> 3) % kBoxes, row = valid + (i >> 3) / kBoxes;
              *reinterpret_cast<uint4 *>(smem + s * S::kStageBytes + b * (kMmaKeys * 128) + row * 128 + c * 16) = make_uint4(0, 0, 0, 0);
            }
          asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
          __syncthreads();
        }
        // ---- scores of keys 8 * warp .. + 7 ----
        float c0[4] = {}, c1[4] = {};
        if (ok) {
          const uint32_t row = stage + (warp * 8 + (lane & 7)) * 128;
#pragma unroll
          for (int b = 0; b < kBoxes; ++b) {
#pragma unroll
            for (int hf = 0; hf < 2; ++hf) {  // 32 elements: four 16-byte chunks of 8 keys
              uint32_t b0, b1, b2, b3;
              ldmatrix_x4(b0, b1, b2, b3, row + b * (kMmaKeys * 128) + (((hf * 4 + (lane >> 3)) ^ (lane & 7)) << 4));
              mma_16816_bf16(c0, qa[b * 4 + hf * 2], b0, b1);
              mma_16816_bf16(c1, qa[b * 4 + hf * 2 + 1], b2, b3);
            }
          }
        }
        float sc[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          sc[i] = (c0[i] + c1[i]) * scale_log2;
          if (warp * 8 + gc + (i & 1) >= valid) sc[i] = -INFINITY;
        }
        float mx[2] = {fmaxf(sc[0], sc[1]), fmaxf(sc[2], sc[3])};
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 1));
          mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 2));
        }
        if ((lane & 3) == 0) {
          smax[warp][gr] = mx[0];
          smax[warp][gr + 8] = mx[1];
        }
        __syncthreads();  // also: every warp is done with the tile before, its stage and its P
        // between the two barriers of a tile no warp can be in another tile's wait: all read the same
        gave_up = *abort_flag;
        if (step > 0 && !gave_up) load_next();
        float corr[2];
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          float mn = m[i];
#pragma unroll
          for (int w = 0; w < kMmaWarps; ++w) mn = fmaxf(mn, smax[w][gr + 8 * i]);
          const float safe = mn == -INFINITY ? 0.f : mn;
          corr[i] = fast_exp2(m[i] - safe);
          m[i] = mn;
          const float pa = fast_exp2(sc[2 * i] - safe), pb = fast_exp2(sc[2 * i + 1] - safe);
          l[i] = l[i] * corr[i] + pa + pb;
          *reinterpret_cast<uint32_t *>(ps + (gr + 8 * i) * kPStride + warp * 8 + gc) = pack_bf16x2(pa, pb);
        }
        __syncthreads();
        if (gave_up) break;
        // ---- sum: elements 8 * kTiles * warp ... of every key ----
#pragma unroll
        for (int j = 0; j < kTiles; ++j) {
          o[j][0] *= corr[0], o[j][1] *= corr[0];
          o[j][2] *= corr[1], o[j][3] *= corr[1];
        }
        {
#pragma unroll
          for (int kk = 0; kk < kMmaKeys / 16; ++kk) {
            uint32_t a[4];
            ldmatrix_x4(a[0], a[1], a[2], a[3], ps_base + ((lane & 15) * kPStride + kk * 16 + (lane >> 4) * 8) * 2);
            const int key = kk * 16 + (lane & 15);
#pragma unroll
            for (int j = 0; j < kTiles; j += 2) {
              const int chunk = warp * kTiles + j + (lane >> 4);  // 8 elements
              uint32_t b0, b1, b2, b3;
              ldmatrix_x4_trans(b0, b1, b2, b3, stage + (chunk >> 3) * (kMmaKeys * 128) + key * 128 + (((chunk & 7) ^ (key & 7)) << 4));
              mma_16816_bf16(o[j], a, b0, b1);
              mma_16816_bf16(o[j + 1], a, b2, b3);
            }
          }
        }
      }
      if (gave_up) break;
      g += k_last - k_first;
      // ---- the segment's end ----
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        l[i] += __shfl_xor_sync(0xffffffffu, l[i], 1);
        l[i] += __shfl_xor_sync(0xffffffffu, l[i], 2);
      }
      if ((lane & 3) == 0) {
        ssum[warp][gr] = l[0];
        ssum[warp][gr + 8] = l[1];
      }
      __syncthreads();
      float lt[2] = {0.f, 0.f};
#pragma unroll
      for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int w = 0; w < kMmaWarps; ++w) lt[i] += ssum[w][gr + 8 * i];
      __syncthreads();  // ssum may be written again
      const bool whole = k_first == 0 && k_last == n;
      const int slot = blockIdx.x * 2 + (k_first == 0 ? 1 : 0);
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int hr = gr + 8 * i, h = h0 + hr;
        if (whole) {
          if (h < p.heads) {
            const float inv = lt[i] > 0.f ? 1.0f / lt[i] : 0.f;
            __nv_bfloat16 *dst = static_cast<__nv_bfloat16 *>(p.out) + ((size_t)r * p.heads + h) * p.kv_rank;
#pragma unroll
            for (int j = 0; j < kTiles; ++j) {
              const int e = (warp * kTiles + j) * 8 + gc;
              if (e < p.kv_rank) *reinterpret_cast<uint32_t *>(dst + e) = pack_bf16x2(o[j][2 * i] * inv, o[j][2 * i + 1] * inv);
            }
          }
        } else {
          float *dst = mp.part_o + ((size_t)slot * kMmaHeads + hr) * p.kv_rank;
#pragma unroll
          for (int j = 0; j < kTiles; ++j) {
            const int e = (warp * kTiles + j) * 8 + gc;
            if (e < p.kv_rank) *reinterpret_cast<float2 *>(dst + e) = make_float2(o[j][2 * i], o[j][2 * i + 1]);
          }
          if (warp == 0 && (lane & 3) == 0) mp.part_ml[slot * kMmaHeads + hr] = make_float2(m[i], lt[i]);
        }
      }
    }
  }
  if (gave_up && warp == 0) {  // no copy may still be on its way when the CTA leaves
    const unsigned long long t0 = global_timer_ns();
    for (int j = max(0, loaded - S::kStages); j < loaded; ++j)
      while (!mbar_try_wait(&full[j % S::kStages], (j / S::kStages) & 1) && global_timer_ns() - t0 < 100000000ull) {
      }
  }
}

// Merges the records of the items that were cut: one CTA per (row, head).
constexpr int kMergeThreads = 128;
__global__ void __launch_bounds__(kMergeThreads) latent_merge_kernel(const MmaParams mp, int ctas) {
  __shared__ int scratch[2][kMergeThreads / 32];
  const AttendParams &p = mp.a;
  const int r = blockIdx.x, h = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  grid_dependency_wait();
  grid_dependency_launch();
  int before = 0, all = 0;
  for (int i = threadIdx.x; i < p.rows; i += kMergeThreads) {
    const int t = tiles_of(p, i);
    all += t;
    before += i < r ? t : 0;
  }
#pragma unroll
  for (int off = 16; off > 0; off >>= 1) {
    before += __shfl_xor_sync(0xffffffffu, before, off);
    all += __shfl_xor_sync(0xffffffffu, all, off);
  }
  if (lane == 0) scratch[0][warp] = before, scratch[1][warp] = all;
  __syncthreads();
  before = all = 0;
#pragma unroll
  for (int w = 0; w < kMergeThreads / 32; ++w) before += scratch[0][w], all += scratch[1][w];
  const int n = tiles_of(p, r), per = tiles_per_cta(all * mp.head_tiles, ctas);
  __nv_bfloat16 *out = static_cast<__nv_bfloat16 *>(p.out) + ((size_t)r * p.heads + h) * p.kv_rank;
  if (n == 0) {  // a row that sees nothing
    for (int e = threadIdx.x; e < p.kv_rank; e += kMergeThreads) stf(out + e, 0.f);
    return;
  }
  const int lo = before * mp.head_tiles + h / kMmaHeads * n, first = lo / per, last = (lo + n - 1) / per;
  if (first == last) return;
  // records: the range that holds the item's first tile filed it under 1, the later ones under 0
  auto slot = [&](int c) { return (c * 2 + (c == first ? 1 : 0)) * kMmaHeads + h % kMmaHeads; };
  float top = -INFINITY, sum = 0.f;
  for (int c = first; c <= last; ++c) top = fmaxf(top, mp.part_ml[slot(c)].x);
  for (int c = first; c <= last; ++c) {
    const float2 ml = mp.part_ml[slot(c)];
    sum = fmaf(fast_exp2(ml.x - top), ml.y, sum);
  }
  const float inv = sum > 0.f ? 1.0f / sum : 0.f;
  for (int e = threadIdx.x * 2; e < p.kv_rank; e += kMergeThreads * 2) {
    float2 acc = make_float2(0.f, 0.f);
#pragma unroll 4
    for (int c = first; c <= last; ++c) {
      const int sl = slot(c);
      const float w = fast_exp2(mp.part_ml[sl].x - top);
      const float2 v = *reinterpret_cast<const float2 *>(mp.part_o + (size_t)sl * p.kv_rank + e);
      acc.x = fmaf(w, v.x, acc.x);
      acc.y = fmaf(w, v.y, acc.y);
    }
    *reinterpret_cast<uint32_t *>(out + e) = pack_bf16x2(acc.x * inv, acc.y * inv);
  }
}

int sm_count() {
  static int counts[64] = {0};
  int dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return 0;
  if (!counts[dev]) cudaDeviceGetAttribute(&counts[dev], cudaDevAttrMultiProcessorCount, dev);
  return counts[dev];
}
constexpr int kMaxSms = 256;  // bound of the workspace

bool mma_sizes(int heads, int kv_rank, int rot_dim, int dtype) {
  return dtype == AXB200_BFLOAT16 && kv_rank % 8 == 0 && rot_dim % 8 == 0 && kv_rank + rot_dim <= 576 && kv_rank <= 512 &&
         heads <= 65535;
}

template <int kBoxes, int kTiles>
int launch_mma(const CUtensorMap &map, const MmaParams &mp, int ctas, cudaStream_t st) {
  auto *kernel = latent_attend_mma_kernel<kBoxes, kTiles>;
  static std::mutex mu;
  static bool opted[64] = {false};
  int dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return AXB200_DEVICE_ERROR;
  {
    std::lock_guard<std::mutex> lock(mu);
    if (!opted[dev]) {
      if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, MmaShape<kBoxes>::kSmem) != cudaSuccess)
        return AXB200_DEVICE_ERROR;
      opted[dev] = true;
    }
  }
  const int rc = launch_dependent(kernel, dim3(ctas), dim3(kMmaThreads), MmaShape<kBoxes>::kSmem, st, map, mp);
  if (rc != AXB200_OK) return rc;
  return launch_dependent(latent_merge_kernel, dim3(mp.a.rows, mp.a.heads), dim3(kMergeThreads), 0, st, mp, ctas);
}

int attend_mma(const AttendParams &p, void *workspace, cudaStream_t st) {
  const int elems = p.kv_rank + p.rot_dim;
  CUtensorMap map;
  EncodeTiledFn fn = tensor_map_encoder();
  const cuuint64_t dims[2] = {(cuuint64_t)elems, (cuuint64_t)p.num_pages * p.page_tokens}, strides[1] = {(cuuint64_t)elems * 2};
  const cuuint32_t box[2] = {64, kMmaKeys}, es[2] = {1, 1};
  if (fn(&map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void *>(p.pages), dims, strides, box, es,
         CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
         CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) != CUDA_SUCCESS)
    return AXB200_INTERNAL_ERROR;
  const int ctas = sm_count();
  if (ctas <= 0 || ctas > kMaxSms) return AXB200_INTERNAL_ERROR;
  for (int r0 = 0; r0 < p.rows; r0 += kMaxMmaRows) {
    MmaParams mp{p, (p.heads + kMmaHeads - 1) / kMmaHeads, nullptr, nullptr};
    AttendParams &a = mp.a;
    a.rows = p.rows - r0 < kMaxMmaRows ? p.rows - r0 : kMaxMmaRows;
    a.q_lat = static_cast<const __nv_bfloat16 *>(p.q_lat) + (size_t)r0 * p.heads * p.kv_rank;
    a.q = static_cast<const __nv_bfloat16 *>(p.q) + (size_t)r0 * p.q_ld;
    a.out = static_cast<__nv_bfloat16 *>(p.out) + (size_t)r0 * p.heads * p.kv_rank;
    a.row_seq = p.row_seq + r0;
    a.row_pos = p.row_pos + r0;
    mp.part_ml = static_cast<float2 *>(workspace);
    mp.part_o = reinterpret_cast<float *>(mp.part_ml + 2 * kMaxSms * kMmaHeads);
    int rc;
    if (elems <= 128)
      rc = launch_mma<2, 2>(map, mp, ctas, st);
    else if (elems <= 256)
      rc = launch_mma<4, 4>(map, mp, ctas, st);
    else if (elems <= 320 && p.kv_rank <= 256)
      rc = launch_mma<5, 4>(map, mp, ctas, st);
    else
      rc = launch_mma<9, 8>(map, mp, ctas, st);
    if (rc != AXB200_OK) return rc;
  }
  return AXB200_OK;
}

// ---- gather: cached rows 0 .. n-1 of one sequence, contiguous -----------------------------------------
__global__ void __launch_bounds__(256)
latent_gather_kernel(const uint8_t *pages, const int32_t *table, uint8_t *out, int n, int row_bytes, int page_tokens,
                     int max_blocks, int num_pages, int unit) {
  grid_dependency_wait();
  grid_dependency_launch();
  const int per = row_bytes / unit;
  const int64_t total = (int64_t)n * per;
  for (int64_t i = blockIdx.x * 256ll + threadIdx.x; i < total; i += gridDim.x * 256ll) {
    const int t = (int)(i / per), c = (int)(i % per), blk = t / page_tokens;
    const int page = blk < max_blocks ? table[blk] : -1;
    if (page < 0 || page >= num_pages) {
      atomicOr(&g_error_word, AXB200_ERR_BAD_PAGE);
      continue;
    }
    const uint8_t *src = pages + ((size_t)page * page_tokens + t % page_tokens) * row_bytes + (size_t)c * unit;
    uint8_t *dst = out + (size_t)t * row_bytes + (size_t)c * unit;
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
    return axb::launch_dependent(axb::latent_prepare_kernel<T>, dim3((unsigned)rows), dim3(axb::kPrepThreads), 0,
                                 static_cast<cudaStream_t>(stream), p);
  };
  return dtype == AXB200_FLOAT32 ? go(float{}) : go(__nv_bfloat16{});
}

size_t axb200_latent_attend_workspace_bytes(int rows, int heads, int kv_rank, int rot_dim, int64_t max_len, int dtype) {
  if (rows <= 0 || heads <= 0 || kv_rank <= 0 || !axb::mma_sizes(heads, kv_rank, rot_dim, dtype)) return 0;
  return (size_t)2 * axb::kMaxSms * axb::kMmaHeads * (sizeof(float2) + (size_t)kv_rank * sizeof(float));
}

int axb200_latent_attend(const void *q_lat, const void *q, int64_t q_ld, int dim, void *out, const void *pages,
                         const int32_t *block_table, const int32_t *row_seq, const int32_t *row_pos, int rows, int heads,
                         int kv_rank, int rot_dim, float scale, int page_tokens, int max_blocks, int num_pages,
                         int max_seqs, int64_t max_len, int dtype, void *workspace, size_t workspace_bytes, void *stream) {
  if (dtype != AXB200_FLOAT32 && dtype != AXB200_BFLOAT16) return AXB200_UNSUPPORTED_TYPE;
  if (!q_lat || !q || !out || !pages || !block_table || !row_seq || !row_pos) return AXB200_INVALID_PTR;
  if (rows < 0 || heads <= 0 || heads > 65535 || kv_rank <= 0 || rot_dim < 0 || dim < 0 || page_tokens <= 0 || max_blocks <= 0 ||
      num_pages <= 0 || max_seqs <= 0 || max_len <= 0 || max_len > 0x7fffffff - 4096)
    return AXB200_INVALID_ARGUMENT;
  if (q_ld < (int64_t)heads * (dim + rot_dim)) return AXB200_SHAPE_MISMATCH;
  if (rows == 0) return AXB200_OK;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  axb::AttendParams p{};
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
  // aligned operands, whole key tiles per page, and key tiles that an int can count
  const uintptr_t bits = reinterpret_cast<uintptr_t>(q_lat) | reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(out) |
                         reinterpret_cast<uintptr_t>(workspace);
  if (axb::mma_sizes(heads, kv_rank, rot_dim, dtype) && page_tokens % axb::kMmaKeys == 0 && q_ld % 2 == 0 && dim % 2 == 0 &&
      (bits & 7u) == 0 && (reinterpret_cast<uintptr_t>(pages) & 15u) == 0 && axb::tensor_map_encoder() &&
      (int64_t)num_pages * page_tokens < 0x7fffffff &&
      (max_len / axb::kMmaKeys + 1) * (int64_t)axb::kMaxMmaRows * ((heads + 15) / 16) < 0x7fffffff) {
    if (!workspace || workspace_bytes < axb200_latent_attend_workspace_bytes(rows, heads, kv_rank, rot_dim, max_len, dtype))
      return AXB200_OUT_OF_MEMORY;
    return axb::attend_mma(p, workspace, st);
  }
  const size_t smem = (size_t)(2 * kv_rank + rot_dim) * sizeof(float);
  if (smem > 200 * 1024) return AXB200_INVALID_ARGUMENT;
  auto *kernel = dtype == AXB200_FLOAT32 ? axb::latent_attend_generic_kernel<float>
                                         : axb::latent_attend_generic_kernel<__nv_bfloat16>;
  if (smem > 40 * 1024 && cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
    return AXB200_DEVICE_ERROR;
  return axb::launch_dependent(kernel, dim3(rows, heads), dim3(axb::kGenThreads), smem, st, p);
}

int axb200_latent_gather(const void *pages, const int32_t *block_row, void *out, int64_t n, int row_elems, int page_tokens,
                         int max_blocks, int num_pages, int dtype, void *stream) {
  const size_t es = axb::dtype_size(dtype);
  if (es == 0) return AXB200_UNSUPPORTED_TYPE;
  if (!pages || !block_row || !out) return AXB200_INVALID_PTR;
  if (n < 0 || n > (int64_t)max_blocks * page_tokens || row_elems <= 0 || page_tokens <= 0 || max_blocks <= 0 || num_pages <= 0)
    return AXB200_INVALID_ARGUMENT;
  if (n == 0) return AXB200_OK;
  const int row_bytes = (int)(row_elems * es);
  const bool vec = row_bytes % 16 == 0 && ((reinterpret_cast<uintptr_t>(pages) | reinterpret_cast<uintptr_t>(out)) & 15u) == 0;
  const int unit = vec ? 16 : 2;
  const int64_t items = n * (row_bytes / unit);
  const int grid = (int)(items / 256 + 1 < 148 * 8 ? items / 256 + 1 : 148 * 8);
  return axb::launch_dependent(axb::latent_gather_kernel, dim3(grid), dim3(256), 0, static_cast<cudaStream_t>(stream),
                               static_cast<const uint8_t *>(pages), block_row, static_cast<uint8_t *>(out), (int)n, row_bytes,
                               page_tokens, max_blocks, num_pages, unit);
}

}  // extern "C"
