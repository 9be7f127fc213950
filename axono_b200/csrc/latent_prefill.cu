// The expanded form of latent attention for portions of prompts: keys W_uk c and values W_uv c are formed for all
// heads by library products, and this kernel attends them with 5th-generation tensor cores.  A head's key is
// [its own dim elements | the rotated part that all heads share], so the two come through tensor maps of
// their own - the shared part is read from the cached rows and never copied per head - and meet in shared
// memory as neighbouring 64-wide blocks of the K dimension; likewise the two parts of a query.  Blocks that are
// not full (dim 32, rot 16, ...) are zero-filled by TMA, so any sizes that are multiples of 8 up to
// dim 128, rot 64, vdim 128 run.  Without a rotated part the key is its own elements alone; kv_heads below heads shares
// a key and value head among a group of query heads, which makes this the prompt form of grouped attention too.
//
// A row may see only the last `window` keys (a CTA starts at the tile that holds its first row's first key), and a
// per-head sink may join the denominator.
//
// Structure as the 256-row form of prefill_attn.cu: one CTA per (256 query rows, head) works on two query tiles
// against key tiles of 128; S_g and O_g in tensor memory; warps 0-7 own one query row per thread and do the
// online softmax; warp 8 issues the MMAs, warp 9 the TMA loads.  What differs: K is 128 x up to 192 elements
// per tile, so K is double-buffered while V has one buffer whose two halves of 64 keys are freed and refilled
// separately; rows stand at positions start .. start + n - 1 of a longer key sequence.  Every wait is bounded.
#include <math.h>

#include <mutex>
#include <type_traits>

#include "tcgen05.cuh"

namespace axb {
namespace {

constexpr int kRows = 128, kKeys = 128, kBox = kRows * 64 * 2;  // one [128 rows][64 elements] block: 16 KB
constexpr int kThreads = 320, kMmaWarp = 8, kLoadWarp = 9;
constexpr float kLog2e = 1.4426950408889634f, kLazy = 8.0f;

struct Params {
  __nv_bfloat16 *out;
  int n, start, skv, heads, group, vdim;  // group: query heads per key and value head
  int window;                             // 0: all
  const float *sink;                      // (heads), or null
  float scale_log2;
  unsigned long long wait_ns;
};

// kQB / kVB: 64-wide blocks of the heads' own key part and of the values; kRot: one more block for the rotated part
template <int kQB, int kVB, int kRot>
struct Layout {
  static constexpr int kBlocks = kQB + kRot;
  static constexpr int kTile = kBlocks * kBox;        // a query tile or a key tile
  static constexpr int kVHalf = 64 * kVB * 64 * 2;    // 64 keys: kVB boxes of [64 keys][64]
  static constexpr int kOffK = 2 * kTile, kOffV = kOffK + 2 * kTile, kOffBar = kOffV + 2 * kVHalf;
  static constexpr int kSmem = kOffBar + 256;
};

template <int kQB, int kVB, int kRot>
__global__ void __launch_bounds__(kThreads, 1)
latent_prefill_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmQr,
                      const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmKr,
                      const __grid_constant__ CUtensorMap tmV, const Params p) {
  using L = Layout<kQB, kVB, kRot>;
  extern __shared__ __align__(1024) uint8_t smem[];
  uint64_t *bars = reinterpret_cast<uint64_t *>(smem + L::kOffBar);
  uint64_t *bar_q = bars, *full_k = bars + 1, *empty_k = bars + 3, *full_v = bars + 5, *empty_v = bars + 7;
  uint64_t *bar_s = bars + 9, *bar_fin = bars + 11, *bar_p = bars + 13;
  uint32_t *tmem_slot = reinterpret_cast<uint32_t *>(bars + 15);
  volatile int *abort_flag = reinterpret_cast<volatile int *>(bars + 16);
  if ((smem_u32(smem) & 1023u) != 0) {
    if (threadIdx.x == 0) atomicOr(&g_error_word, AXB200_ERR_WAIT_TIMEOUT);
    return;
  }
  // heaviest blocks first: the last query block has the most key tiles
  const int h = blockIdx.y, q0 = (gridDim.x - 1 - blockIdx.x) * 2 * kRows;
  const int warp = uniform_warp(), lane = threadIdx.x & 31;
  const int hk = h / p.group;
  const int tile0 = p.window > 0 ? max(0, p.start + q0 + 1 - p.window) / kKeys : 0;  // the first key tile
  int nkv_g[2];
#pragma unroll
  for (int g = 0; g < 2; ++g) {
    const int first = q0 + g * kRows, last = min(first + kRows, p.n) - 1;
    nkv_g[g] = first < p.n ? (min(p.start + last + 1, p.skv) + kKeys - 1) / kKeys - tile0 : 0;
  }
  const int nkv = max(nkv_g[0], nkv_g[1]);

  if (threadIdx.x == 0) {
    for (int i = 0; i < 13; ++i) mbar_init(&bars[i], 1);
    mbar_init(&bar_p[0], 4);
    mbar_init(&bar_p[1], 4);
    *abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == kMmaWarp) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], 512;" ::"r"(smem_u32(tmem_slot)) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  grid_dependency_wait();
  grid_dependency_launch();
  // S_g at g * 128.  With 128 value columns O_g is at 256 + g * 128 and P_g overwrites the front of S_g; with 64,
  // O_g is at 256 + g * 64 and P_g has columns of its own (the products then differ in shape, and the reuse of
  // S_g would lean on the issue order of unlike products).
  const uint32_t tmem = *tmem_slot;
  auto tmem_o = [&](int g) { return tmem + 256 + g * (kVB * 64); };
  auto tmem_p = [&](int g) { return kVB == 2 ? tmem + g * 128 : tmem + 384 + g * 64; };

  if (warp == kLoadWarp) {
    if (lane == 0) {
      tma_prefetch_descriptor(&tmK);
      if (kRot) tma_prefetch_descriptor(&tmKr);
      tma_prefetch_descriptor(&tmV);
      mbar_arrive_expect_tx(bar_q, 2 * L::kTile);
#pragma unroll
      for (int g = 0; g < 2; ++g) {  // rows past n are zero-filled
        uint8_t *dst = smem + g * L::kTile;
        for (int b = 0; b < kQB; ++b) tma_load_3d(dst + b * kBox, &tmQ, bar_q, b * 64, h, q0 + g * kRows);
        if (kRot) tma_load_3d(dst + kQB * kBox, &tmQr, bar_q, 0, h, q0 + g * kRows);
      }
      bool ok = true;
      auto load_k = [&](int t) {
        const int s = t & 1;
        if (t >= 2) ok = mbar_wait_bounded(&empty_k[s], ((t >> 1) - 1) & 1, abort_flag, p.wait_ns);
        if (!ok) return;
        uint8_t *dst = smem + L::kOffK + s * L::kTile;
        mbar_arrive_expect_tx(&full_k[s], L::kTile);
        for (int b = 0; b < kQB; ++b) tma_load_3d(dst + b * kBox, &tmK, &full_k[s], b * 64, hk, (tile0 + t) * kKeys);
        if (kRot) tma_load_3d(dst + kQB * kBox, &tmKr, &full_k[s], 0, 0, (tile0 + t) * kKeys);
      };
      load_k(0);
      int j = 0;
      for (; j < nkv; ++j) {
        if (j + 1 < nkv) load_k(j + 1);
#pragma unroll
        for (int half = 0; half < 2 && ok; ++half) {
          if (j >= 1) ok = mbar_wait_bounded(&empty_v[half], (j - 1) & 1, abort_flag, p.wait_ns);
          if (!ok) break;
          uint8_t *dst = smem + L::kOffV + half * L::kVHalf;
          mbar_arrive_expect_tx(&full_v[half], L::kVHalf);
          for (int b = 0; b < kVB; ++b) tma_load_3d(dst + b * (64 * 64 * 2), &tmV, &full_v[half], b * 64, hk, (tile0 + j) * kKeys + half * 64);
        }
        if (!ok) break;
      }
      if (*abort_flag) {  // no copy may still be on its way when the CTA leaves
        const unsigned long long t0 = global_timer_ns();
        auto drain = [&](uint64_t *bar, uint32_t parity) {
          while (!mbar_try_wait(bar, parity) && global_timer_ns() - t0 < 100000000ull) {
          }
        };
        drain(bar_q, 0);
        for (int t = max(0, j - 1); t <= min(j + 1, nkv - 1); ++t) drain(&full_k[t & 1], (t >> 1) & 1);
        for (int half = 0; half < 2; ++half) drain(&full_v[half], max(0, min(j, nkv - 1) - (j < nkv ? 1 : 0)) & 1);
      }
    }
  } else if (warp == kMmaWarp) {
    if (lane == 0) {
      // fp32 accumulate, bf16 operands, M = 128.  Q.K^T: N = 128, B K-major; P.V: N = kVB * 64, B MN-major
      constexpr uint32_t kBf16 = (1u << 4) | (1u << 7) | (1u << 10) | ((kRows >> 4) << 24);
      constexpr uint32_t idesc_qk = kBf16 | ((kKeys >> 3) << 17), idesc_pv = kBf16 | (1u << 16) | ((kVB * 64 >> 3) << 17);
      const uint64_t dq = smem_desc(smem_u32(smem), 16, 1024);
      const uint64_t dk = smem_desc(smem_u32(smem + L::kOffK), 16, 1024);
      const uint64_t dv = smem_desc(smem_u32(smem + L::kOffV), 64 * 64 * 2, 1024);
      auto issue_s = [&](int g, int t) {
        const uint64_t dqg = dq + (uint64_t)(g * (L::kTile >> 4)), dks = dk + (uint64_t)((t & 1) * (L::kTile >> 4));
#pragma unroll
        for (int ks = 0; ks < L::kBlocks * 4; ++ks) {
          const uint32_t off = ((ks >> 2) * kBox + (ks & 3) * 32) >> 4;
          umma_f16(tmem + g * 128, dqg + off, dks + off, idesc_qk, ks > 0);
        }
        umma_commit(&bar_s[g]);
      };
      bool ok = mbar_wait_bounded(bar_q, 0, abort_flag, p.wait_ns) && mbar_wait_bounded(&full_k[0], 0, abort_flag, p.wait_ns);
      if (ok) {
        tc_fence_after();
        if (nkv_g[0] > 0) issue_s(0, 0);
        if (nkv_g[1] > 0) issue_s(1, 0);
        umma_commit(&empty_k[0]);
      }
      for (int j = 0; j < nkv && ok; ++j) {
        const int last_g = nkv_g[1] > j ? 1 : 0;
        bool have_k = false;
#pragma unroll
        for (int g = 0; g < 2; ++g) {
          if (j >= nkv_g[g]) continue;
          ok = mbar_wait_bounded(&bar_p[g], j & 1, abort_flag, p.wait_ns);
          if (!ok) break;
#pragma unroll
          for (int half = 0; half < 2; ++half) {
            ok = ok && mbar_wait_bounded(&full_v[half], j & 1, abort_flag, p.wait_ns);
            if (!ok) break;
            tc_fence_after();
            const uint64_t dvh = dv + (uint64_t)(half * (L::kVHalf >> 4));
#pragma unroll
            for (int ks = 0; ks < 4; ++ks)  // 16 keys: 8 columns of P, 2 KB of V
              umma_f16_ts(tmem_o(g), tmem_p(g) + half * 32 + ks * 8, dvh + (uint64_t)(ks * (2048 >> 4)), idesc_pv,
                          j > 0 || half > 0 || ks > 0);
            if (g == last_g) umma_commit(&empty_v[half]);
          }
          if (!ok) break;
          if (j == nkv_g[g] - 1) umma_commit(&bar_fin[g]);
          if (j + 1 < nkv_g[g]) {
            if (!have_k) ok = mbar_wait_bounded(&full_k[(j + 1) & 1], ((j + 1) >> 1) & 1, abort_flag, p.wait_ns);
            if (!ok) break;
            have_k = true;
            tc_fence_after();
            issue_s(g, j + 1);
          }
        }
        if (ok && j + 1 < nkv) umma_commit(&empty_k[(j + 1) & 1]);
      }
    }
  } else {
    // ---- softmax warps: query tile g, thread = row ----
    const int g = warp >> 2, row = threadIdx.x & (kRows - 1);
    const int my_nkv = g ? nkv_g[1] : nkv_g[0];
    const int t_row = q0 + g * kRows + row;
    const int kv_end = min(p.start + t_row + 1, p.skv), kv_begin = p.window > 0 ? max(0, p.start + t_row + 1 - p.window) : 0;
    const uint32_t lane_base = (uint32_t)((warp & 3) * 32) << 16;
    const uint32_t ts = tmem + g * 128 + lane_base, to = tmem_o(g) + lane_base, tp = tmem_p(g) + lane_base;
    float m_run = -INFINITY, l_run = 0.f;
    bool ok = true;
    for (int j = 0; j < my_nkv && ok; ++j) {
      ok = __all_sync(0xffffffffu, mbar_wait_bounded(&bar_s[g], j & 1, abort_flag, p.wait_ns));
      if (!ok) break;
      tc_fence_after();
      uint32_t sr[4][32];
#pragma unroll
      for (int c = 0; c < 4; ++c) tmem_ld32_async(ts + c * 32, sr[c]);
      tmem_wait_ld();
      const int n0 = (tile0 + j) * kKeys;
      if (n0 < kv_begin) {
#pragma unroll
        for (int c = 0; c < 4; ++c)
#pragma unroll
          for (int i = 0; i < 32; ++i)
            if (n0 + c * 32 + i < kv_begin) sr[c][i] = 0xff800000u;  // -inf
      }
      if (n0 + kKeys > kv_end) {
#pragma unroll
        for (int c = 0; c < 4; ++c)
#pragma unroll
          for (int i = 0; i < 32; ++i)
            if (n0 + c * 32 + i >= kv_end) sr[c][i] = 0xff800000u;  // -inf
      }
      float mx4[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
      for (int c = 0; c < 4; ++c)
#pragma unroll
        for (int i = 0; i < 32; ++i) mx4[i & 3] = fmaxf(mx4[i & 3], __uint_as_float(sr[c][i]));
      const float mx = fmaxf(fmaxf(mx4[0], mx4[1]), fmaxf(mx4[2], mx4[3]));
      // scale may be negative or zero in principle: the running maximum is kept of the scaled scores
      const float m_tile = mx * p.scale_log2;
      float corr = 1.f;
      const bool moved = __any_sync(0xffffffffu, m_tile > m_run + kLazy);
      if (moved) {
        const float m_new = fmaxf(m_run, m_tile);
        corr = fast_exp2(m_run - ((m_new == -INFINITY) ? 0.f : m_new));
        m_run = m_new;
      }
      const float m_safe = (m_run == -INFINITY) ? 0.f : m_run;
      float sum4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int c = 0; c < 4; ++c) {
        uint32_t packed[16];
#pragma unroll
        for (int i = 0; i < 32; i += 2) {
          const float a = fast_exp2(fmaf(__uint_as_float(sr[c][i]), p.scale_log2, -m_safe));
          const float b = fast_exp2(fmaf(__uint_as_float(sr[c][i + 1]), p.scale_log2, -m_safe));
          sum4[(i >> 1) & 3] += a + b;
          packed[i >> 1] = pack_bf16x2(a, b);
        }
        tmem_st16(tp + c * 16, packed);
      }
      l_run = l_run * corr + ((sum4[0] + sum4[1]) + (sum4[2] + sum4[3]));
      // bar_s of tile j was committed after P(j-1).V_{j-1}: that product is complete and O_g may be rescaled
      if (j > 0 && moved) {
#pragma unroll
        for (int c = 0; c < kVB * 2; ++c) {
          uint32_t r[32];
          tmem_ld32(to + c * 32, r);
#pragma unroll
          for (int i = 0; i < 32; ++i) r[i] = __float_as_uint(__uint_as_float(r[i]) * corr);
          tmem_st32(to + c * 32, r);
        }
      }
      asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&bar_p[g]);
    }
    if (ok && my_nkv > 0) ok = __all_sync(0xffffffffu, mbar_wait_bounded(&bar_fin[g], 0, abort_flag, p.wait_ns));
    tc_fence_after();
    if (ok && my_nkv > 0) {
      float inv = l_run > 0.f ? 1.0f / l_run : 0.f;
      if (p.sink) {
        const float s = p.sink[h] * kLog2e, top = fmaxf(m_run, s), w = fast_exp2(m_run - top);
        inv = w / fmaf(l_run, w, fast_exp2(s - top));
      }
      __nv_bfloat16 *dst = p.out + ((size_t)t_row * p.heads + h) * p.vdim;
#pragma unroll
      for (int c = 0; c < kVB * 2; ++c) {
        uint32_t r[32];
        tmem_ld32(to + c * 32, r);
        if (t_row < p.n) {
#pragma unroll
          for (int u = 0; u < 4; ++u) {
            if (c * 32 + u * 8 >= p.vdim) break;
            uint4 w;
            w.x = pack_bf16x2(__uint_as_float(r[u * 8 + 0]) * inv, __uint_as_float(r[u * 8 + 1]) * inv);
            w.y = pack_bf16x2(__uint_as_float(r[u * 8 + 2]) * inv, __uint_as_float(r[u * 8 + 3]) * inv);
            w.z = pack_bf16x2(__uint_as_float(r[u * 8 + 4]) * inv, __uint_as_float(r[u * 8 + 5]) * inv);
            w.w = pack_bf16x2(__uint_as_float(r[u * 8 + 6]) * inv, __uint_as_float(r[u * 8 + 7]) * inv);
            *reinterpret_cast<uint4 *>(dst + c * 32 + u * 8) = w;
          }
        }
      }
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == kMmaWarp)
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, 512;" ::"r"(tmem) : "memory");
}

// (rows, heads, elems) with row and head strides in elements -> boxes of [box_rows rows][64 elements]
bool map_of(CUtensorMap *map, const void *base, int elems, int heads, int64_t rows, int64_t head_stride, int64_t row_stride,
            int box_rows) {
  EncodeTiledFn fn = tensor_map_encoder();
  const cuuint64_t dims[3] = {(cuuint64_t)elems, (cuuint64_t)heads, (cuuint64_t)rows};
  const cuuint64_t strides[2] = {(cuuint64_t)head_stride * 2, (cuuint64_t)row_stride * 2};
  const cuuint32_t box[3] = {64, 1, (cuuint32_t)box_rows}, es[3] = {1, 1, 1};
  return fn && fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void *>(base), dims, strides, box, es,
                  CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                  CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

template <int kQB, int kVB, int kRot>
int launch(const CUtensorMap (&m)[5], const Params &p, cudaStream_t st) {
  using L = Layout<kQB, kVB, kRot>;
  auto *kernel = latent_prefill_kernel<kQB, kVB, kRot>;
  static std::mutex mu;
  static bool opted[64] = {false};
  int dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return AXB200_DEVICE_ERROR;
  {
    std::lock_guard<std::mutex> lock(mu);
    if (!opted[dev]) {
      if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, L::kSmem) != cudaSuccess)
        return AXB200_DEVICE_ERROR;
      opted[dev] = true;
    }
  }
  const dim3 grid((p.n + 2 * kRows - 1) / (2 * kRows), p.heads);
  return launch_dependent(kernel, grid, dim3(kThreads), L::kSmem, st, m[0], m[1], m[2], m[3], m[4], p);
}

bool al16(const void *p) { return (reinterpret_cast<uintptr_t>(p) & 15u) == 0; }

}  // namespace
}  // namespace axb

extern "C" {

int axb200_latent_prefill_supported(int heads, int dim, int rot_dim, int vdim, int dtype) {
  return dtype == AXB200_BFLOAT16 && heads > 0 && heads <= 65535 && dim >= 8 && dim <= 128 && dim % 8 == 0 && rot_dim >= 0 &&
         rot_dim <= 64 && rot_dim % 8 == 0 && vdim >= 8 && vdim <= 128 && vdim % 8 == 0;
}

int axb200_latent_prefill(const void *q, int64_t q_ld, const void *k, const void *v, const void *rot, int64_t rot_ld,
                          const float *sink, void *out, int n, int64_t start, int heads, int kv_heads, int dim, int rot_dim,
                          int vdim, int window, float scale, int dtype, void *stream) {
  if (!axb200_latent_prefill_supported(heads, dim, rot_dim, vdim, dtype)) return AXB200_UNSUPPORTED_TYPE;
  if (!q || !k || !v || (rot_dim > 0 && !rot) || !out) return AXB200_INVALID_PTR;
  if (n < 0 || start < 0 || start + n > 0x7fffffff - 4096 || !(scale > 0.f) || kv_heads <= 0 || heads % kv_heads != 0 || window < 0)
    return AXB200_INVALID_ARGUMENT;
  if (q_ld < (int64_t)heads * (dim + rot_dim) || rot_ld < rot_dim) return AXB200_SHAPE_MISMATCH;
  if (q_ld % 8 || rot_ld % 8 || !axb::al16(q) || !axb::al16(k) || !axb::al16(v) || !axb::al16(rot) || !axb::al16(out))
    return AXB200_UNSUPPORTED_TYPE;
  if (n == 0) return AXB200_OK;
  const int per = dim + rot_dim;
  const int64_t skv = start + n;
  CUtensorMap m[5] = {};
  const __nv_bfloat16 *qb = static_cast<const __nv_bfloat16 *>(q);
  if (!axb::map_of(&m[0], qb, dim, heads, n, per, q_ld, axb::kRows) ||
      !axb::map_of(&m[2], k, dim, kv_heads, skv, dim, (int64_t)kv_heads * dim, axb::kKeys) ||
      !axb::map_of(&m[4], v, vdim, kv_heads, skv, vdim, (int64_t)kv_heads * vdim, 64))
    return AXB200_INTERNAL_ERROR;
  if (rot_dim > 0 && (!axb::map_of(&m[1], qb + dim, rot_dim, heads, n, per, q_ld, axb::kRows) ||
                      !axb::map_of(&m[3], rot, rot_dim, 1, skv, rot_ld, rot_ld, axb::kKeys)))
    return AXB200_INTERNAL_ERROR;
  axb::Params p{static_cast<__nv_bfloat16 *>(out), n, (int)start, (int)skv, heads, heads / kv_heads, vdim, window, sink,
                scale * axb::kLog2e, axb::wait_limit_ns()};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  auto go = [&](auto rot_tag) {
    constexpr int kRot = decltype(rot_tag)::value;
    if (dim > 64) return vdim > 64 ? axb::launch<2, 2, kRot>(m, p, st) : axb::launch<2, 1, kRot>(m, p, st);
    return vdim > 64 ? axb::launch<1, 2, kRot>(m, p, st) : axb::launch<1, 1, kRot>(m, p, st);
  };
  return rot_dim > 0 ? go(std::integral_constant<int, 1>{}) : go(std::integral_constant<int, 0>{});
}

}  // extern "C"
