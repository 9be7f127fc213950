// Latent attention (latent_attn.cu) in bf16 on the 5th-generation tensor cores, in the cached form: decoded
// tokens and short portions.
//
// The cached rows are the M side of both products, the heads the N side:
//     S^T (keys x heads)   = rows . Q^T            M = 128 keys, K = the row's kv_rank + rot_dim elements
//     O^T (latent x heads) = C^T  . P^T            M = 128 latent elements at a time, K = 128 keys
// so a tile of 128 cached rows is staged once by TMA and is operand A of both (K-major for the scores, MN-major for
// the sum), and 16 or 32 heads cost the same tensor time, less than reading the rows takes.  The other way round,
// 128 query rows would fill shared memory, and 16 heads would waste 7 / 8 of them.
//
// Thread = key: the scores of a key for all heads stand in one lane of tensor memory.  The running maximum of a head
// is a reference that moves only when some key exceeds it by 2^8 (a vote among the 128 threads, no reduction); sums
// over keys stay in registers, one per head, until the item ends.  The weights go to shared memory as P (heads x
// keys).  A moved reference rescales O^T in tensor memory.
//
// Work: an item is (row, tile of heads).  The 128-key tiles of all rows are laid end to end and cut into equal
// ranges, one per group of CTAs, a CTA of the group for each tile of heads - they walk the same cached rows side by
// side and all but one of them read from L2.  The cut is made from the positions in device memory, so a captured
// graph stays balanced as the cache grows.  An item that lies in one range is finished there; otherwise every range
// leaves an un-normalised record, and the merge kernel adds them up.
//
// Warps 0-3: softmax, queries into shared memory, results; warps 4 and 6: the products of the scores and of the sum (one
// warp's issue of small products, not the tensor core, would set the pace of both); one lane of warp 5: TMA.  The staged chunks
// (128 keys x 64 elements) lie in rings: pairs of chunks that hold latent elements, freed when their part of the sum
// is done, and single chunks with the rest of the row (the rotated part), freed after the scores.  Every wait is
// bounded.
#include <math.h>

#include <mutex>

#include "latent_attn.cuh"

namespace axb {
namespace {

constexpr int kKeys = 128, kChunk = kKeys * 128;  // bytes of a chunk
constexpr int kThreads = 224, kMmaWarp = 4, kLoadWarp = 5, kSumWarp = 6, kSoftmax = 128;
constexpr int kMaxRows = 1024, kMinTiles = 2, kMaxCtas = 256, kMaxSlots = 8;
constexpr float kLog2e = 1.4426950408889634f, kLazy = 8.0f;

struct UmmaAttend {
  AttendParams a;
  int part_tiles;          // tiles of heads that read one part of the rows
  int head_tiles, groups;  // kv_heads * part_tiles
  int pairs, singles;            // per tile
  int pair_slots, single_slots;  // in the rings
  int chunks;                    // per row: ceil(elements / 64)
  int p_slots;                   // buffers of P: two where the rings hold two tiles, so that scores run ahead of sums
  float *part_o;                 // (2 * CTAs, N, kv_rank)
  float2 *part_ml;               // (2 * CTAs, N): reference (log2 domain), sum
};

// Tiles start at the multiple of 64 keys (half a tile lies in one page) at or before the row's first key.
__device__ __forceinline__ int first_tile_key(const AttendParams &p, int r) { return first_key(p, r) & ~63; }
__device__ __forceinline__ int tiles_of(const AttendParams &p, int r) {
  return max(0, visible_keys(p, r) - first_tile_key(p, r) + kKeys - 1) / kKeys;
}
__device__ __forceinline__ int tiles_per_group(int total, int groups) { return max(kMinTiles, (total + groups - 1) / groups); }

// start[r] = key tiles of the rows before r, r = 0 .. rows; all threads of the CTA.
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

// What un-normalised results with sum l at reference ref (log2 domain) are multiplied by when a sink joins the sum.
__device__ __forceinline__ float inverse_with_sink(float ref, float l, float sink) {
  const float s = sink * kLog2e, top = fmaxf(ref, s), w = fast_exp2(ref - top);
  return w / fmaf(l, w, fast_exp2(s - top));
}

// Whether any of the 128 softmax threads says so.
__device__ __forceinline__ bool any_of_softmax(bool mine) {
  uint32_t r;
  asm volatile(
      "{\n.reg .pred p, q;\nsetp.ne.u32 p, %1, 0;\nbarrier.cta.red.or.pred q, 1, 128, p;\nselp.u32 %0, 1, 0, q;\n}\n"
      : "=r"(r)
      : "r"((uint32_t)mine)
      : "memory");
  return r != 0;
}

// Reduces v[h], h < kN, over the 32 lanes by halving exchanges; a lane ends with the result of head
// lane * kN / 32 (below 32 heads several lanes have the same one).
template <int kN, typename Op>
__device__ __forceinline__ float reduce_heads(float (&v)[kN], int lane, Op op) {
  int n = kN;
#pragma unroll
  for (int off = 16; off > 0; off >>= 1) {
    if (n > 1) {
      n >>= 1;
      const bool upper = lane & off;
#pragma unroll
      for (int i = 0; i < kN / 2; ++i)
        if (i < n) {
          const float send = upper ? v[i] : v[i + n], keep = upper ? v[i + n] : v[i];
          v[i] = op(keep, __shfl_xor_sync(0xffffffffu, send, off));
        }
    } else {
      v[0] = op(v[0], __shfl_xor_sync(0xffffffffu, v[0], off));
    }
  }
  return v[0];
}

template <int kN>
__device__ __forceinline__ void tmem_ld_heads(uint32_t taddr, float (&v)[kN]) {
  if constexpr (kN == 4) {
    asm volatile("tcgen05.ld.sync.aligned.32x32b.x4.b32 {%0,%1,%2,%3}, [%4];" : "=f"(v[0]), "=f"(v[1]), "=f"(v[2]), "=f"(v[3]) : "r"(taddr));
  } else if constexpr (kN == 8) {
    asm volatile("tcgen05.ld.sync.aligned.32x32b.x8.b32 {%0,%1,%2,%3,%4,%5,%6,%7}, [%8];"
                 : "=f"(v[0]), "=f"(v[1]), "=f"(v[2]), "=f"(v[3]), "=f"(v[4]), "=f"(v[5]), "=f"(v[6]), "=f"(v[7])
                 : "r"(taddr));
  } else {
#pragma unroll
    for (int c = 0; c < kN; c += 16) tmem_ld16_async(taddr + c, reinterpret_cast<uint32_t(&)[16]>(v[c]));
  }
  tmem_wait_ld();
}

template <int kN>
__device__ __forceinline__ void tmem_st_heads(uint32_t taddr, float (&v)[kN]) {
  if constexpr (kN == 4) {
    asm volatile("tcgen05.st.sync.aligned.32x32b.x4.b32 [%0], {%1,%2,%3,%4};" ::"r"(taddr), "f"(v[0]), "f"(v[1]), "f"(v[2]), "f"(v[3]) : "memory");
  } else if constexpr (kN == 8) {
    asm volatile("tcgen05.st.sync.aligned.32x32b.x8.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8};" ::"r"(taddr), "f"(v[0]), "f"(v[1]), "f"(v[2]),
                 "f"(v[3]), "f"(v[4]), "f"(v[5]), "f"(v[6]), "f"(v[7])
                 : "memory");
  } else {
#pragma unroll
    for (int c = 0; c < kN; c += 16) tmem_st16(taddr + c, reinterpret_cast<uint32_t(&)[16]>(v[c]));
  }
}

// The heads' references out of shared memory; before an item's first tile they may be anything.
template <int kN>
__device__ __forceinline__ void load_refs(const float *ref, float (&v)[kN]) {
#pragma unroll
  for (int h = 0; h < kN; h += 4) {
    const float4 t = *reinterpret_cast<const float4 *>(ref + h);
    v[h] = t.x, v[h + 1] = t.y, v[h + 2] = t.z, v[h + 3] = t.w;
  }
}

// fp32 accumulators, bf16 operands, M = 128, N = kN
template <int kN>
constexpr uint32_t kIdesc = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(kN >> 3) << 17) | ((128u >> 4) << 24);

template <int kN>
struct Smem {
  static constexpr int kP = kN * kKeys * 2;
  static constexpr int kQBox = kN * 128;
  // after the rings: Q (chunks boxes), P, the keys' factors (for each pair slot, filled with a tile's first pair),
  // reference and reduction scratch, barriers, row starts
  __host__ __device__ static int off_q(const UmmaAttend &u) { return u.pair_slots * 2 * kChunk + u.single_slots * kChunk; }
  __host__ __device__ static int off_p(const UmmaAttend &u) { return off_q(u) + u.chunks * kQBox; }
  __host__ __device__ static int off_factor(const UmmaAttend &u) { return off_p(u) + u.p_slots * kP; }
  __host__ __device__ static int off_ref(const UmmaAttend &u) { return off_factor(u) + (u.a.key_scale ? u.pair_slots * kKeys * 4 : 0); }
  __host__ __device__ static int off_red(const UmmaAttend &u) { return off_ref(u) + 2 * kN * 4; }
  __host__ __device__ static int off_bar(const UmmaAttend &u) { return off_red(u) + 4 * kN * 4; }
  __host__ __device__ static int off_start(const UmmaAttend &u) { return off_bar(u) + 512; }
  __host__ __device__ static int bytes(const UmmaAttend &u, int rows) { return off_start(u) + (rows + 1) * 4; }
};

// kN: heads of a tile, the products' N side; kH <= kN: how many of them a part can have (the softmax skips the rest, whose
// columns hold nothing that is read).
template <int kN, int kH>
__global__ void __launch_bounds__(kThreads, 1)
latent_umma_kernel(const __grid_constant__ CUtensorMap tmPages, const __grid_constant__ UmmaAttend u) {
  using S = Smem<kN>;
  extern __shared__ __align__(1024) uint8_t smem[];
  const AttendParams &p = u.a;
  uint64_t *full_p = reinterpret_cast<uint64_t *>(smem + S::off_bar(u)), *empty_p = full_p + kMaxSlots;
  uint64_t *full_s = empty_p + kMaxSlots, *empty_s = full_s + kMaxSlots;
  uint64_t *bar_s = empty_s + kMaxSlots, *bar_o = bar_s + 2, *bar_p = bar_o + 2, *bar_q = bar_p + 2;
  uint32_t *tmem_slot = reinterpret_cast<uint32_t *>(bar_q + 1);
  volatile int *abort_flag = reinterpret_cast<volatile int *>(bar_q + 2);
  int *start = reinterpret_cast<int *>(smem + S::off_start(u));
  if ((smem_u32(smem) & 1023u) != 0) {
    if (threadIdx.x == 0) atomicOr(&g_error_word, AXB200_ERR_WAIT_TIMEOUT);
    return;
  }
  const int warp = uniform_warp(), lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    for (int i = 0; i < 4 * kMaxSlots + 4; ++i) mbar_init(&full_p[i], 1);  // rings, bar_s and bar_o
    mbar_init(&bar_p[0], 4);
    mbar_init(&bar_p[1], 4);
    mbar_init(bar_q, 4);
    *abort_flag = 0;
    mbar_fence_init();
  }
  grid_dependency_wait();
  grid_dependency_launch();
  scan_tiles(p, start);
  __syncthreads();
  const int total = start[p.rows], per = tiles_per_group(total, u.groups);
  const int lo = (int)(blockIdx.x / u.head_tiles) * per, hi = min(total, lo + per);
  if (lo >= hi) return;
  const int head_tile = (int)(blockIdx.x % u.head_tiles), part = head_tile / u.part_tiles, part_heads = p.heads / p.kv_heads;
  const int h0 = part * part_heads + (head_tile - part * u.part_tiles) * kN, h_end = (part + 1) * part_heads;
  // the row that holds tile lo: the last r with start[r] <= lo
  int r_first = 0;
  for (int a = 0, b = p.rows - 1; a < b;) {
    const int m = (a + b + 1) >> 1;
    if (start[m] <= lo)
      a = m;
    else
      b = m - 1;
    r_first = a;
  }

  constexpr uint32_t kTmemCols = kN == 16 ? 128 : 256;  // two S buffers and up to four O tiles of kN columns
  if (warp == kMmaWarp) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(tmem_slot)), "n"(kTmemCols) : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot, tmem_o = tmem + 2 * kN;
  const int off_single = u.pair_slots * 2 * kChunk;

  if (warp == kLoadWarp) {
    // ================= loader (one lane) =================
    if (lane == 0) {
      tma_prefetch_descriptor(&tmPages);
      RingPos rp, rs;      // chunk pairs and singles
      int np = 0, ns = 0;  // how many were issued
      bool ok = true;
      for (int r = r_first, g = lo; g < hi && ok; ++r) {
        const int keys = visible_keys(p, r), key0 = first_tile_key(p, r);
        const int32_t *table = p.block_table + (size_t)p.row_seq[r] * p.max_blocks;
        for (; g < hi && g < start[r + 1] && ok; ++g) {
          const int t0 = key0 + (g - start[r]) * kKeys;
          // two halves of 64 keys, each within one page; a half past the end is not loaded
          const int halves = keys - t0 > 64 ? 2 : 1;
          int at[2], page_at[2];
#pragma unroll
          for (int i = 0; i < 2; ++i) {
            const int t = t0 + 64 * (i < halves ? i : 0);
            int page = table[t / p.page_tokens];
            if (page < 0 || page >= p.num_pages) {
              atomicOr(&g_error_word, AXB200_ERR_BAD_PAGE);
              page = 0;
            }
            at[i] = t % p.page_tokens;
            page_at[i] = page;
          }
          auto load_chunk = [&](uint8_t *dst, uint64_t *bar, int c) {
            for (int i = 0; i < halves; ++i) tma_load_4d(dst + i * (kChunk / 2), &tmPages, bar, c * 64, part, at[i], page_at[i]);
          };
          for (int i = 0; i < u.singles && ok; ++i, ++ns, rs.next(u.single_slots)) {
            const int s = rs.slot;
            if (ns >= u.single_slots) ok = mbar_wait_bounded(&empty_s[s], rs.parity ^ 1, abort_flag, p.wait_ns);
            if (!ok) break;
            mbar_arrive_expect_tx(&full_s[s], halves * (kChunk / 2));
            load_chunk(smem + off_single + s * kChunk, &full_s[s], 2 * u.pairs + i);
          }
          for (int i = 0; i < u.pairs && ok; ++i, ++np, rp.next(u.pair_slots)) {
            const int s = rp.slot, n = min(2, u.chunks - 2 * i);
            if (np >= u.pair_slots) ok = mbar_wait_bounded(&empty_p[s], rp.parity ^ 1, abort_flag, p.wait_ns);
            if (!ok) break;
            const bool factors = p.key_scale && i == 0;
            mbar_arrive_expect_tx(&full_p[s], n * halves * (kChunk / 2) + (factors ? halves * 256 : 0));
            if (factors)
              for (int k = 0; k < halves; ++k)
                bulk_load(smem + S::off_factor(u) + s * kKeys * 4 + k * 256,
                          page_factors(static_cast<const __nv_bfloat16 *>(p.pages) + (size_t)page_at[k] * p.page_elems, p) + at[k], 256,
                          &full_p[s]);
            for (int c = 0; c < n; ++c) load_chunk(smem + s * 2 * kChunk + c * kChunk, &full_p[s], 2 * i + c);
          }
        }
      }
      if (*abort_flag) {  // no copy may still be on its way when the CTA leaves
        const unsigned long long t0 = global_timer_ns();
        auto drain = [&](uint64_t *full, int issued, int slots) {
          for (int j = max(0, issued - slots); j < issued; ++j)
            while (!mbar_try_wait(&full[j % slots], (j / slots) & 1) && global_timer_ns() - t0 < 100000000ull) {
            }
        };
        drain(full_p, np, u.pair_slots);
        if (u.singles) drain(full_s, ns, u.single_slots);
      }
    }
  } else if (warp == kMmaWarp) {
    // ================= products of the scores (the warp walks, one lane issues) =================
    const uint32_t lead = lane == 0;
    constexpr uint32_t idesc = kIdesc<kN>;                                // A K-major
    const uint64_t da = smem_desc(smem_u32(smem), 16, 1024);             // a chunk as [keys][elements]
    const uint64_t dq = smem_desc(smem_u32(smem + S::off_q(u)), 16, 1024);
    RingPos rp, rs;
    bool ok = true;
    for (int r = r_first, g = lo, tile = 0, seg = 0; g < hi && ok; ++g, ++tile) {
      while (start[r + 1] <= g) ++r;
      if (g == lo || g == start[r]) {  // a new item: its queries are in place
        ok = mbar_wait_warp(bar_q, seg & 1, abort_flag, p.wait_ns);
        ++seg;
      }
      // the scores two tiles back have been read
      if (tile >= 2) ok = ok && mbar_wait_warp(&bar_p[tile & 1], ((tile - 2) >> 1) & 1, abort_flag, p.wait_ns);
      const uint32_t ts = tmem + (tile & 1) * kN;
      bool first = true;
      auto score_chunk = [&](int offset, int c) {
        const uint64_t a = da + (uint64_t)(offset >> 4), b = dq + (uint64_t)(c * (S::kQBox >> 4));
#pragma unroll
        for (int ks = 0; ks < 4; ++ks) umma_f16_lead(ts, a + ks * 2, b + ks * 2, idesc, !first || ks > 0, lead);
        first = false;
      };
      for (int i = 0; i < u.singles && ok; ++i, rs.next(u.single_slots)) {
        const int s = rs.slot;
        ok = mbar_wait_warp(&full_s[s], rs.parity, abort_flag, p.wait_ns);
        if (!ok) break;
        tc_fence_after();
        score_chunk(off_single + s * kChunk, 2 * u.pairs + i);
        umma_commit_lead(&empty_s[s], lead);
      }
      for (int i = 0; i < u.pairs && ok; ++i, rp.next(u.pair_slots)) {
        const int s = rp.slot;
        ok = mbar_wait_warp(&full_p[s], rp.parity, abort_flag, p.wait_ns);
        if (!ok) break;
        tc_fence_after();
        for (int c = 0; c < 2 && 2 * i + c < u.chunks; ++c) score_chunk(s * 2 * kChunk + c * kChunk, 2 * i + c);
      }
      if (ok) umma_commit_lead(&bar_s[tile & 1], lead);
    }
  } else if (warp == kSumWarp) {
    // ================= products of the sum =================
    const uint32_t lead = lane == 0;
    constexpr uint32_t idesc = kIdesc<kN> | (1u << 15);             // A MN-major
    const uint64_t dv = smem_desc(smem_u32(smem), kChunk, 1024);    // a pair as latent elements x keys
    const uint64_t dp = smem_desc(smem_u32(smem + S::off_p(u)), 16, 1024);
    RingPos pv;
    for (int r = r_first, g = lo, tile = 0; g < hi; ++g, ++tile) {
      while (start[r + 1] <= g) ++r;
      if (!mbar_wait_warp(&bar_p[tile & 1], (tile >> 1) & 1, abort_flag, p.wait_ns)) break;
      tc_fence_after();
      const bool fresh = g == lo || g == start[r];
      const uint64_t dpt = dp + (uint64_t)((u.p_slots == 2 ? tile & 1 : 0) * (S::kP >> 4));
      for (int i = 0; i < u.pairs; ++i, pv.next(u.pair_slots)) {
        const int s = pv.slot;
        const uint64_t a = dv + (uint64_t)(s * (2 * kChunk >> 4));
#pragma unroll
        for (int ks = 0; ks < kKeys / 16; ++ks)  // 16 keys: 2 KB of the chunk, 32 bytes of P
          umma_f16_lead(tmem_o + i * kN, a + (uint64_t)(ks * (2048 >> 4)),
                        dpt + (uint64_t)(((ks >> 2) * (kN * 128) + (ks & 3) * 32) >> 4), idesc, !fresh || ks > 0, lead);
        umma_commit_lead(&empty_p[s], lead);
      }
      umma_commit_lead(&bar_o[tile & 1], lead);
    }
  } else {
    // ================= softmax warps: thread = key of the tile =================
    float *ref = reinterpret_cast<float *>(smem + S::off_ref(u)), *corr_s = ref + kN;
    float(*red)[kN] = reinterpret_cast<float(*)[kN]>(smem + S::off_red(u));
    uint8_t *qs = smem + S::off_q(u), *ps = smem + S::off_p(u);
    const uint32_t lane_base = (uint32_t)(warp * 32) << 16;
    const float scale_log2 = p.scale * kLog2e;
    const int tid = threadIdx.x, elems = p.kv_rank + p.rot_dim;
    int tile = 0, seg = 0, np = 0;
    bool ok = true;
    // an item's queries, heads x elements, in 16-byte pieces into the swizzled boxes
    auto put_queries = [&](int r) {
      for (int i = tid; i < kN * u.chunks * 8; i += kSoftmax) {
        const int h = i / (u.chunks * 8), e = (i - h * (u.chunks * 8)) * 8;
        uint4 v = make_uint4(0, 0, 0, 0);
        if (h0 + h < h_end && e < elems)
          v = e < p.kv_rank ? *reinterpret_cast<const uint4 *>(static_cast<const __nv_bfloat16 *>(p.q_lat) +
                                                               ((size_t)r * p.heads + h0 + h) * p.kv_rank + e)
                            : *reinterpret_cast<const uint4 *>(static_cast<const __nv_bfloat16 *>(p.q) + (size_t)r * p.q_ld +
                                                               (size_t)(h0 + h) * (p.dim + p.rot_dim) + p.dim + (e - p.kv_rank));
        *reinterpret_cast<uint4 *>(qs + (e >> 6) * S::kQBox + h * 128 + ((((e >> 3) & 7) ^ (h & 7)) << 4)) = v;
      }
      asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
      __syncwarp();
      if (lane == 0) mbar_arrive(bar_q);
    };
    const float *factors = reinterpret_cast<const float *>(smem + S::off_factor(u));
    RingPos fp;  // of a tile's first pair
    for (int r = r_first, g = lo; g < hi && ok; ++r) {
      if (start[r + 1] <= g) continue;
      const int k_first = g - start[r], g_end = min(hi, start[r + 1]), keys = visible_keys(p, r);
      const int key0 = first_tile_key(p, r), hidden = first_key(p, r) - key0;  // keys of the first tile before the window
      if (seg == 0) put_queries(r);
      ++seg;
      float l[kH];
#pragma unroll
      for (int h = 0; h < kH; ++h) l[h] = 0.f;
      for (const int g_first = g; g < g_end; ++g, ++tile, np += u.pairs) {
        const int valid = min(kKeys, keys - key0 - (g - start[r]) * kKeys);
        const bool seen = tid < valid && (g > start[r] || tid >= hidden);
        float factor = scale_log2;
        ok = mbar_wait_warp(&bar_s[tile & 1], (tile >> 1) & 1, abort_flag, p.wait_ns) && ok;
        tc_fence_after();
        if (p.key_scale) {
          ok = mbar_wait_warp(&full_p[fp.slot], fp.parity, abort_flag, p.wait_ns) && ok;
          factor *= factors[fp.slot * kKeys + tid];
          for (int i = 0; i < u.pairs; ++i) fp.next(u.pair_slots);
        }
        // the last tile's sum has to be done before O^T is rescaled, that of `p_slots` tiles back before its weights are
        // overwritten
        auto wait_sum = [&](int back) {
          if (tile >= back) ok = mbar_wait_warp(&bar_o[(tile - back) & 1], ((tile - back) >> 1) & 1, abort_flag, p.wait_ns) && ok;
          tc_fence_after();
        };
        float s[kH], rf[kH];
        load_refs<kH>(ref, rf);
        if (ok) {
          tmem_ld_heads<kH>(tmem + (tile & 1) * kN + lane_base, s);
        } else {
#pragma unroll
          for (int h = 0; h < kH; ++h) s[h] = 0.f;
        }
        float most = -INFINITY;  // how far a score exceeds its head's reference
#pragma unroll
        for (int h = 0; h < kH; ++h) {
          s[h] = seen ? s[h] * factor : -INFINITY;
          most = fmaxf(most, s[h] - rf[h]);
        }
        const bool over = g == g_first || most > kLazy;
        // a warp that gave up says so here, and all four leave together
        if (any_of_softmax(over || !ok)) {
          if (any_of_softmax(!ok)) {
            ok = false;
            break;
          }
          // the references move: the maximum over the tile, head by head
          float t[kH];
#pragma unroll
          for (int h = 0; h < kH; ++h) t[h] = s[h];
          const float best = reduce_heads<kH>(t, lane, [](float a, float b) { return fmaxf(a, b); });
          if (lane % (32 / kH) == 0) red[warp][lane * kH / 32] = best;
          named_bar_sync(1, kSoftmax);
          if (tid < kH) {
            float m = fmaxf(fmaxf(red[0][tid], red[1][tid]), fmaxf(red[2][tid], red[3][tid]));
            const float old = g == g_first ? -INFINITY : ref[tid];
            m = fmaxf(m, old);
            if (m == -INFINITY) m = 0.f;
            corr_s[tid] = fast_exp2(old - m);
            ref[tid] = m;
          }
          named_bar_sync(1, kSoftmax);
          load_refs<kH>(ref, rf);
          if (g > g_first) {
#pragma unroll
            for (int h = 0; h < kH; ++h) l[h] *= corr_s[h];
            wait_sum(1);
            for (int i = 0; i < u.pairs; ++i) {
              float o[kH];
              tmem_ld_heads<kH>(tmem_o + i * kN + lane_base, o);
#pragma unroll
              for (int h = 0; h < kH; ++h) o[h] *= corr_s[h];
              tmem_st_heads<kH>(tmem_o + i * kN + lane_base, o);
            }
            asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory");
          }
        }
        uint8_t *pk = ps + (u.p_slots == 2 ? tile & 1 : 0) * S::kP + (tid >> 6) * (kN * 128) + (tid & 7) * 2;
        const int chunk = (tid >> 3) & 7;
#pragma unroll
        for (int h = 0; h < kH; ++h) {
          s[h] = fast_exp2(s[h] - rf[h]);
          l[h] += s[h];
        }
        wait_sum(u.p_slots);
#pragma unroll
        for (int h = 0; h < kH; ++h)
          *reinterpret_cast<__nv_bfloat16 *>(pk + h * 128 + ((chunk ^ (h & 7)) << 4)) = __float2bfloat16_rn(s[h]);
        if (valid < kKeys) {
          // the sequence's last tile: what stands in the rows past its end is not its own, and weight 0 is not
          // enough against a NaN: clear them where the sum will read them
          const int pieces = (kKeys - valid) * 8;
          for (int i = 0; i < 2 * u.pairs; ++i) {
            uint8_t *c = smem + (np + (i >> 1)) % u.pair_slots * 2 * kChunk + (i & 1) * kChunk + valid * 128;
            for (int j = tid; j < pieces; j += kSoftmax) *reinterpret_cast<uint4 *>(c + j * 16) = make_uint4(0, 0, 0, 0);
          }
        }
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
        tc_fence_before();
        __syncwarp();
        if (lane == 0) mbar_arrive(&bar_p[tile & 1]);
      }
      if (!ok) break;
      // The scores of the item's last tile are done (bar_s), so its queries may be replaced: the next item's first
      // scores are then computed while this item's result is stored.
      if (g < hi) {
        int r_next = r + 1;
        while (start[r_next + 1] <= g) ++r_next;
        put_queries(r_next);
      }
      // ---- the item, or this range's part of it ----
      const float sum = reduce_heads<kH>(l, lane, [](float a, float b) { return a + b; });
      if (lane % (32 / kH) == 0) red[warp][lane * kH / 32] = sum;
      ok = mbar_wait_warp(&bar_o[(tile - 1) & 1], ((tile - 1) >> 1) & 1, abort_flag, p.wait_ns) && ok;
      tc_fence_after();
      if (any_of_softmax(!ok)) {  // also: red is complete
        ok = false;
        break;
      }
      const bool whole = k_first == 0 && g_end == start[r + 1];
      const int slot = (int)blockIdx.x * 2 + (k_first == 0 ? 1 : 0);
      if (!whole && tid < kH) u.part_ml[slot * kN + tid] = make_float2(ref[tid], red[0][tid] + red[1][tid] + red[2][tid] + red[3][tid]);
      for (int i = 0; i < u.pairs; ++i) {
        float o[kH];
        tmem_ld_heads<kH>(tmem_o + i * kN + lane_base, o);
        const int e = i * 128 + tid;
        if (e >= p.kv_rank) continue;
#pragma unroll
        for (int h = 0; h < kH; ++h) {
          if (whole) {
            if (h0 + h < h_end) {
              const float lt = red[0][h] + red[1][h] + red[2][h] + red[3][h];
              const float inv = p.sink ? inverse_with_sink(ref[h], lt, p.sink[h0 + h]) : 1.0f / lt;
              static_cast<__nv_bfloat16 *>(p.out)[((size_t)r * p.heads + h0 + h) * p.kv_rank + e] = __float2bfloat16_rn(o[h] * inv);
            }
          } else {
            u.part_o[((size_t)slot * kN + h) * p.kv_rank + e] = o[h];
          }
        }
      }
      named_bar_sync(1, kSoftmax);  // red, ref and the O tiles may be written again
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == kMmaWarp)
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "n"(kTmemCols) : "memory");
}

// Merges the records of the items that were cut: one CTA per (row, head).
constexpr int kMergeThreads = 128;
template <int kN>
__global__ void __launch_bounds__(kMergeThreads) latent_merge_kernel(const UmmaAttend u) {
  __shared__ int scratch[2][kMergeThreads / 32];
  __shared__ float weight[kMaxCtas];
  const AttendParams &p = u.a;
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
  const int n = tiles_of(p, r), per = tiles_per_group(all, u.groups);
  __nv_bfloat16 *out = static_cast<__nv_bfloat16 *>(p.out) + ((size_t)r * p.heads + h) * p.kv_rank;
  if (n == 0) {  // a row that sees nothing
    for (int e = threadIdx.x; e < p.kv_rank; e += kMergeThreads) stf(out + e, 0.f);
    return;
  }
  const int first = before / per, last = (before + n - 1) / per, count = last - first + 1;
  if (count == 1) return;
  // records: the range that holds the item's first tile filed it under 1, the later ones under 0
  const int part_heads = p.heads / p.kv_heads, in_part = h % part_heads, head_tile = h / part_heads * u.part_tiles + in_part / kN;
  auto slot = [&](int c) { return (((first + c) * u.head_tiles + head_tile) * 2 + (c == 0 ? 1 : 0)) * kN + in_part % kN; };
  float top = -INFINITY, sum = 0.f;
  for (int c = 0; c < count; ++c) top = fmaxf(top, u.part_ml[slot(c)].x);
  for (int c = 0; c < count; ++c) {
    const float2 ml = u.part_ml[slot(c)];
    const float w = fast_exp2(ml.x - top);
    sum = fmaf(w, ml.y, sum);
    if (threadIdx.x == 0) weight[c] = w;
  }
  __syncthreads();
  const float inv = p.sink ? inverse_with_sink(top, sum, p.sink[h]) : sum > 0.f ? 1.0f / sum : 0.f;
  for (int e = threadIdx.x * 4; e < p.kv_rank; e += kMergeThreads * 4) {
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
    for (int c = 0; c < count; ++c) {
      const float w = weight[c];
      const float4 v = *reinterpret_cast<const float4 *>(u.part_o + (size_t)slot(c) * p.kv_rank + e);
      acc.x = fmaf(w, v.x, acc.x), acc.y = fmaf(w, v.y, acc.y), acc.z = fmaf(w, v.z, acc.z), acc.w = fmaf(w, v.w, acc.w);
    }
    *reinterpret_cast<uint2 *>(out + e) = make_uint2(pack_bf16x2(acc.x * inv, acc.y * inv), pack_bf16x2(acc.z * inv, acc.w * inv));
  }
}

int sm_count() {
  static int counts[64] = {0};
  int dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return 0;
  if (!counts[dev]) cudaDeviceGetAttribute(&counts[dev], cudaDevAttrMultiProcessorCount, dev);
  return counts[dev];
}

constexpr int kSmemLimit = 227 * 1024 - 1024;  // beside the kernel's static shared memory

// Chunks and ring sizes of a row; false when the sizes do not fit.
template <int kN>
bool layout(UmmaAttend &u) {
  u.chunks = (u.a.kv_rank + u.a.rot_dim + 63) / 64;
  u.pairs = (u.a.kv_rank + 127) / 128;
  u.singles = u.chunks > 2 * u.pairs ? u.chunks - 2 * u.pairs : 0;
  if (u.pairs > 4 || u.singles > 1) return false;
  // every pair of a tile has to be in place before the first is freed; what is left is read-ahead
  u.single_slots = u.singles;
  u.pair_slots = u.pairs;
  u.p_slots = 1;
  if (Smem<kN>::bytes(u, kMaxRows) > kSmemLimit) return false;
  while (u.pair_slots < kMaxSlots) {
    ++u.pair_slots;
    if (Smem<kN>::bytes(u, kMaxRows) > kSmemLimit) {
      --u.pair_slots;
      break;
    }
  }
  if (u.singles) {
    ++u.single_slots;
    if (Smem<kN>::bytes(u, kMaxRows) > kSmemLimit) --u.single_slots;
  }
  if (u.pair_slots >= 2 * u.pairs && u.single_slots >= 2 * u.singles) {
    UmmaAttend two = u;
    two.p_slots = 2;
    while (Smem<kN>::bytes(two, kMaxRows) > kSmemLimit && two.pair_slots > 2 * u.pairs) --two.pair_slots;
    if (Smem<kN>::bytes(two, kMaxRows) <= kSmemLimit) u = two;
  }
  return true;
}

template <int kN, int kH>
int run(const AttendParams &p, void *workspace, cudaStream_t st) {
  auto *kernel = latent_umma_kernel<kN, kH>;
  static std::mutex mu;
  static bool opted[64] = {false};
  int dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return AXB200_DEVICE_ERROR;
  {
    std::lock_guard<std::mutex> lock(mu);
    if (!opted[dev]) {
      if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, kSmemLimit) != cudaSuccess)
        return AXB200_DEVICE_ERROR;
      opted[dev] = true;
    }
  }
  // a row's elements, the heads and the tokens of a page, the pages: a box ends with its row, zero-filled beyond
  CUtensorMap map;
  const cuuint64_t dims[4] = {(cuuint64_t)p.row_elems, (cuuint64_t)p.kv_heads, (cuuint64_t)p.page_tokens,
                              (cuuint64_t)p.num_pages};
  const cuuint64_t strides[3] = {(cuuint64_t)p.page_tokens * p.row_elems * 2, (cuuint64_t)p.row_elems * 2,
                                 (cuuint64_t)p.page_elems * 2};
  const cuuint32_t box[4] = {64, 1, 64, 1}, es[4] = {1, 1, 1, 1};
  if (tensor_map_encoder()(&map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 4, const_cast<void *>(p.pages), dims, strides, box, es,
                           CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                           CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) != CUDA_SUCCESS)
    return AXB200_INTERNAL_ERROR;
  const int sms = sm_count();
  if (sms <= 0) return AXB200_DEVICE_ERROR;
  for (int r0 = 0; r0 < p.rows; r0 += kMaxRows) {
    UmmaAttend u{};
    u.a = p;
    AttendParams &a = u.a;
    a.rows = p.rows - r0 < kMaxRows ? p.rows - r0 : kMaxRows;
    a.q_lat = static_cast<const __nv_bfloat16 *>(p.q_lat) + (size_t)r0 * p.heads * p.kv_rank;
    if (p.q) a.q = static_cast<const __nv_bfloat16 *>(p.q) + (size_t)r0 * p.q_ld;
    a.out = static_cast<__nv_bfloat16 *>(p.out) + (size_t)r0 * p.heads * p.kv_rank;
    a.row_seq = p.row_seq + r0;
    a.row_pos = p.row_pos + r0;
    if (!layout<kN>(u)) return AXB200_INTERNAL_ERROR;
    u.part_tiles = (p.heads / p.kv_heads + kN - 1) / kN;
    u.head_tiles = p.kv_heads * u.part_tiles;
    u.groups = sms / u.head_tiles > 0 ? sms / u.head_tiles : 1;
    const int ctas = u.groups * u.head_tiles;
    u.part_ml = static_cast<float2 *>(workspace);
    u.part_o = reinterpret_cast<float *>(u.part_ml + 2 * kMaxCtas * kN);
    int rc = launch_dependent(kernel, dim3(ctas), dim3(kThreads), (size_t)Smem<kN>::bytes(u, a.rows), st, map, u);
    if (rc == AXB200_OK)
      rc = launch_dependent(latent_merge_kernel<kN>, dim3(a.rows, a.heads), dim3(kMergeThreads), 0, st, u);
    if (rc != AXB200_OK) return rc;
  }
  return AXB200_OK;
}

int heads_per_tile(int heads) { return heads <= 16 ? 16 : 32; }

}  // namespace

size_t latent_umma_workspace_bytes(int part_heads, int kv_rank, int rot_dim) {
  return (size_t)2 * kMaxCtas * heads_per_tile(part_heads) * (sizeof(float2) + (size_t)kv_rank * sizeof(float));
}

bool latent_umma_supported(const AttendParams &p) {
  const uintptr_t bits = reinterpret_cast<uintptr_t>(p.q_lat) | reinterpret_cast<uintptr_t>(p.q) | reinterpret_cast<uintptr_t>(p.out) |
                         reinterpret_cast<uintptr_t>(p.pages);
  const int n = heads_per_tile(p.heads / p.kv_heads), sms = sm_count();
  UmmaAttend u{};
  u.a = p;
  return p.kv_rank % 8 == 0 && p.rot_dim % 8 == 0 && p.row_elems % 8 == 0 && p.page_elems % 8 == 0 && (p.rot_dim == 0 || (p.dim % 8 == 0 && p.q_ld % 8 == 0)) &&
         (bits & 15u) == 0 && p.page_tokens % 64 == 0 && p.kv_heads * ((p.heads / p.kv_heads + n - 1) / n) <= kMaxCtas && sms > 0 && sms <= kMaxCtas && tensor_map_encoder() &&
         (p.max_len / kKeys + 1) * (int64_t)kMaxRows < 0x7fffffff &&
         (n == 16 ? layout<16>(u) : layout<32>(u));
}

int latent_umma(const AttendParams &p, void *workspace, cudaStream_t st) {
  const int part_heads = p.heads / p.kv_heads;
  if (heads_per_tile(part_heads) == 32) return run<32, 32>(p, workspace, st);
  return part_heads <= 4 ? run<16, 4>(p, workspace, st) : part_heads <= 8 ? run<16, 8>(p, workspace, st) : run<16, 16>(p, workspace, st);
}

}  // namespace axb
