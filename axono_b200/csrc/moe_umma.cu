// The expert products on the 5th-generation tensor cores, bf16 with fp32 accumulation.
//
// The weights are the M side: a CTA owns 128 rows of the gate matrix and the same 128 of the up matrix (or 256
// rows of the down matrix) of one expert, and a tile of kN routed rows as the N side - the MMA's M is fixed at
// 128, while the number of rows an expert gets ranges from one (decoding) to thousands (prompts), and N can
// follow it: 16 ... 256.  Both accumulators live in tensor memory (2 * kN columns), lane = output feature,
// column = routed row, so the gate and up values of an element meet in one thread and the activation needs no
// exchange.  The shared expert's tiles ride in the same launch (first in the grid: with few rows its CTAs alone
// could not fill the GPU), through tensor maps of their own.
//
// Warps 0-7 read the accumulators and store (every other 16 columns each four); warp 8 issues the MMAs, one lane of
// warp 9 the TMA loads, 64 elements of K per stage with 128-byte swizzle.  Sizes that are no multiple of the tile are
// zero-filled by TMA on the way in and masked on the way out.  Every wait is bounded.
#include <mutex>

#include "moe.cuh"

namespace axb {
namespace {

constexpr int kThreads = 320, kMmaWarp = 8, kLoadWarp = 9;
constexpr int kMTile = 128, kKTile = 64, kATile = kMTile * kKTile * 2;

template <int kN>
struct Shape {
  static constexpr int kBTile = kN * kKTile * 2;
  static constexpr int kStageBytes = 2 * kATile + kBTile;
  static constexpr int kStages = kN <= 32 ? 3 : kN == 64 ? 5 : kN == 128 ? 4 : 3;
  static constexpr int kCtasPerSm = kN <= 32 ? 2 : 1;
  static constexpr int kTmemCols = 2 * kN < 32 ? 32 : 2 * kN;
  static constexpr int kOffBar = kStages * kStageBytes;
  static constexpr int kSmem = kOffBar + 128;
};

struct UmmaParams {
  MoeProduct p[2];     // 0: routed, 1: shared (rows == 0: none)
  int shared_tiles;    // grid rows of the shared expert, before the routed ones
};

template <int kN, bool kGateUp>
__global__ void __launch_bounds__(kThreads, Shape<kN>::kCtasPerSm)
moe_umma_kernel(const __grid_constant__ CUtensorMap tmW, const __grid_constant__ CUtensorMap tmX,
                const __grid_constant__ CUtensorMap tmWs, const __grid_constant__ CUtensorMap tmXs,
                const __grid_constant__ UmmaParams up) {
  using S = Shape<kN>;
  extern __shared__ __align__(1024) uint8_t smem[];
  uint64_t *full = reinterpret_cast<uint64_t *>(smem + S::kOffBar), *empty = full + S::kStages, *done = empty + S::kStages;
  uint32_t *tmem_slot = reinterpret_cast<uint32_t *>(done + 1);
  volatile int *abort_flag = reinterpret_cast<volatile int *>(done + 2);
  if ((smem_u32(smem) & 1023u) != 0) {  // the swizzled tiles need it; nothing is written otherwise
    if (threadIdx.x == 0) atomicOr(&g_error_word, AXB200_ERR_WAIT_TIMEOUT);
    return;
  }
  const int warp = uniform_warp(), lane = threadIdx.x & 31;
  const bool shared = (int)blockIdx.y < up.shared_tiles;
  const MoeProduct &p = up.p[shared ? 1 : 0];
  constexpr int kMStep = kGateUp ? kMTile : 2 * kMTile;
  const int m0 = blockIdx.x * kMStep;
  grid_dependency_wait();
  grid_dependency_launch();
  int4 tile;  // expert, first row, rows
  if (m0 >= p.out || !moe_tile(p, shared ? blockIdx.y : blockIdx.y - up.shared_tiles, kN, tile)) return;
  const int steps = (p.in + kKTile - 1) / kKTile;

  if (threadIdx.x == 0) {
    for (int i = 0; i < 2 * S::kStages + 1; ++i) mbar_init(&full[i], 1);
    *abort_flag = 0;
    mbar_fence_init();
  }
  if (warp == kMmaWarp) {
    asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(tmem_slot)), "n"(S::kTmemCols)
                 : "memory");
    asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;

  if (warp == kLoadWarp) {
    if (lane == 0) {
      const CUtensorMap *mw = shared ? &tmWs : &tmW, *mx = shared ? &tmXs : &tmX;
      // gate rows of matrix 2e and up rows of matrix 2e + 1, or two neighbouring row blocks of matrix e
      const int mat0 = kGateUp ? 2 * tile.x : tile.x, mat1 = kGateUp ? mat0 + 1 : mat0, row1 = kGateUp ? m0 : m0 + kMTile;
      int k = 0;
      for (; k < steps; ++k) {
        const int s = k % S::kStages;
        if (k >= S::kStages && !mbar_wait_bounded(&empty[s], (k / S::kStages - 1) & 1, abort_flag, p.wait_ns)) break;
        uint8_t *dst = smem + s * S::kStageBytes;
        mbar_arrive_expect_tx(&full[s], S::kStageBytes);
        tma_load_3d(dst, mw, &full[s], k * kKTile, m0, mat0);
        tma_load_3d(dst + kATile, mw, &full[s], k * kKTile, row1, mat1);
        tma_load_2d(dst + 2 * kATile, mx, &full[s], k * kKTile, tile.y);
      }
      // after a wait that ran out: no copy may still be on its way when the CTA leaves
      if (*abort_flag)
        for (int j = max(0, k - S::kStages); j < k; ++j)
          for (int spin = 0; spin < (1 << 20) && !mbar_try_wait(&full[j % S::kStages], (j / S::kStages) & 1); ++spin) {
          }
    }
  } else if (warp == kMmaWarp) {
    const uint32_t lead = lane == 0;  // the warp walks, one lane issues
    {
      // fp32 accumulate, bf16 operands, both K-major, M = 128, N = kN
      constexpr uint32_t idesc = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(kN >> 3) << 17) | ((kMTile >> 4) << 24);
      const uint64_t base = smem_desc(smem_u32(smem), 16, 1024);
      bool ok = true;
      for (int k = 0; k < steps && ok; ++k) {
        const int s = k % S::kStages;
        ok = mbar_wait_warp(&full[s], (k / S::kStages) & 1, abort_flag, p.wait_ns);
        if (!ok) break;
        tc_fence_after();
        const uint64_t a0 = base + (uint64_t)(s * (S::kStageBytes >> 4)), a1 = a0 + (kATile >> 4), b = a0 + (2 * kATile >> 4);
#pragma unroll
        for (int ks = 0; ks < kKTile / 16; ++ks) umma_f16_lead(tmem, a0 + ks * 2, b + ks * 2, idesc, k > 0 || ks > 0, lead);
#pragma unroll
        for (int ks = 0; ks < kKTile / 16; ++ks) umma_f16_lead(tmem + kN, a1 + ks * 2, b + ks * 2, idesc, k > 0 || ks > 0, lead);
        umma_commit_lead(&empty[s], lead);
      }
      if (ok) umma_commit_lead(done, lead);
    }
  } else {
    mbar_wait_bounded(done, 0, abort_flag, p.wait_ns);
    named_bar_sync(1, 256);  // a wait that ran out raised the flag before this: all eight warps see the same
    tc_fence_after();
    const int rows = *abort_flag ? 0 : tile.z;
    // warps w and w + 4 share a quarter of the lanes (features) and take every other 16 columns (rows); the results
    // cross shared memory - every stage has been consumed - so that whole rows of features leave in 16-byte pieces
    const uint32_t base = tmem + ((uint32_t)((warp & 3) * 32) << 16);
    constexpr int kPitch = kMStep * 2, kPieces = kPitch / 16;
    uint8_t *mine = smem + ((warp & 3) * 32 + lane) * 2;
#pragma unroll 1
    for (int c = (warp >> 2) * 16; c < kN && c < rows; c += 32) {
      uint32_t a[16], b[16];
      tmem_ld16_async(base + c, a);
      tmem_ld16_async(base + kN + c, b);
      tmem_wait_ld();
#pragma unroll
      for (int i = 0; i < 16; ++i) {
        __nv_bfloat16 *row = reinterpret_cast<__nv_bfloat16 *>(mine + (c + i) * kPitch);
        const float va = __uint_as_float(a[i]), vb = __uint_as_float(b[i]);
        if (kGateUp) {
          row[0] = __float2bfloat16_rn(clamped_gate<false>(va, vb, p.act));
        } else {
          row[0] = __float2bfloat16_rn(va);
          row[kMTile] = __float2bfloat16_rn(vb);
        }
      }
    }
    named_bar_sync(1, 256);
    __nv_bfloat16 *y = static_cast<__nv_bfloat16 *>(p.y) + (size_t)tile.y * p.out + m0;
    for (int i = threadIdx.x; i < rows * kPieces; i += 256) {
      const int n = i / kPieces, f = i % kPieces * 8;
      if (m0 + f < p.out) *reinterpret_cast<uint4 *>(y + (size_t)n * p.out + f) = *reinterpret_cast<const uint4 *>(smem + n * kPitch + f * 2);
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == kMmaWarp)
    asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "n"(S::kTmemCols) : "memory");
}

bool al16(const void *p) { return (reinterpret_cast<uintptr_t>(p) & 15u) == 0; }

bool encode(CUtensorMap *map, const void *base, int rank, const cuuint64_t *dims, const cuuint64_t *strides, const cuuint32_t *box) {
  EncodeTiledFn fn = tensor_map_encoder();
  const cuuint32_t es[3] = {1, 1, 1};
  return fn && fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, rank, const_cast<void *>(base), dims, strides, box, es,
                  CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                  CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

bool maps_of(const MoeProduct &p, bool gate_up, int n_tile, CUtensorMap *w, CUtensorMap *x) {
  const cuuint64_t wd[3] = {(cuuint64_t)p.in, (cuuint64_t)p.out, (cuuint64_t)p.experts * (gate_up ? 2 : 1)};
  const cuuint64_t ws[2] = {(cuuint64_t)p.in * 2, (cuuint64_t)p.in * p.out * 2};
  const cuuint32_t wb[3] = {kKTile, kMTile, 1};
  const cuuint64_t xd[2] = {(cuuint64_t)p.in, (cuuint64_t)p.rows}, xs[1] = {(cuuint64_t)p.in * 2};
  const cuuint32_t xb[2] = {kKTile, (cuuint32_t)n_tile};
  return encode(w, p.w, 3, wd, ws, wb) && encode(x, p.x, 2, xd, xs, xb);
}

template <int kN, bool kGateUp>
int launch(const UmmaParams &up, const CUtensorMap (&maps)[4], dim3 grid, cudaStream_t st) {
  auto *kernel = moe_umma_kernel<kN, kGateUp>;
  static std::mutex mu;
  static bool opted[64] = {false};
  int dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return AXB200_DEVICE_ERROR;
  {
    std::lock_guard<std::mutex> lock(mu);
    if (!opted[dev]) {
      if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, Shape<kN>::kSmem) != cudaSuccess)
        return AXB200_DEVICE_ERROR;
      opted[dev] = true;
    }
  }
  return launch_dependent(kernel, grid, dim3(kThreads), Shape<kN>::kSmem, st, maps[0], maps[1], maps[2], maps[3], up);
}

template <bool kGateUp>
int launch_n(int n, const UmmaParams &up, const CUtensorMap (&maps)[4], dim3 grid, cudaStream_t st) {
  switch (n) {
    case 16: return launch<16, kGateUp>(up, maps, grid, st);
    case 32: return launch<32, kGateUp>(up, maps, grid, st);
    case 64: return launch<64, kGateUp>(up, maps, grid, st);
    case 128: return launch<128, kGateUp>(up, maps, grid, st);
    case 256: return launch<256, kGateUp>(up, maps, grid, st);
    default: return AXB200_INVALID_ARGUMENT;
  }
}

}  // namespace

bool moe_umma_takes(int width, int ff) { return width % 8 == 0 && ff % 8 == 0; }

// Rows per tile.  Few rows per expert: the time is the reading of the weights, and a tile that holds nearly every
// expert's rows reads them once at the least cost per column.  Many: the columns that the tiles of an expert with a
// typical number of rows (average plus two standard deviations) cover, those of 128 weighted with what they lose to
// operand traffic against 256.
int moe_umma_tile_rows(int64_t rows, int experts) {
  const int64_t avg = rows / experts;
  if (avg <= 36) return avg <= 7 ? 16 : avg <= 30 ? 32 : 64;
  int64_t sd = 1;
  while (sd * sd < avg) ++sd;
  const int64_t typical = avg + 2 * sd;
  return 10 * ((typical + 255) / 256) * 256 <= 12 * ((typical + 127) / 128) * 128 ? 256 : 128;
}

bool moe_umma_supported(const MoeProduct &p, bool gate_up) {
  return moe_umma_takes(p.in, p.out) && al16(p.x) && al16(p.w) && al16(p.y) && tensor_map_encoder();
}

int moe_umma(const MoeProduct &routed, const MoeProduct &shared, bool gate_up, cudaStream_t st) {
  UmmaParams up{};
  up.p[0] = routed;
  up.p[1] = shared;
  const int n = routed.tile_rows;
  up.p[1].tile_rows = n;
  const bool has_shared = shared.rows > 0;
  up.shared_tiles = has_shared ? (shared.rows + n - 1) / n : 0;
  CUtensorMap maps[4];
  if (!maps_of(routed, gate_up, n, &maps[0], &maps[1])) return AXB200_INTERNAL_ERROR;
  if (has_shared) {
    if (!maps_of(shared, gate_up, n, &maps[2], &maps[3])) return AXB200_INTERNAL_ERROR;
  } else {
    maps[2] = maps[0];
    maps[3] = maps[1];
  }
  const int step = gate_up ? kMTile : 2 * kMTile, out = has_shared && shared.out > routed.out ? shared.out : routed.out;
  const dim3 grid((out + step - 1) / step, up.shared_tiles + routed.max_tiles);
  if (grid.y > 65535) return AXB200_INVALID_ARGUMENT;
  return gate_up ? launch_n<true>(n, up, maps, grid, st) : launch_n<false>(n, up, maps, grid, st);
}

}  // namespace axb
