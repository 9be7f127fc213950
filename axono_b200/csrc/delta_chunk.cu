// The gated delta rule over portions of prompts, 64 tokens at a time on tensor cores (bf16 activations).
//
// Inside a chunk, with G_t the sum of the log decays up to token t and S the state before it, the rule unrolls to
//     X_t = v_t - e^{G_t} S^T k_t,      (I + A) U = diag(beta) X,   A_ts = beta_t e^{G_t - G_s} (k_t . k_s), s < t,
//     o_t = e^{G_t} S^T q_t + sum_{s <= t} P_ts u_s,                P_ts = e^{G_t - G_s} (q_t . k_s),
//     S'  = e^{G_64} S + sum_s e^{G_64 - G_s} k_s u_s^T.
// delta_chunk_prepare does what needs no state, all chunks at once: convolutions and silu, the products of queries and
// keys, T = (I + A)^-1 diag(beta) by blocked forward substitution in fp32, P, and the scale vectors.  delta_chunk_scan
// walks a sequence's chunks: a warp owns 16 value columns of a head's state and is independent of all others.
//
// Precision.  The outputs of the short convolutions are bf16, so they are exact tensor-core operands: unit norms and
// decays stay outside the products, as fp32 factors of rows.  Everything else that enters a product - state, X, U, T, P -
// is split into two bf16 parts and multiplied part by part (high.high + low.high + high.low), accumulated in fp32.
//
// The transposed products chain in registers: S^T (values x keys) is the accumulator of the update and operand A of the
// next chunk's products, X^T and U^T likewise, so the recurrence touches no shared memory.  Keys, T and P are operand B
// and come as ready-made, swizzled tiles by bulk copies, two or three chunks ahead.
#include <math.h>

#include <mutex>

#include "delta.cuh"

namespace axb {
namespace {

constexpr int kC = 64;                    // tokens of a chunk
constexpr int kSquare = kC * kC * 2;      // bytes of one bf16 part of T or P
constexpr int kVec = 4 * kSquare;         // where the scale vectors start in a head's tiles: ek, eq, eu [64], total
constexpr int kHeadTiles = kVec + 1024;   // T high, T low, P high, P low, vectors
constexpr int kValueTile = kC * 16 * 2;   // [64 tokens][16 value columns]
constexpr float kUnitEps = 1e-6f;

// Byte offset of 16-byte piece `piece` of row `row` in a tile of rows of `pieces` pieces, swizzled for ldmatrix.
__device__ __forceinline__ uint32_t tile_at(int row, int piece, int pieces) { return (uint32_t)((row * pieces + (piece ^ (row & 7))) << 4); }

__device__ __forceinline__ float bf_lo(uint32_t v) { return __uint_as_float(v << 16); }
__device__ __forceinline__ float bf_hi(uint32_t v) { return __uint_as_float(v & 0xffff0000u); }

// (a, b) as two packed bf16 pairs whose sum is nearly exact.
__device__ __forceinline__ void split(float a, float b, uint32_t &high, uint32_t &low) {
  high = pack_bf16x2(a, b);
  low = pack_bf16x2(a - bf_lo(high), b - bf_hi(high));
}

// Where the chunks of portion i (of those that start at row `first`) lie among all tiles.
__device__ __forceinline__ int first_chunk(const int4 &portion, int i, int first) { return (portion.y - first) / kC + i; }

// ---- chunks by themselves ----------------------------------------------------------------------------
constexpr int kPrepThreads = 256, kLd = kC + 4;  // fp32 matrices in shared memory have rows of kLd

// Convolution and silu of four channels from c on over tokens t0 .. t0 + count - 1 of a chunk; put(t, values).
template <typename Put>
__device__ __forceinline__ void conv_walk(const DeltaParams<__nv_bfloat16> &p, int64_t row0, int valid, int c, int t0, int count, Put put) {
  const int channels = p.channels();
  if (p.taps <= 4) {
    float w[4][4], past[3][4];
#pragma unroll
    for (int j = 0; j < 4; ++j) {
#pragma unroll
      for (int e = 0; e < 4; ++e) w[j][e] = 0.f;
      if (j < p.taps) load_vec<4>(p.conv + (size_t)(p.taps - 1 - j) * channels + c, w[j]);
    }
#pragma unroll
    for (int j = 0; j < 3; ++j) {
#pragma unroll
      for (int e = 0; e < 4; ++e) past[j][e] = 0.f;
      if (j + 1 < p.taps && t0 < valid) earlier_input<4>(p, row0 + t0, j + 1, c, past[j]);
    }
#pragma unroll 4
    for (int t = t0; t < t0 + count; ++t) {
      float now[4] = {}, y[4] = {};
      if (t < valid) {
        load_vec<4>(p.proj + (row0 + t) * p.ld + c, now);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          y[e] = silu(fmaf(past[2][e], w[3][e], fmaf(past[1][e], w[2][e], fmaf(past[0][e], w[1][e], now[e] * w[0][e]))));
          past[2][e] = past[1][e];
          past[1][e] = past[0][e];
          past[0][e] = now[e];
        }
      }
      put(t, y);
    }
    return;
  }
  for (int t = t0; t < t0 + count; ++t) {
    float y[4] = {};
    if (t < valid) {
      for (int j = 0; j < p.taps; ++j) {
        float in[4], w[4];
        earlier_input<4>(p, row0 + t, j, c, in);
        load_vec<4>(p.conv + (size_t)(p.taps - 1 - j) * channels + c, w);
#pragma unroll
        for (int e = 0; e < 4; ++e) y[e] = fmaf(in[e], w[e], y[e]);
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) y[e] = silu(y[e]);
    }
    put(t, y);
  }
}

// out[i0 .. i0 + rows)[j0 .. j0 + 4 per thread) = sign * a (rows x inner) . b (inner x cols), matrices of stride kLd; four
// neighbouring outputs per thread.
__device__ __forceinline__ void square_product(float *out, const float *a, const float *b, int rows, int inner, int cols, float sign,
                                               int tid, int threads) {
  const int quads = cols / 4;
  for (int i = tid; i < rows * quads; i += threads) {
    const int r = i / quads, c = i % quads * 4;
    float acc[4] = {};
    for (int k = 0; k < inner; ++k) {
      const float x = a[r * kLd + k];
      const float4 y = *reinterpret_cast<const float4 *>(b + k * kLd + c);
      acc[0] = fmaf(x, y.x, acc[0]), acc[1] = fmaf(x, y.y, acc[1]), acc[2] = fmaf(x, y.z, acc[2]), acc[3] = fmaf(x, y.w, acc[3]);
    }
    *reinterpret_cast<float4 *>(out + r * kLd + c) = make_float4(sign * acc[0], sign * acc[1], sign * acc[2], sign * acc[3]);
  }
}

template <int kDK>
struct PrepSmem {
  static constexpr int kTile = kC * kDK * 2, kMatrix = kC * kLd * 4;
  static constexpr int kOffKK = 2 * kTile, kOffQK = kOffKK + kMatrix, kOffA = kOffQK + kMatrix, kOffT = kOffA + kMatrix;
  static constexpr int kOffVec = kOffT + kMatrix, kBytes = kOffVec + 5 * kC * 4;
};

// Block z < kv_heads: one chunk of one query / key head, and T, P and the vectors of its group of value heads; the others:
// the values of one head.
template <int kDK>
__global__ void __launch_bounds__(kPrepThreads, 2)
delta_chunk_prepare_kernel(const DeltaParams<__nv_bfloat16> p, const int4 *portions, int first, uint8_t *keys, uint8_t *heads,
                           uint8_t *values) {
  using S = PrepSmem<kDK>;
  extern __shared__ __align__(128) uint8_t smem[];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  grid_dependency_wait();
  grid_dependency_launch();
  const int4 portion = portions[blockIdx.y];
  const int t_first = blockIdx.x * kC, valid = min(kC, portion.z - t_first);
  if (valid <= 0) return;
  if (portion.x < 0 || portion.x >= p.max_seqs) {
    if (tid == 0) atomicOr(&g_error_word, AXB200_ERR_CAPACITY);
    return;
  }
  const int64_t row0 = portion.y + t_first;
  const size_t chunk = first_chunk(portion, blockIdx.y, first) + blockIdx.x;
  const int qk_channels = 2 * p.kv_heads * p.dim;

  if ((int)blockIdx.z >= p.kv_heads) {
    // a quad of channels, a run of 8 tokens at a time
    const int h = blockIdx.z - p.kv_heads, blocks = (p.vdim + 15) / 16, quads = blocks * 4;
    uint8_t *dst = values + (chunk * p.heads + h) * (size_t)blocks * kValueTile;
    for (int i = tid; i < quads * (kC / 8); i += kPrepThreads) {
      const int quad = i % quads, c = quad * 4;
      auto put = [&](int t, const float (&y)[4]) {
        *reinterpret_cast<uint2 *>(dst + (c >> 4) * kValueTile + t * 32 + (c & 15) * 2) =
            make_uint2(pack_bf16x2(y[0], y[1]), pack_bf16x2(y[2], y[3]));
      };
      // past the last column the tile is zero
      conv_walk(p, row0, c < p.vdim ? valid : 0, c < p.vdim ? qk_channels + h * p.vdim + c : 0, i / quads * 8, 8, put);
    }
    return;
  }

  const int hk = blockIdx.z, group = p.heads / p.kv_heads;
  uint8_t *ck = smem, *cq = smem + S::kTile;
  float *kk = reinterpret_cast<float *>(smem + S::kOffKK), *qk = reinterpret_cast<float *>(smem + S::kOffQK);
  float *am = reinterpret_cast<float *>(smem + S::kOffA), *tm = reinterpret_cast<float *>(smem + S::kOffT);
  float *inv_k = reinterpret_cast<float *>(smem + S::kOffVec), *inv_q = inv_k + kC, *gsum = inv_q + kC, *beta = gsum + kC;
  constexpr int kPieces = kDK / 8;

  // convolutions: even warps the keys, odd warps the queries, 16 tokens each; a warp holds a whole row
  {
    const bool is_q = warp & 1;
    const int c = lane * 4, t0 = (warp >> 1) * 16;
    uint8_t *tile = is_q ? cq : ck;
    float *inv = is_q ? inv_q : inv_k;
    const float gain = is_q ? 1.0f / sqrtf((float)p.dim) : 1.f;
    auto put = [&](int t, const float (&y)[4]) {
      const uint2 packed = make_uint2(pack_bf16x2(y[0], y[1]), pack_bf16x2(y[2], y[3]));
      const float a = bf_lo(packed.x), b = bf_hi(packed.x), d = bf_lo(packed.y), e = bf_hi(packed.y);
      const float sq = warp_sum(a * a + b * b + d * d + e * e);  // of the rounded row: its unit vector is exact
      if (c < kDK) *reinterpret_cast<uint2 *>(tile + tile_at(t, c >> 3, kPieces) + (c & 4) * 2) = packed;
      if (lane == 0) inv[t] = gain / sqrtf(sq + kUnitEps);
    };
    const bool real = c < p.dim;
    conv_walk(p, row0, real ? valid : 0, real ? (is_q ? hk : p.kv_heads + hk) * p.dim + c : 0, t0, 16, put);
  }
  __syncthreads();
  {
    uint8_t *dst = keys + (chunk * p.kv_heads + hk) * (size_t)(2 * S::kTile);
    for (int i = tid * 16; i < 2 * S::kTile; i += kPrepThreads * 16)
      *reinterpret_cast<uint4 *>(dst + i) = *reinterpret_cast<const uint4 *>(smem + i);
  }
  // K.K^T (even warps) and Q.K^T (odd warps), 16 rows each
  {
    const uint32_t a_tile = smem_u32(warp & 1 ? cq : ck), b_tile = smem_u32(ck);
    float *out = warp & 1 ? qk : kk;
    const int m0 = (warp >> 1) * 16;
    float acc[8][4] = {};
#pragma unroll
    for (int k = 0; k < kDK / 16; ++k) {
      uint32_t a[4];
      ldmatrix_x4(a[0], a[1], a[2], a[3], a_tile + tile_at(m0 + (lane & 15), 2 * k + (lane >> 4), kPieces));
#pragma unroll
      for (int j = 0; j < 8; j += 2) {
        uint32_t b0, b1, b2, b3;
        ldmatrix_x4(b0, b1, b2, b3, b_tile + tile_at(8 * (j + (lane >> 4)) + (lane & 7), 2 * k + ((lane >> 3) & 1), kPieces));
        mma_16816_bf16(acc[j], a, b0, b1);
        mma_16816_bf16(acc[j + 1], a, b2, b3);
      }
    }
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const int r = m0 + (lane >> 2), c = j * 8 + (lane & 3) * 2;
      *reinterpret_cast<float2 *>(out + r * kLd + c) = make_float2(acc[j][0], acc[j][1]);
      *reinterpret_cast<float2 *>(out + (r + 8) * kLd + c) = make_float2(acc[j][2], acc[j][3]);
    }
  }

  for (int g = 0; g < group; ++g) {
    const int h = hk * group + g;
    uint8_t *dst = heads + (chunk * p.heads + h) * (size_t)kHeadTiles;
    __syncthreads();  // the products (first head); the last head's T has been stored
    if (warp == 0) {
      float lg[2], b[2];
#pragma unroll
      for (int i = 0; i < 2; ++i) {  // token 2 * lane + i
        const int t = 2 * lane + i;
        lg[i] = b[i] = 0.f;
        if (t < valid) {
          const __nv_bfloat16 *x = p.proj + (row0 + t) * p.ld;
          lg[i] = log_decay(ldf(x + p.a_at() + h), p.a_log[h], p.dt_bias[h]);
          b[i] = sigmoid(ldf(x + p.b_at() + h));
        }
      }
      float sum = lg[0] + lg[1];
#pragma unroll
      for (int d = 1; d < 32; d <<= 1) {
        const float o = __shfl_up_sync(0xffffffffu, sum, d);
        if (lane >= d) sum += o;
      }
      gsum[2 * lane] = sum - lg[1];
      gsum[2 * lane + 1] = sum;
      beta[2 * lane] = b[0];
      beta[2 * lane + 1] = b[1];
      const float last = __shfl_sync(0xffffffffu, sum, 31);
      float *vec = reinterpret_cast<float *>(dst + kVec);
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int t = 2 * lane + i;
        const float gt = i ? sum : sum - lg[1];
        vec[t] = expf(gt) * inv_k[t];
        vec[kC + t] = expf(gt) * inv_q[t];
        vec[2 * kC + t] = expf(last - gt) * inv_k[t];
      }
      if (lane == 0) vec[3 * kC] = expf(last);
    }
    __syncthreads();
    // A in shared memory, P straight to its tiles; a thread takes two neighbouring columns
    for (int i = tid; i < kC * kC / 2; i += kPrepThreads) {
      const int t = i / (kC / 2), s = i % (kC / 2) * 2;
      float a[2] = {}, pr[2] = {};
#pragma unroll
      for (int e = 0; e < 2; ++e)
        if (s + e <= t) {
          const float f = expf(gsum[t] - gsum[s + e]) * inv_k[s + e];
          pr[e] = f * inv_q[t] * qk[t * kLd + s + e];
          if (s + e < t) a[e] = beta[t] * f * inv_k[t] * kk[t * kLd + s + e];
        }
      *reinterpret_cast<float2 *>(am + t * kLd + s) = make_float2(a[0], a[1]);
      uint32_t high, low;
      split(pr[0], pr[1], high, low);
      const uint32_t at = tile_at(t, s >> 3, 8) + (s & 7) * 2;
      *reinterpret_cast<uint32_t *>(dst + 2 * kSquare + at) = high;
      *reinterpret_cast<uint32_t *>(dst + 3 * kSquare + at) = low;
    }
    __syncthreads();
    // (I + A)^-1: the four diagonal blocks of 16, a thread per column; then pairs of blocks
    if (tid < kC) {
      const int b0 = tid & ~15, j = tid & 15;
      float x[16];
#pragma unroll
      for (int i = 0; i < 16; ++i) {
        float acc = 0.f;
#pragma unroll
        for (int m = 0; m < i; ++m) acc = fmaf(am[(b0 + i) * kLd + b0 + m], x[m], acc);
        x[i] = i == j ? 1.f : i < j ? 0.f : -acc;
        tm[(b0 + i) * kLd + b0 + j] = x[i];
      }
    }
    __syncthreads();
    // lower left blocks: -T_low . (A . T_up); the inner product uses the (still unused) upper right of T
    {
      const int half = tid >> 7, o = half * 32;
      square_product(tm + o * kLd + o + 16, am + (o + 16) * kLd + o, tm + o * kLd + o, 16, 16, 16, 1.f, tid & 127, 128);
      __syncthreads();
      square_product(tm + (o + 16) * kLd + o, tm + (o + 16) * kLd + o + 16, tm + o * kLd + o + 16, 16, 16, 16, -1.f, tid & 127, 128);
      __syncthreads();
      if ((tid & 127) < 64) {  // clear the scratch: level two reads whole blocks
        const int r = (tid & 63) / 4, c = tid % 4 * 4;
        *reinterpret_cast<float4 *>(tm + (o + r) * kLd + o + 16 + c) = make_float4(0.f, 0.f, 0.f, 0.f);
      }
      __syncthreads();
      square_product(tm + 32, am + 32 * kLd, tm, 32, 32, 32, 1.f, tid, kPrepThreads);
      __syncthreads();
      square_product(tm + 32 * kLd, tm + 32 * kLd + 32, tm + 32, 32, 32, 32, -1.f, tid, kPrepThreads);
      __syncthreads();
    }
    for (int i = tid; i < kC * kC / 2; i += kPrepThreads) {
      const int t = i / (kC / 2), s = i % (kC / 2) * 2;
      const float a = s <= t ? tm[t * kLd + s] * beta[s] : 0.f, b = s + 1 <= t ? tm[t * kLd + s + 1] * beta[s + 1] : 0.f;
      uint32_t high, low;
      split(a, b, high, low);
      const uint32_t at = tile_at(t, s >> 3, 8) + (s & 7) * 2;
      *reinterpret_cast<uint32_t *>(dst + at) = high;
      *reinterpret_cast<uint32_t *>(dst + kSquare + at) = low;
    }
  }
}

// ---- the walk over a sequence's chunks ------------------------------------------------------------------
template <int kDK, int kWarps>
struct ScanSmem {
  static constexpr int kTile = kC * kDK * 2;
  static constexpr int kOffHead = 2 * kTile, kOffValues = kOffHead + kHeadTiles, kStage = kOffValues + kWarps * kValueTile;
  static constexpr int kStages = 3 * kStage + kWarps * kValueTile + 256 <= 227 * 1024 ? 3 : 2;
  static constexpr int kOffOut = kStages * kStage, kOffBar = kOffOut + kWarps * kValueTile, kBytes = kOffBar + 256;
};

__device__ __forceinline__ void bulk_load(void *dst, const void *src, uint32_t bytes, uint64_t *bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(smem_u32(dst)),
               "l"(__cvta_generic_to_global(src)), "r"(bytes), "r"(smem_u32(bar))
               : "memory");
}

__device__ __forceinline__ void stmatrix_x4_trans(uint32_t addr, uint32_t r0, uint32_t r1, uint32_t r2, uint32_t r3) {
  asm volatile("stmatrix.sync.aligned.m8n8.x4.trans.shared.b16 [%0], {%1,%2,%3,%4};" ::"r"(addr), "r"(r0), "r"(r1), "r"(r2), "r"(r3)
               : "memory");
}

// Operand A (16 x 16) in two parts from two neighbouring accumulator tiles.
__device__ __forceinline__ void split_operand(const float (&c0)[4], const float (&c1)[4], uint32_t (&high)[4], uint32_t (&low)[4]) {
  split(c0[0], c0[1], high[0], low[0]);
  split(c0[2], c0[3], high[1], low[1]);
  split(c1[0], c1[1], high[2], low[2]);
  split(c1[2], c1[3], high[3], low[3]);
}

// acc (16 x 64) += x (16 x 64, in two parts) . m^T for a lower triangular m (64 x 64) in two parts.
__device__ __forceinline__ void triangular_product(float (&acc)[8][4], const uint32_t (&high)[4][4], const uint32_t (&low)[4][4],
                                                   uint32_t m_high, uint32_t m_low, int lane) {
#pragma unroll
  for (int k = 0; k < 4; ++k) {
#pragma unroll
    for (int j = 2 * k; j < 8; j += 2) {
      const uint32_t at = tile_at(8 * (j + (lane >> 4)) + (lane & 7), 2 * k + ((lane >> 3) & 1), 8);
      uint32_t b[4], c[4];
      ldmatrix_x4(b[0], b[1], b[2], b[3], m_high + at);
      ldmatrix_x4(c[0], c[1], c[2], c[3], m_low + at);
      mma_16816_bf16(acc[j], high[k], b[0], b[1]);
      mma_16816_bf16(acc[j + 1], high[k], b[2], b[3]);
      mma_16816_bf16(acc[j], low[k], b[0], b[1]);
      mma_16816_bf16(acc[j + 1], low[k], b[2], b[3]);
      mma_16816_bf16(acc[j], high[k], c[0], c[1]);
      mma_16816_bf16(acc[j + 1], high[k], c[2], c[3]);
    }
  }
}

struct ScanParams {
  const int4 *portions;
  int first;
  const uint8_t *keys, *heads_tiles, *values;
  float *state;
  __nv_bfloat16 *out;  // (rows - first, heads, vdim)
  int heads, kv_heads, dim, vdim, max_seqs;
  unsigned long long wait_ns;
};

template <int kDK, int kWarps>
__global__ void __launch_bounds__((kWarps + 1) * 32, 1) delta_chunk_scan_kernel(const ScanParams p) {
  using L = ScanSmem<kDK, kWarps>;
  constexpr int kPieces = kDK / 8, kKeyTiles = kDK / 8;  // 8-wide tiles of S^T
  extern __shared__ __align__(128) uint8_t smem[];
  uint64_t *full = reinterpret_cast<uint64_t *>(smem + L::kOffBar), *empty = full + L::kStages;
  volatile int *abort_flag = reinterpret_cast<volatile int *>(empty + L::kStages);
  const int warp = __shfl_sync(0xffffffffu, (int)(threadIdx.x >> 5), 0), lane = threadIdx.x & 31;
  const int h = blockIdx.y, hk = h / (p.heads / p.kv_heads), blocks = (p.vdim + 15) / 16, block0 = blockIdx.z * kWarps;
  const int warps = min(kWarps, blocks - block0);  // with columns of their own
  if (threadIdx.x == 0) {
    for (int i = 0; i < L::kStages; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&empty[i], warps);
    }
    *abort_flag = 0;
    mbar_fence_init();
  }
  __syncthreads();
  grid_dependency_wait();
  grid_dependency_launch();
  const int4 portion = p.portions[blockIdx.x];
  if (portion.x < 0 || portion.x >= p.max_seqs) {
    if (threadIdx.x == 0) atomicOr(&g_error_word, AXB200_ERR_CAPACITY);
    return;
  }
  const int chunks = (portion.z + kC - 1) / kC;
  const size_t chunk0 = first_chunk(portion, blockIdx.x, p.first);

  if (warp == kWarps) {
    if (lane == 0) {
      bool ok = true;
      int n = 0;
      for (; n < chunks; ++n) {
        const int s = n % L::kStages;
        if (n >= L::kStages) ok = mbar_wait_bounded(&empty[s], (n / L::kStages - 1) & 1, abort_flag, p.wait_ns);
        if (!ok) break;
        const size_t chunk = chunk0 + n;
        uint8_t *dst = smem + s * L::kStage;
        mbar_arrive_expect_tx(&full[s], 2 * L::kTile + kHeadTiles + warps * kValueTile);
        bulk_load(dst, p.keys + (chunk * p.kv_heads + hk) * (2 * L::kTile), 2 * L::kTile, &full[s]);
        bulk_load(dst + L::kOffHead, p.heads_tiles + (chunk * p.heads + h) * kHeadTiles, kHeadTiles, &full[s]);
        bulk_load(dst + L::kOffValues, p.values + ((chunk * p.heads + h) * blocks + block0) * kValueTile, warps * kValueTile, &full[s]);
      }
      if (*abort_flag) {  // no copy may still be on its way when the CTA leaves
        const unsigned long long t0 = global_timer_ns();
        for (int i = max(0, n - L::kStages); i < n; ++i)
          while (!mbar_try_wait(&full[i % L::kStages], (i / L::kStages) & 1) && global_timer_ns() - t0 < 100000000ull) {
          }
      }
    }
    return;
  }
  if (warp >= warps) return;

  // S^T: tile j holds keys 8j .. 8j + 7; rows lane / 4 and + 8 are value columns, (lane % 4) * 2 and + 1 the keys
  const int v0 = (block0 + warp) * 16, va = v0 + (lane >> 2), vb = va + 8, kc = (lane & 3) * 2;
  float *state = p.state + ((size_t)portion.x * p.heads + h) * p.dim * p.vdim;
  float st[kKeyTiles][4];
#pragma unroll
  for (int j = 0; j < kKeyTiles; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int k = 8 * j + kc + (e & 1), v = e < 2 ? va : vb;
      st[j][e] = portion.w > 0 && k < p.dim && v < p.vdim ? state[(size_t)k * p.vdim + v] : 0.f;
    }
  uint8_t *staged = smem + L::kOffOut + warp * kValueTile;

  for (int n = 0; n < chunks; ++n) {
    const int s = n % L::kStages;
    if (!__all_sync(0xffffffffu, mbar_wait_bounded(&full[s], (n / L::kStages) & 1, abort_flag, p.wait_ns))) return;
    const uint32_t base = smem_u32(smem + s * L::kStage), ck = base, cq = base + L::kTile, tiles = base + L::kOffHead;
    const float *vec = reinterpret_cast<const float *>(smem + s * L::kStage + L::kOffHead + kVec);

    // S^T k and S^T q of all tokens
    float x[8][4] = {}, o[8][4] = {};
#pragma unroll
    for (int k = 0; k < kDK / 16; ++k) {
      uint32_t high[4], low[4];
      split_operand(st[2 * k], st[2 * k + 1], high, low);
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        float(&acc)[8][4] = half ? o : x;
        const uint32_t tile = half ? cq : ck;
        uint32_t b[4][4];
#pragma unroll
        for (int j = 0; j < 4; ++j)
          ldmatrix_x4(b[j][0], b[j][1], b[j][2], b[j][3],
                      tile + tile_at(8 * (2 * j + (lane >> 4)) + (lane & 7), 2 * k + ((lane >> 3) & 1), kPieces));
#pragma unroll
        for (int j = 0; j < 8; ++j) mma_16816_bf16(acc[j], high, b[j >> 1][(j & 1) * 2], b[j >> 1][(j & 1) * 2 + 1]);
#pragma unroll
        for (int j = 0; j < 8; ++j) mma_16816_bf16(acc[j], low, b[j >> 1][(j & 1) * 2], b[j >> 1][(j & 1) * 2 + 1]);
      }
    }
    // X^T = v^T - e^G S^T k
#pragma unroll
    for (int j = 0; j < 8; j += 2) {
      uint32_t v[4];
      ldmatrix_x4_trans(v[0], v[1], v[2], v[3], base + L::kOffValues + warp * kValueTile + (8 * (j + (lane >> 4)) + (lane & 7)) * 32 +
                                                    ((lane >> 3) & 1) * 16);
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const float2 e = *reinterpret_cast<const float2 *>(vec + 8 * (j + i) + kc);
        x[j + i][0] = fmaf(-e.x, x[j + i][0], bf_lo(v[2 * i]));
        x[j + i][1] = fmaf(-e.y, x[j + i][1], bf_hi(v[2 * i]));
        x[j + i][2] = fmaf(-e.x, x[j + i][2], bf_lo(v[2 * i + 1]));
        x[j + i][3] = fmaf(-e.y, x[j + i][3], bf_hi(v[2 * i + 1]));
      }
    }
    uint32_t high[4][4], low[4][4];
#pragma unroll
    for (int k = 0; k < 4; ++k) split_operand(x[2 * k], x[2 * k + 1], high[k], low[k]);
    float u[8][4] = {};
    triangular_product(u, high, low, tiles, tiles + kSquare, lane);
    // S'^T = e^G_64 S^T + (e^{G_64 - G} u)^T k
    const float total = vec[3 * kC];
#pragma unroll
    for (int j = 0; j < kKeyTiles; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) st[j][e] *= total;
#pragma unroll
    for (int k = 0; k < 4; ++k) {
      float w[2][4];
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const float2 e = *reinterpret_cast<const float2 *>(vec + 2 * kC + 8 * (2 * k + i) + kc);
        w[i][0] = e.x * u[2 * k + i][0], w[i][1] = e.y * u[2 * k + i][1];
        w[i][2] = e.x * u[2 * k + i][2], w[i][3] = e.y * u[2 * k + i][3];
      }
      split_operand(w[0], w[1], high[k], low[k]);
#pragma unroll
      for (int j = 0; j < kKeyTiles; j += 2) {
        uint32_t b[4];
        ldmatrix_x4_trans(b[0], b[1], b[2], b[3], ck + tile_at(16 * k + 8 * ((lane >> 3) & 1) + (lane & 7), j + (lane >> 4), kPieces));
        mma_16816_bf16(st[j], high[k], b[0], b[1]);
        mma_16816_bf16(st[j + 1], high[k], b[2], b[3]);
        mma_16816_bf16(st[j], low[k], b[0], b[1]);
        mma_16816_bf16(st[j + 1], low[k], b[2], b[3]);
      }
    }
    // o^T = e^G S^T q + u^T P^T
#pragma unroll
    for (int j = 0; j < 8; ++j) {
      const float2 e = *reinterpret_cast<const float2 *>(vec + kC + 8 * j + kc);
      o[j][0] *= e.x, o[j][1] *= e.y, o[j][2] *= e.x, o[j][3] *= e.y;
    }
#pragma unroll
    for (int k = 0; k < 4; ++k) split_operand(u[2 * k], u[2 * k + 1], high[k], low[k]);
    triangular_product(o, high, low, tiles + 2 * kSquare, tiles + 3 * kSquare, lane);
    __syncwarp();
    if (lane == 0) mbar_arrive(&empty[s]);
    // through shared memory into rows of 16 columns
#pragma unroll
    for (int j = 0; j < 8; j += 2)
      stmatrix_x4_trans(smem_u32(staged) + (8 * (j + (lane >> 4)) + (lane & 7)) * 32 + ((lane >> 3) & 1) * 16, pack_bf16x2(o[j][0], o[j][1]),
                        pack_bf16x2(o[j][2], o[j][3]), pack_bf16x2(o[j + 1][0], o[j + 1][1]), pack_bf16x2(o[j + 1][2], o[j + 1][3]));
    __syncwarp();
    const int valid = min(kC, portion.z - n * kC);
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int t = (i * 32 + lane) >> 1, c = v0 + (lane & 1) * 8;
      if (t < valid && c < p.vdim)
        *reinterpret_cast<uint4 *>(p.out + ((int64_t)(portion.y - p.first + n * kC + t) * p.heads + h) * p.vdim + c) =
            *reinterpret_cast<const uint4 *>(staged + t * 32 + (lane & 1) * 16);
    }
    __syncwarp();
  }
#pragma unroll
  for (int j = 0; j < kKeyTiles; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int k = 8 * j + kc + (e & 1), v = e < 2 ? va : vb;
      if (k < p.dim && v < p.vdim) state[(size_t)k * p.vdim + v] = st[j][e];
    }
}

bool al16(const void *p) { return (reinterpret_cast<uintptr_t>(p) & 15u) == 0; }

template <auto kKernel>
int opt_in(int bytes) {
  static std::mutex mu;
  static bool done[64] = {false};
  int dev = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return AXB200_DEVICE_ERROR;
  std::lock_guard<std::mutex> lock(mu);
  if (!done[dev] && cudaFuncSetAttribute(kKernel, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes) != cudaSuccess)
    return AXB200_DEVICE_ERROR;
  done[dev] = true;
  return AXB200_OK;
}

template <int kDK, int kWarps>
int run_scan(const ScanParams &p, int count, cudaStream_t st) {
  using L = ScanSmem<kDK, kWarps>;
  if (int rc = opt_in<delta_chunk_scan_kernel<kDK, kWarps>>(L::kBytes)) return rc;
  const int blocks = (p.vdim + 15) / 16;
  return launch_dependent(delta_chunk_scan_kernel<kDK, kWarps>, dim3(count, p.heads, (blocks + kWarps - 1) / kWarps),
                          dim3((kWarps + 1) * 32), (size_t)L::kBytes, st, p);
}

template <int kDK>
int run(const DeltaParams<__nv_bfloat16> &d, const ScanParams &s, int count, int longest, uint8_t *keys, uint8_t *heads, uint8_t *values,
        cudaStream_t st) {
  using P = PrepSmem<kDK>;
  if (int rc = opt_in<delta_chunk_prepare_kernel<kDK>>(P::kBytes)) return rc;
  const dim3 grid((longest + kC - 1) / kC, count, d.kv_heads + d.heads);
  if (int rc = launch_dependent(delta_chunk_prepare_kernel<kDK>, grid, dim3(kPrepThreads), (size_t)P::kBytes, st, d, s.portions, s.first, keys,
                                heads, values))
    return rc;
  // as few warps in a CTA as give every SM at most one
  int dev = 0, sms = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess)
    return AXB200_DEVICE_ERROR;
  const int64_t warps = (int64_t)count * d.heads * ((d.vdim + 15) / 16);
  if (warps <= sms) return run_scan<kDK, 1>(s, count, st);
  if (warps <= 2 * sms) return run_scan<kDK, 2>(s, count, st);
  return run_scan<kDK, 4>(s, count, st);
}

int padded_dim(int dim) { return dim <= 64 ? 64 : 128; }
int64_t chunk_slots(int64_t rows, int count) { return rows / kC + count; }

}  // namespace
}  // namespace axb

extern "C" {

int axb200_delta_chunks_supported(int dim, int vdim, int dtype) {
  return dtype == AXB200_BFLOAT16 && dim > 0 && dim <= 128 && dim % 4 == 0 && vdim > 0 && vdim <= 4096 && vdim % 8 == 0;
}

size_t axb200_delta_chunks_workspace_bytes(int64_t rows, int count, int heads, int kv_heads, int dim, int vdim) {
  if (rows <= 0 || count <= 0) return 0;
  return (size_t)axb::chunk_slots(rows, count) *
         ((size_t)kv_heads * 2 * axb::kC * axb::padded_dim(dim) * 2 +
          (size_t)heads * (axb::kHeadTiles + (size_t)((vdim + 15) / 16) * axb::kValueTile));
}

int axb200_delta_chunks(const void *proj, int64_t ld, const int32_t *row_seq, const int32_t *row_pos, const int32_t *row_back,
                        int first, int rows, const float *conv, const float *a_log, const float *dt_bias, void *ring, float *state,
                        const int32_t *portions, int count, int longest, void *out, int heads, int kv_heads, int dim, int vdim,
                        int taps, int max_seqs, int dtype, void *workspace, size_t workspace_bytes, void *stream) {
  if (!axb200_delta_chunks_supported(dim, vdim, dtype)) return AXB200_UNSUPPORTED_TYPE;
  if (!proj || !row_seq || !row_pos || !row_back || !conv || !a_log || !dt_bias || !ring || !state || !portions || !out || !workspace)
    return AXB200_INVALID_PTR;
  if (first < 0 || first > rows || count < 0 || count > 65535 || longest < 0 || heads <= 0 || kv_heads <= 0 || heads % kv_heads != 0 ||
      heads + kv_heads > 65535 || taps <= 0 || max_seqs <= 0)
    return AXB200_INVALID_ARGUMENT;
  if (ld < (int64_t)2 * kv_heads * dim + (int64_t)heads * (2 * vdim + 2)) return AXB200_SHAPE_MISMATCH;
  if (ld % 4 || !axb::al16(proj) || !axb::al16(conv) || !axb::al16(ring) || !axb::al16(portions) || !axb::al16(out) ||
      (reinterpret_cast<uintptr_t>(workspace) & 127u))
    return AXB200_UNSUPPORTED_TYPE;
  if (count == 0 || first == rows) return AXB200_OK;
  if (workspace_bytes < axb200_delta_chunks_workspace_bytes(rows - first, count, heads, kv_heads, dim, vdim)) return AXB200_OUT_OF_MEMORY;
  const axb::DeltaParams<__nv_bfloat16> d{static_cast<const __nv_bfloat16 *>(proj), ld, row_seq, row_pos, row_back, rows, conv, a_log,
                                          dt_bias, nullptr, static_cast<__nv_bfloat16 *>(ring), state, heads, kv_heads, dim, vdim, taps,
                                          max_seqs, 0.f};
  const size_t slots = (size_t)axb::chunk_slots(rows - first, count);
  uint8_t *keys = static_cast<uint8_t *>(workspace);
  uint8_t *tiles = keys + slots * kv_heads * 2 * axb::kC * axb::padded_dim(dim) * 2;
  uint8_t *values = tiles + slots * heads * axb::kHeadTiles;
  const axb::ScanParams s{reinterpret_cast<const int4 *>(portions), first, keys, tiles, values, state, static_cast<__nv_bfloat16 *>(out),
                          heads, kv_heads, dim, vdim, max_seqs, axb::wait_limit_ns()};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return axb::padded_dim(dim) == 64 ? axb::run<64>(d, s, count, longest, keys, tiles, values, st)
                                    : axb::run<128>(d, s, count, longest, keys, tiles, values, st);
}

}  // extern "C"
