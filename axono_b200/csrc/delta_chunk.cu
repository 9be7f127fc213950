// The gated delta rule over portions of prompts, 64 tokens at a time on tensor cores (bf16 activations).
//
// Inside a chunk, with G_t the sum of the log decays up to token t and S the state before it, the rule unrolls to
//     X_t = v_t - e^{G_t} S^T k_t,      (I + A) U = diag(beta) X,   A_ts = beta_t e^{G_t - G_s} (k_t . k_s), s < t,
//     o_t = e^{G_t} S^T q_t + sum_{s <= t} P_ts u_s,                P_ts = e^{G_t - G_s} (q_t . k_s),
//     S'  = e^{G_64} S + sum_s e^{G_64 - G_s} k_s u_s^T.
// Two kernels do what needs no state, all chunks at once: delta_chunk_conv the convolutions and silu, into tiles;
// delta_chunk_prepare the products of queries and keys, T = (I + A)^-1 diag(beta) by blocked forward substitution, P, and
// the scale vectors.  delta_chunk_scan walks a sequence's chunks: a warp owns 8 or 16 value columns of a head's state and
// is independent of all others.
//
// Precision.  The outputs of the short convolutions are bf16, so they are exact tensor-core operands: unit norms and
// decays stay outside the products, as fp32 factors of rows.  Everything else that enters a product - state, X, U, T, P -
// is split into two bf16 parts and multiplied part by part (high.high + low.high + high.low), accumulated in fp32.
//
// The products chain in registers: S (keys x values) is the accumulator of the update and, transposed in the register
// file (movmatrix), operand B of the next chunk's products; X and U likewise.  So the recurrence touches no shared memory.
// Keys, queries, T and P are operand A and come as ready-made, swizzled tiles by bulk copies, some chunks ahead.
// The walk is bound by the length of this chain, not by the tensor cores of a whole SM: 64 tokens take 250 warp-wide
// products of 16 x 8 x 16 at about ten cycles each, of which the 94 of the read-out (q S + P U) move to a second warp that
// gets S and U through shared memory.  Products of tcgen05 size would need 64 or more columns and four round trips
// through tensor and shared memory per chunk, which together take longer.
#include <math.h>

#include <mutex>

#include "delta.cuh"

namespace axb {
namespace {

constexpr int kC = 64;                    // tokens of a chunk
constexpr int kSquare = 10 * 512;         // bytes of one bf16 part of T or P: its ten lower 16 x 16 blocks
constexpr int kVec = 4 * kSquare;         // where the scale vectors start in a head's tiles: ek, eq, eu [64], total
constexpr int kHeadTiles = kVec + 1024;   // T high, T low, P high, P low, vectors
constexpr int kValueTile = kC * 8 * 2;    // [64 tokens][8 value columns]
constexpr int kPrepHeads = 4;             // heads whose gates a block holds at a time
constexpr float kUnitEps = 1e-6f;

// Byte offset of 16-byte piece `piece` of row `row` in a tile of rows of `pieces` pieces, swizzled for ldmatrix.
__device__ __forceinline__ uint32_t tile_at(int row, int piece, int pieces) { return (uint32_t)((row * pieces + (piece ^ (row & 7))) << 4); }

// Byte offset of 16-byte piece `piece` (0, 1) of row `row` of block (m, k), k <= m, in one part of T or P.
__device__ __forceinline__ uint32_t block_at(int m, int k, int row, int piece) {
  return (uint32_t)((m * (m + 1) / 2 + k) * 512 + row * 32 + ((piece ^ ((row >> 2) & 1)) << 4));
}

// A chunk of one query / key head: the tiles of k and q as the convolutions put them out, and 1 / norm of their rows (of q
// also / sqrt(dim)).
template <int kDK>
struct KeyTiles {
  static constexpr int kTile = kC * kDK * 2, kOffInv = 2 * kTile, kBytes = kOffInv + 2 * kC * 4;
};

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
constexpr int kPrepThreads = 256, kLd = kC + 8;  // fp32 matrices in shared memory have rows of kLd

// silu of what a convolution puts out (an activation that is rounded to bf16)
__device__ __forceinline__ float fast_silu(float z) { return __fdividef(z, 1.0f + __expf(-z)); }

// The inputs of four channels at token t of a portion: a row of this step, the ring, or zero before the sequence's start.
__device__ __forceinline__ void portion_input(const DeltaParams<__nv_bfloat16> &p, const int4 &portion, int t, int c, float (&v)[4]) {
  if (t >= 0) {
    load_vec<4>(p.proj + (int64_t)(portion.y + t) * p.ld + c, v);
  } else if (portion.w + t >= 0) {
    load_vec<4>(p.ring + ((size_t)portion.x * p.taps + (portion.w + t) % p.taps) * p.channels() + c, v);
  } else {
#pragma unroll
    for (int e = 0; e < 4; ++e) v[e] = 0.f;
  }
}

// Convolution and silu of four channels from c on over kCount tokens from t0 on of a portion, of which `valid` are real;
// put(i, values).
template <int kCount, typename Put>
__device__ __forceinline__ void conv_walk(const DeltaParams<__nv_bfloat16> &p, const int4 &portion, int t0, int valid, int c, Put put) {
  const int channels = p.channels();
  if (p.taps <= 4) {
    uint2 raw[kCount];  // all on their way at once
#pragma unroll
    for (int i = 0; i < kCount; ++i) {
      raw[i] = make_uint2(0, 0);
      if (i < valid) raw[i] = *reinterpret_cast<const uint2 *>(p.proj + (int64_t)(portion.y + t0 + i) * p.ld + c);
    }
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
      if (j + 1 < p.taps && valid > 0) portion_input(p, portion, t0 - j - 1, c, past[j]);
    }
#pragma unroll
    for (int i = 0; i < kCount; ++i) {
      const float now[4] = {bf_lo(raw[i].x), bf_hi(raw[i].x), bf_lo(raw[i].y), bf_hi(raw[i].y)};
      float y[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        y[e] = fmaf(past[2][e], w[3][e], fmaf(past[1][e], w[2][e], fmaf(past[0][e], w[1][e], now[e] * w[0][e])));
        y[e] = i < valid ? fast_silu(y[e]) : 0.f;
        past[2][e] = past[1][e];
        past[1][e] = past[0][e];
        past[0][e] = now[e];
      }
      put(i, y);
    }
    return;
  }
#pragma unroll
  for (int i = 0; i < kCount; ++i) {
    float y[4] = {};
    if (i < valid) {
      for (int j = 0; j < p.taps; ++j) {
        float in[4], w[4];
        portion_input(p, portion, t0 + i - j, c, in);
        load_vec<4>(p.conv + (size_t)(p.taps - 1 - j) * channels + c, w);
#pragma unroll
        for (int e = 0; e < 4; ++e) y[e] = fmaf(in[e], w[e], y[e]);
      }
#pragma unroll
      for (int e = 0; e < 4; ++e) y[e] = fast_silu(y[e]);
    }
    put(i, y);
  }
}

// A warp takes 16 tokens of a query or key head (all its channels: the unit norm stays inside the warp) or of 128 value
// channels; the four warps of a block the four runs of a chunk.
template <int kDK>
__global__ void __launch_bounds__(128)
delta_chunk_conv_kernel(const DeltaParams<__nv_bfloat16> p, const int4 *portions, int first, uint8_t *keys, uint8_t *values) {
  using K = KeyTiles<kDK>;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, unit = blockIdx.z;
  grid_dependency_wait();
  grid_dependency_launch();
  const int4 portion = portions[blockIdx.y];
  const int c_first = blockIdx.x * kC;
  if (c_first >= portion.z) return;
  if (portion.x < 0 || portion.x >= p.max_seqs) {
    if (threadIdx.x == 0) atomicOr(&g_error_word, AXB200_ERR_CAPACITY);
    return;
  }
  const size_t chunk = first_chunk(portion, blockIdx.y, first) + blockIdx.x;
  const int run = warp * 16, t0 = c_first + run, valid = portion.z - t0;
  if (unit >= 2 * p.kv_heads) {
    const int c = (unit - 2 * p.kv_heads) * 128 + lane * 4;
    if (c >= p.heads * p.vdim) return;
    uint8_t *dst = values + (chunk * (p.heads * p.vdim / 8) + c / 8) * (size_t)kValueTile + (c & 7) * 2;
    conv_walk<16>(p, portion, t0, valid, 2 * p.kv_heads * p.dim + c, [&](int i, const float (&y)[4]) {
      *reinterpret_cast<uint2 *>(dst + (run + i) * 16) = make_uint2(pack_bf16x2(y[0], y[1]), pack_bf16x2(y[2], y[3]));
    });
    return;
  }
  const bool is_k = unit >= p.kv_heads;
  const int hk = is_k ? unit - p.kv_heads : unit, c = lane * 4;
  uint8_t *tiles = keys + (chunk * p.kv_heads + hk) * (size_t)K::kBytes, *tile = tiles + (is_k ? 0 : K::kTile);
  const bool real = c < p.dim;
  float sq[16];  // of the rounded rows: their unit vectors are exact
  conv_walk<16>(p, portion, t0, real ? valid : 0, real ? unit * p.dim + c : 0, [&](int i, const float (&y)[4]) {
    const uint2 packed = make_uint2(pack_bf16x2(y[0], y[1]), pack_bf16x2(y[2], y[3]));
    const float a = bf_lo(packed.x), b = bf_hi(packed.x), d = bf_lo(packed.y), e = bf_hi(packed.y);
    sq[i] = a * a + b * b + d * d + e * e;
    if (c < kDK) *reinterpret_cast<uint2 *>(tile + tile_at(run + i, c >> 3, kDK / 8) + (c & 4) * 2) = packed;
  });
  // all sixteen sums over the warp by halving exchanges: lanes 2 i and 2 i + 1 end with row i's
#pragma unroll
  for (int n = 8, off = 16; n > 0; n >>= 1, off >>= 1) {
    const bool upper = lane & off;
#pragma unroll
    for (int i = 0; i < n; ++i) {
      const float send = upper ? sq[i] : sq[i + n], keep = upper ? sq[i + n] : sq[i];
      sq[i] = keep + __shfl_xor_sync(0xffffffffu, send, off);
    }
  }
  sq[0] += __shfl_xor_sync(0xffffffffu, sq[0], 1);
  const float gain = is_k ? 1.f : 1.0f / sqrtf((float)p.dim);
  if ((lane & 1) == 0)
    reinterpret_cast<float *>(tiles + K::kOffInv)[(is_k ? 0 : kC) + run + (lane >> 1)] = gain / sqrtf(sq[0] + kUnitEps);
}

// One warp: out (16 x 8) = sign * a (16 x 16 n) . b (16 n x 8), fp32 matrices of stride kLd in shared memory, in bf16
// parts on the tensor core.
__device__ __forceinline__ void small_product(float *out, const float *a, const float *b, int n, float sign, int lane) {
  const int g = lane >> 2, q = (lane & 3) * 2;
  float acc[4] = {};
  for (int k = 0; k < n; ++k, a += 16, b += 16 * kLd) {
    uint32_t ah[4], al[4], bh[2], bl[2];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const float2 v = *reinterpret_cast<const float2 *>(a + (g + (i & 1) * 8) * kLd + q + (i >> 1) * 8);
      split(v.x, v.y, ah[i], al[i]);
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) split(b[(q + i * 8) * kLd + g], b[(q + i * 8 + 1) * kLd + g], bh[i], bl[i]);
    mma_16816_bf16(acc, ah, bh[0], bh[1]);
    mma_16816_bf16(acc, al, bh[0], bh[1]);
    mma_16816_bf16(acc, ah, bl[0], bl[1]);
  }
  *reinterpret_cast<float2 *>(out + g * kLd + q) = make_float2(sign * acc[0], sign * acc[1]);
  *reinterpret_cast<float2 *>(out + (g + 8) * kLd + q) = make_float2(sign * acc[2], sign * acc[3]);
}

template <int kDK>
struct PrepSmem {
  static constexpr int kMatrix = kC * kLd * 4;
  static constexpr int kOffKK = KeyTiles<kDK>::kBytes, kOffQK = kOffKK + kMatrix, kOffA = kOffQK + kMatrix;  // A: one per half
  static constexpr int kOffGates = kOffA + 2 * kMatrix, kOffBar = kOffGates + 2 * kPrepHeads * kC * 4, kBytes = kOffBar + 16;
};

// One chunk of one query / key head: T, P and the vectors of its group of value heads.
template <int kDK>
__global__ void __launch_bounds__(kPrepThreads, 2)
delta_chunk_prepare_kernel(const DeltaParams<__nv_bfloat16> p, const int4 *portions, int first, const uint8_t *keys, uint8_t *heads,
                           unsigned long long wait_ns) {
  using S = PrepSmem<kDK>;
  using K = KeyTiles<kDK>;
  extern __shared__ __align__(128) uint8_t smem[];
  uint64_t *bar = reinterpret_cast<uint64_t *>(smem + S::kOffBar);
  volatile int *abort_flag = reinterpret_cast<volatile int *>(bar + 1);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  if (tid == 0) {
    mbar_init(bar, 1);
    *abort_flag = 0;
    mbar_fence_init();
  }
  __syncthreads();
  grid_dependency_wait();
  grid_dependency_launch();
  const int4 portion = portions[blockIdx.y];
  const int t_first = blockIdx.x * kC, valid = min(kC, portion.z - t_first);
  if (valid <= 0 || portion.x < 0 || portion.x >= p.max_seqs) return;
  const int64_t row0 = portion.y + t_first;
  const size_t chunk = first_chunk(portion, blockIdx.y, first) + blockIdx.x;
  const int hk = blockIdx.z, group = p.heads / p.kv_heads;
  if (tid == 0) {
    mbar_arrive_expect_tx(bar, K::kBytes);
    bulk_load(smem, keys + (chunk * p.kv_heads + hk) * K::kBytes, K::kBytes, bar);
  }
  const uint8_t *ck = smem, *cq = smem + K::kTile;
  float *kk = reinterpret_cast<float *>(smem + S::kOffKK), *qk = reinterpret_cast<float *>(smem + S::kOffQK);
  const float *inv_k = reinterpret_cast<const float *>(smem + K::kOffInv), *inv_q = inv_k + kC;
  float *gates = reinterpret_cast<float *>(smem + S::kOffGates);
  constexpr int kPieces = kDK / 8;

  // decays, summed up (in the log2 domain), and steps of up to kPrepHeads heads: a warp per head, two tokens per lane
  auto gates_of = [&](int g0) {
    for (int g = g0 + warp; g < min(g0 + kPrepHeads, group); g += kPrepThreads / 32) {
      const int h = hk * group + g;
      float lg[2], b[2];
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int t = 2 * lane + i;
        lg[i] = b[i] = 0.f;
        if (t < valid) {
          const __nv_bfloat16 *x = p.proj + (row0 + t) * p.ld;
          lg[i] = log_decay(ldf(x + p.a_at() + h), p.a_log[h], p.dt_bias[h]) * 1.4426950408889634f;
          b[i] = sigmoid(ldf(x + p.b_at() + h));
        }
      }
      float sum = lg[0] + lg[1];
#pragma unroll
      for (int d = 1; d < 32; d <<= 1) {
        const float o = __shfl_up_sync(0xffffffffu, sum, d);
        if (lane >= d) sum += o;
      }
      float *dst = gates + (g - g0) * 2 * kC;
      *reinterpret_cast<float2 *>(dst + 2 * lane) = make_float2(sum - lg[1], sum);
      *reinterpret_cast<float2 *>(dst + kC + 2 * lane) = make_float2(b[0], b[1]);
    }
  };
  gates_of(0);
  if (!mbar_wait_bounded(bar, 0, abort_flag, wait_ns)) {  // no copy may still be on its way when the CTA leaves
    const unsigned long long t0 = global_timer_ns();
    while (!mbar_try_wait(bar, 0) && global_timer_ns() - t0 < 100000000ull) {
    }
    return;
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

  // T and P: each half of the block (four warps) takes every second head
  __syncthreads();
  const int half = warp >> 2, ht = tid & 127, hw = warp & 3;
  auto half_sync = [&] { named_bar_sync(1 + half, 128); };
  float *am = reinterpret_cast<float *>(smem + S::kOffA) + half * kC * kLd;  // A, and in its place (I + A)^-1
  for (int g0 = 0; g0 < group; g0 += 2) {
    const int g = g0 + half, h = hk * group + g;
    if (g0 > 0 && g0 % kPrepHeads == 0) {
      __syncthreads();
      gates_of(g0);
      __syncthreads();
    }
    if (g >= group) continue;  // the other half has the last head
    uint8_t *dst = heads + (chunk * p.heads + h) * (size_t)kHeadTiles;
    const float *gsum = gates + g % kPrepHeads * 2 * kC, *beta = gsum + kC;
    if (ht < kC) {
      float *vec = reinterpret_cast<float *>(dst + kVec);
      const float last = gsum[kC - 1], e = fast_exp2(gsum[ht]);
      vec[ht] = e * inv_k[ht];
      vec[kC + ht] = e * inv_q[ht];
      vec[2 * kC + ht] = fast_exp2(last - gsum[ht]) * inv_k[ht];
      if (ht == 0) vec[3 * kC] = fast_exp2(last);
    }
    half_sync();  // the last head's T has been stored
    // the lower blocks of A in shared memory, of P straight to their place; a thread takes two neighbouring columns
#pragma unroll
    for (int blk = 0; blk < 10; ++blk) {
      const int m = blk < 1 ? 0 : blk < 3 ? 1 : blk < 6 ? 2 : 3, k = blk - m * (m + 1) / 2;
      const int r = ht >> 3, c = (ht & 7) * 2, t = m * 16 + r, s = k * 16 + c;
      const float2 x = *reinterpret_cast<const float2 *>(kk + t * kLd + s), y = *reinterpret_cast<const float2 *>(qk + t * kLd + s);
      const float2 gs = *reinterpret_cast<const float2 *>(gsum + s), ik = *reinterpret_cast<const float2 *>(inv_k + s);
      const float gt = gsum[t], f0 = s <= t ? fast_exp2(gt - gs.x) * ik.x : 0.f, f1 = s < t ? fast_exp2(gt - gs.y) * ik.y : 0.f;
      const float at = beta[t] * inv_k[t], pt = inv_q[t];
      *reinterpret_cast<float2 *>(am + t * kLd + s) = make_float2(at * f0 * x.x, at * f1 * x.y);  // the diagonal is not read
      uint32_t high, low;
      split(pt * f0 * y.x, pt * f1 * y.y, high, low);
      const uint32_t off = block_at(m, k, r, c >> 3) + (c & 7) * 2;
      *reinterpret_cast<uint32_t *>(dst + 2 * kSquare + off) = high;
      *reinterpret_cast<uint32_t *>(dst + 3 * kSquare + off) = low;
    }
    half_sync();
    // the four diagonal blocks of 16 by forward substitution, a thread per column
    float inv[16];
    const int b0 = ht & 48, bj = ht & 15;
    if (ht < kC) {
#pragma unroll
      for (int i = 0; i < 16; ++i) {
        float acc[2] = {};
#pragma unroll
        for (int m = 0; m < i; ++m) acc[m & 1] = fmaf(am[(b0 + i) * kLd + b0 + m], inv[m], acc[m & 1]);
        inv[i] = i == bj ? 1.f : i < bj ? 0.f : -(acc[0] + acc[1]);
      }
    }
    half_sync();
    if (ht < kC) {
#pragma unroll
      for (int i = 0; i < 16; ++i) am[(b0 + i) * kLd + b0 + bj] = inv[i];
    }
    half_sync();
    // then the lower left blocks, -T_low . (A . T_up), of 16 and of 32; the inner products lie in the unused upper right
    {
      const int o = hw & 2 ? 32 : 0, c = (hw & 1) * 8;
      float *scratch = am + o * kLd + o + 16 + c;
      small_product(scratch, am + (o + 16) * kLd + o, am + o * kLd + o + c, 1, 1.f, lane);
      half_sync();
      small_product(am + (o + 16) * kLd + o + c, am + (o + 16) * kLd + o + 16, scratch, 1, -1.f, lane);
      half_sync();
      const int n = hw * 8, k0 = n >> 4;  // blocks of T_up above its diagonal are zero, and not read
#pragma unroll
      for (int m = 0; m < 2; ++m)
        small_product(am + m * 16 * kLd + 32 + n, am + (32 + m * 16) * kLd + k0 * 16, am + k0 * 16 * kLd + n, 2 - k0, 1.f, lane);
      half_sync();
#pragma unroll
      for (int m = 0; m < 2; ++m) small_product(am + (32 + m * 16) * kLd + n, am + (32 + m * 16) * kLd + 32, am + 32 + n, m + 1, -1.f, lane);
      half_sync();
    }
#pragma unroll
    for (int blk = 0; blk < 10; ++blk) {
      const int m = blk < 1 ? 0 : blk < 3 ? 1 : blk < 6 ? 2 : 3, k = blk - m * (m + 1) / 2;
      const int r = ht >> 3, c = (ht & 7) * 2, s = k * 16 + c;
      const float2 v = *reinterpret_cast<const float2 *>(am + (m * 16 + r) * kLd + s), b = *reinterpret_cast<const float2 *>(beta + s);
      uint32_t high, low;
      split(v.x * b.x, v.y * b.y, high, low);
      const uint32_t off = block_at(m, k, r, c >> 3) + (c & 7) * 2;
      *reinterpret_cast<uint32_t *>(dst + off) = high;
      *reinterpret_cast<uint32_t *>(dst + kSquare + off) = low;
    }
  }
}

// ---- the walk over a sequence's chunks ------------------------------------------------------------------
// kWarps pairs of warps (the chain and the read-out) per CTA, kN tiles of 8 value columns each.  One tile makes the shorter
// chain; two read the operands from shared memory once for both, whose bandwidth is the limit when an SM has many pairs.
template <int kDK, int kWarps, int kN>
struct ScanSmem {
  static constexpr int kTile = KeyTiles<kDK>::kTile, kTiles = kWarps * kN;
  static constexpr int kOffHead = 2 * kTile, kOffValues = kOffHead + kHeadTiles, kStage = kOffValues + kTiles * kValueTile;
  static constexpr int kState = kDK / 16 * kN * 512, kHandOver = kState + 4 * kN * 512;  // S as operands B, U as accumulators
  static constexpr int kRest = kWarps * kHandOver + 512, kRoom = 227 * 1024 - kRest;
  static constexpr int kStages = kRoom >= 4 * kStage ? 4 : kRoom >= 3 * kStage ? 3 : 2;
  static constexpr int kOffHand = kStages * kStage, kOffBar = kOffHand + kWarps * kHandOver, kBytes = kOffBar + 512;
  static constexpr int kThreads = (2 * kWarps + 1) * 32;
};

// An 8 x 8 matrix of 16-bit elements, a row's pairs in four lanes, transposed.
__device__ __forceinline__ uint32_t transposed(uint32_t v) {
  uint32_t r;
  asm("movmatrix.sync.aligned.m8n8.trans.b16 %0, %1;" : "=r"(r) : "r"(v));
  return r;
}

// Operand B (16 x 8) in two parts from an accumulator tile (16 x 8).
__device__ __forceinline__ void split_operand(const float (&c)[4], uint32_t (&high)[2], uint32_t (&low)[2]) {
#pragma unroll
  for (int i = 0; i < 2; ++i) {
    uint32_t h, l;
    split(c[2 * i], c[2 * i + 1], h, l);
    high[i] = transposed(h);
    low[i] = transposed(l);
  }
}

// acc (64 x 8 kN) += m (lower triangular, 64 x 64, in two parts) . x (64 x 8 kN, in two parts)
template <int kN>
__device__ __forceinline__ void triangular_product(float (&acc)[kN][4][4], uint32_t m_high, uint32_t m_low, const uint32_t (&high)[kN][4][2],
                                                   const uint32_t (&low)[kN][4][2], int lane) {
#pragma unroll
  for (int k = 0; k < 4; ++k) {
    uint32_t a[4][4], b[4][4];
#pragma unroll
    for (int m = k; m < 4; ++m) {
      const uint32_t at = block_at(m, k, lane & 15, lane >> 4);
      ldmatrix_x4(a[m][0], a[m][1], a[m][2], a[m][3], m_high + at);
      ldmatrix_x4(b[m][0], b[m][1], b[m][2], b[m][3], m_low + at);
    }
#pragma unroll
    for (int c = 0; c < kN; ++c)
#pragma unroll
      for (int m = k; m < 4; ++m) mma_16816_bf16(acc[c][m], a[m], high[c][k][0], high[c][k][1]);
#pragma unroll
    for (int c = 0; c < kN; ++c)
#pragma unroll
      for (int m = k; m < 4; ++m) mma_16816_bf16(acc[c][m], a[m], low[c][k][0], low[c][k][1]);
#pragma unroll
    for (int c = 0; c < kN; ++c)
#pragma unroll
      for (int m = k; m < 4; ++m) mma_16816_bf16(acc[c][m], b[m], high[c][k][0], high[c][k][1]);
  }
}

// acc (64 x 8 kN) += rows of a tile . s, for one slice of 16 keys, s in two parts
template <int kN>
__device__ __forceinline__ void slice_product(float (&acc)[kN][4][4], uint32_t tile, int k, int pieces, const uint32_t (&high)[kN][2],
                                              const uint32_t (&low)[kN][2], int lane) {
  uint32_t a[4][4];
#pragma unroll
  for (int m = 0; m < 4; ++m)
    ldmatrix_x4(a[m][0], a[m][1], a[m][2], a[m][3], tile + tile_at(16 * m + (lane & 15), 2 * k + (lane >> 4), pieces));
#pragma unroll
  for (int c = 0; c < kN; ++c)
#pragma unroll
    for (int m = 0; m < 4; ++m) mma_16816_bf16(acc[c][m], a[m], high[c][0], high[c][1]);
#pragma unroll
  for (int c = 0; c < kN; ++c)
#pragma unroll
    for (int m = 0; m < 4; ++m) mma_16816_bf16(acc[c][m], a[m], low[c][0], low[c][1]);
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

template <int kDK, int kWarps, int kN>
__global__ void __launch_bounds__(ScanSmem<kDK, kWarps, kN>::kThreads, 1) delta_chunk_scan_kernel(const ScanParams p) {
  using L = ScanSmem<kDK, kWarps, kN>;
  constexpr int kPieces = kDK / 8, kKeyTiles = kDK / 16;  // 16-high tiles of S
  extern __shared__ __align__(128) uint8_t smem[];
  uint64_t *full = reinterpret_cast<uint64_t *>(smem + L::kOffBar), *empty = full + L::kStages;
  uint64_t *s_full = empty + L::kStages, *s_empty = s_full + kWarps, *u_full = s_empty + kWarps, *u_empty = u_full + kWarps;
  volatile int *abort_flag = reinterpret_cast<volatile int *>(u_empty + kWarps);
  const int warp = __shfl_sync(0xffffffffu, (int)(threadIdx.x >> 5), 0), lane = threadIdx.x & 31;
  const int h = blockIdx.y, hk = h / (p.heads / p.kv_heads), blocks = p.vdim / 8, block0 = blockIdx.z * L::kTiles;
  const int tiles_here = min(L::kTiles, blocks - block0), warps = (tiles_here + kN - 1) / kN;  // with columns of their own
  if (threadIdx.x == 0) {
    for (int i = 0; i < L::kStages; ++i) {
      mbar_init(&full[i], 1);
      mbar_init(&empty[i], 2 * warps);
    }
    for (int i = 0; i < 4 * kWarps; ++i) mbar_init(&s_full[i], 1);
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

  if (warp == 2 * kWarps) {
    // ---- bulk copies ----
    if (lane == 0) {
      bool ok = true;
      int n = 0;
      for (; n < chunks; ++n) {
        const int s = n % L::kStages;
        if (n >= L::kStages) ok = mbar_wait_bounded(&empty[s], (n / L::kStages - 1) & 1, abort_flag, p.wait_ns);
        if (!ok) break;
        const size_t chunk = chunk0 + n;
        uint8_t *dst = smem + s * L::kStage;
        mbar_arrive_expect_tx(&full[s], 2 * L::kTile + kHeadTiles + tiles_here * kValueTile);
        bulk_load(dst, p.keys + (chunk * p.kv_heads + hk) * KeyTiles<kDK>::kBytes, 2 * L::kTile, &full[s]);
        bulk_load(dst + L::kOffHead, p.heads_tiles + (chunk * p.heads + h) * kHeadTiles, kHeadTiles, &full[s]);
        bulk_load(dst + L::kOffValues, p.values + ((chunk * p.heads + h) * blocks + block0) * kValueTile, tiles_here * kValueTile, &full[s]);
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
  const int w = warp % kWarps;
  if (w >= warps) return;
  auto wait = [&](uint64_t *bar, int phase) { return __all_sync(0xffffffffu, mbar_wait_bounded(bar, phase & 1, abort_flag, p.wait_ns)); };
  auto release = [&](uint64_t *bar) {
    __syncwarp();
    if (lane == 0) mbar_arrive(bar);
  };
  // an accumulator tile's rows are lane / 4 and + 8, its columns (lane % 4) * 2 and + 1
  const int g = lane >> 2, v0 = (block0 + w * kN) * 8 + (lane & 3) * 2;
  auto mine = [&](int c) { return v0 + 8 * c < p.vdim; };  // a last tile of a pair may not exist: its columns are never stored
  uint4 *hand_s = reinterpret_cast<uint4 *>(smem + L::kOffHand + w * L::kHandOver) + lane;
  float4 *hand_u = reinterpret_cast<float4 *>(smem + L::kOffHand + w * L::kHandOver + L::kState) + lane;

  if (warp >= kWarps) {
    // ---- the read-out: o = e^G q S + P u ----
    for (int n = 0; n < chunks; ++n) {
      const int s = n % L::kStages;
      if (!wait(&full[s], n / L::kStages) || !wait(&s_full[w], n)) return;
      const uint32_t cq = smem_u32(smem + s * L::kStage + L::kTile), tiles = smem_u32(smem + s * L::kStage + L::kOffHead);
      const float *vec = reinterpret_cast<const float *>(smem + s * L::kStage + L::kOffHead + kVec);
      float o[kN][4][4] = {};
#pragma unroll
      for (int k = 0; k < kKeyTiles; ++k) {
        uint32_t sh[kN][2], sl[kN][2];
#pragma unroll
        for (int c = 0; c < kN; ++c) {
          const uint4 v = hand_s[(k * kN + c) * 32];
          sh[c][0] = v.x, sh[c][1] = v.y, sl[c][0] = v.z, sl[c][1] = v.w;
        }
        slice_product<kN>(o, cq, k, kPieces, sh, sl, lane);
      }
      release(&s_empty[w]);
      if (!wait(&u_full[w], n)) return;
      uint32_t high[kN][4][2], low[kN][4][2];
#pragma unroll
      for (int m = 0; m < 4; ++m) {
        const float e0 = vec[kC + 16 * m + g], e1 = vec[kC + 16 * m + g + 8];
#pragma unroll
        for (int c = 0; c < kN; ++c) {
          o[c][m][0] *= e0, o[c][m][1] *= e0, o[c][m][2] *= e1, o[c][m][3] *= e1;
          const float4 v = hand_u[(m * kN + c) * 32];
          const float u[4] = {v.x, v.y, v.z, v.w};
          split_operand(u, high[c][m], low[c][m]);
        }
      }
      release(&u_empty[w]);
      triangular_product<kN>(o, tiles + 2 * kSquare, tiles + 3 * kSquare, high, low, lane);
      release(&empty[s]);
      const int valid = portion.z - n * kC;
      __nv_bfloat16 *dst = p.out + ((int64_t)(portion.y - p.first + n * kC) * p.heads + h) * p.vdim + v0;
#pragma unroll
      for (int c = 0; c < kN; ++c)
#pragma unroll
        for (int m = 0; m < 4; ++m)
#pragma unroll
          for (int i = 0; i < 2; ++i) {
            const int t = 16 * m + g + 8 * i;
            if (t < valid && mine(c))
              *reinterpret_cast<uint32_t *>(dst + (int64_t)t * p.heads * p.vdim + 8 * c) = pack_bf16x2(o[c][m][2 * i], o[c][m][2 * i + 1]);
          }
    }
    return;
  }

  // ---- the chain ----
  float *state = p.state + ((size_t)portion.x * p.heads + h) * p.dim * p.vdim;
  float st[kN][kKeyTiles][4];  // S: tile j holds keys 16j .. 16j + 15
#pragma unroll
  for (int c = 0; c < kN; ++c)
#pragma unroll
    for (int j = 0; j < kKeyTiles; ++j)
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int k = 16 * j + g + 8 * i;
        float2 v = make_float2(0.f, 0.f);
        if (portion.w > 0 && k < p.dim && mine(c)) v = *reinterpret_cast<const float2 *>(state + (size_t)k * p.vdim + v0 + 8 * c);
        st[c][j][2 * i] = v.x, st[c][j][2 * i + 1] = v.y;
      }

  for (int n = 0; n < chunks; ++n) {
    const int s = n % L::kStages;
    if (n > 0 && !wait(&s_empty[w], n - 1)) return;
    if (!wait(&full[s], n / L::kStages)) return;
    const uint32_t base = smem_u32(smem + s * L::kStage), ck = base, tiles = base + L::kOffHead;
    const float *vec = reinterpret_cast<const float *>(smem + s * L::kStage + L::kOffHead + kVec);
    const uint8_t *value = smem + s * L::kStage + L::kOffValues + w * kN * kValueTile + (lane & 3) * 4;

    // k S of all tokens; S is handed over on the way
    float x[kN][4][4] = {};
#pragma unroll
    for (int k = 0; k < kKeyTiles; ++k) {
      uint32_t sh[kN][2], sl[kN][2];
#pragma unroll
      for (int c = 0; c < kN; ++c) {
        split_operand(st[c][k], sh[c], sl[c]);
        hand_s[(k * kN + c) * 32] = make_uint4(sh[c][0], sh[c][1], sl[c][0], sl[c][1]);
      }
      slice_product<kN>(x, ck, k, kPieces, sh, sl, lane);
    }
    release(&s_full[w]);
    // X = v - e^G k S
    uint32_t high[kN][4][2], low[kN][4][2];
#pragma unroll
    for (int m = 0; m < 4; ++m)
#pragma unroll
      for (int c = 0; c < kN; ++c) {
#pragma unroll
        for (int i = 0; i < 2; ++i) {
          const int t = 16 * m + g + 8 * i;
          const uint32_t v = *reinterpret_cast<const uint32_t *>(value + c * kValueTile + t * 16);
          const float e = vec[t];
          x[c][m][2 * i] = fmaf(-e, x[c][m][2 * i], bf_lo(v));
          x[c][m][2 * i + 1] = fmaf(-e, x[c][m][2 * i + 1], bf_hi(v));
        }
        split_operand(x[c][m], high[c][m], low[c][m]);
      }
    float u[kN][4][4] = {};
    triangular_product<kN>(u, tiles, tiles + kSquare, high, low, lane);
    if (n > 0 && !wait(&u_empty[w], n - 1)) return;
#pragma unroll
    for (int m = 0; m < 4; ++m)
#pragma unroll
      for (int c = 0; c < kN; ++c) hand_u[(m * kN + c) * 32] = make_float4(u[c][m][0], u[c][m][1], u[c][m][2], u[c][m][3]);
    release(&u_full[w]);
    // S' = e^G_64 S + k^T (e^{G_64 - G} u)
    const float total = vec[3 * kC];
#pragma unroll
    for (int c = 0; c < kN; ++c)
#pragma unroll
      for (int j = 0; j < kKeyTiles; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) st[c][j][e] *= total;
#pragma unroll
    for (int m = 0; m < 4; ++m) {
      const float e0 = vec[2 * kC + 16 * m + g], e1 = vec[2 * kC + 16 * m + g + 8];
      uint32_t wh[kN][2], wl[kN][2];
#pragma unroll
      for (int c = 0; c < kN; ++c) {
        const float wu[4] = {e0 * u[c][m][0], e0 * u[c][m][1], e1 * u[c][m][2], e1 * u[c][m][3]};
        split_operand(wu, wh[c], wl[c]);
      }
#pragma unroll
      for (int j0 = 0; j0 < kKeyTiles; j0 += 4) {
        uint32_t a[4][4];
#pragma unroll
        for (int j = 0; j < 4; ++j)
          ldmatrix_x4_trans(a[j][0], a[j][1], a[j][2], a[j][3],
                            ck + tile_at(16 * m + ((lane >> 4) & 1) * 8 + (lane & 7), 2 * (j0 + j) + ((lane >> 3) & 1), kPieces));
#pragma unroll
        for (int c = 0; c < kN; ++c)
#pragma unroll
          for (int j = 0; j < 4; ++j) mma_16816_bf16(st[c][j0 + j], a[j], wh[c][0], wh[c][1]);
#pragma unroll
        for (int c = 0; c < kN; ++c)
#pragma unroll
          for (int j = 0; j < 4; ++j) mma_16816_bf16(st[c][j0 + j], a[j], wl[c][0], wl[c][1]);
      }
    }
    release(&empty[s]);
  }
#pragma unroll
  for (int c = 0; c < kN; ++c)
#pragma unroll
    for (int j = 0; j < kKeyTiles; ++j)
#pragma unroll
      for (int i = 0; i < 2; ++i) {
        const int k = 16 * j + g + 8 * i;
        if (k < p.dim && mine(c))
          *reinterpret_cast<float2 *>(state + (size_t)k * p.vdim + v0 + 8 * c) = make_float2(st[c][j][2 * i], st[c][j][2 * i + 1]);
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

template <int kDK, int kWarps, int kN>
int run_scan(const ScanParams &p, int count, cudaStream_t st) {
  using L = ScanSmem<kDK, kWarps, kN>;
  if (int rc = opt_in<delta_chunk_scan_kernel<kDK, kWarps, kN>>(L::kBytes)) return rc;
  return launch_dependent(delta_chunk_scan_kernel<kDK, kWarps, kN>, dim3(count, p.heads, (p.vdim / 8 + L::kTiles - 1) / L::kTiles),
                          dim3(L::kThreads), (size_t)L::kBytes, st, p);
}

template <int kDK>
int run(const DeltaParams<__nv_bfloat16> &d, const ScanParams &s, int count, int longest, uint8_t *keys, uint8_t *heads, uint8_t *values,
        cudaStream_t st) {
  using P = PrepSmem<kDK>;
  if (int rc = opt_in<delta_chunk_prepare_kernel<kDK>>(P::kBytes)) return rc;
  const int chunks = (longest + kC - 1) / kC;
  if (int rc = launch_dependent(delta_chunk_conv_kernel<kDK>, dim3(chunks, count, 2 * d.kv_heads + (d.heads * d.vdim + 127) / 128), dim3(128),
                                0, st, d, s.portions, s.first, keys, values))
    return rc;
  if (int rc = launch_dependent(delta_chunk_prepare_kernel<kDK>, dim3(chunks, count, d.kv_heads), dim3(kPrepThreads), (size_t)P::kBytes, st, d,
                                s.portions, s.first, keys, heads, s.wait_ns))
    return rc;
  // as few columns in a CTA as give every SM at most one
  int dev = 0, sms = 0;
  if (cudaGetDevice(&dev) != cudaSuccess || cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess)
    return AXB200_DEVICE_ERROR;
  const int64_t tiles = (int64_t)count * d.heads * (d.vdim / 8);
  if (tiles <= sms) return run_scan<kDK, 1, 1>(s, count, st);
  if (tiles <= 2 * sms) return run_scan<kDK, 2, 1>(s, count, st);
  if (tiles <= 4 * sms) return run_scan<kDK, 4, 1>(s, count, st);
  return run_scan<kDK, 4, 2>(s, count, st);
}

int padded_dim(int dim) { return dim <= 64 ? 64 : 128; }
size_t key_bytes(int dim) { return padded_dim(dim) == 64 ? KeyTiles<64>::kBytes : KeyTiles<128>::kBytes; }
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
         ((size_t)kv_heads * axb::key_bytes(dim) +
          (size_t)heads * (axb::kHeadTiles + (size_t)(vdim / 8) * axb::kValueTile));
}

int axb200_delta_chunks(const void *proj, int64_t ld, int first, int rows, const float *conv, const float *a_log,
                        const float *dt_bias, const void *ring, float *state, const int32_t *portions, int count, int longest, void *out, int heads, int kv_heads, int dim, int vdim,
                        int taps, int max_seqs, int dtype, void *workspace, size_t workspace_bytes, void *stream) {
  if (!axb200_delta_chunks_supported(dim, vdim, dtype)) return AXB200_UNSUPPORTED_TYPE;
  if (!proj || !conv || !a_log || !dt_bias || !ring || !state || !portions || !out || !workspace)
    return AXB200_INVALID_PTR;
  if (first < 0 || first > rows || count < 0 || count > 65535 || longest < 0 || heads <= 0 || kv_heads <= 0 || heads % kv_heads != 0 ||
      heads > 65535 || 2 * (int64_t)kv_heads + ((int64_t)heads * vdim + 127) / 128 > 65535 || taps <= 0 || max_seqs <= 0)
    return AXB200_INVALID_ARGUMENT;
  if (ld < (int64_t)2 * kv_heads * dim + (int64_t)heads * (2 * vdim + 2)) return AXB200_SHAPE_MISMATCH;
  if (ld % 4 || !axb::al16(proj) || !axb::al16(conv) || !axb::al16(ring) || !axb::al16(portions) || !axb::al16(out) ||
      (reinterpret_cast<uintptr_t>(workspace) & 127u))
    return AXB200_UNSUPPORTED_TYPE;
  if (count == 0 || first == rows) return AXB200_OK;
  if (workspace_bytes < axb200_delta_chunks_workspace_bytes(rows - first, count, heads, kv_heads, dim, vdim)) return AXB200_OUT_OF_MEMORY;
  const axb::DeltaParams<__nv_bfloat16> d{static_cast<const __nv_bfloat16 *>(proj), ld, nullptr, nullptr, nullptr, rows, conv, a_log,
                                          dt_bias, nullptr, static_cast<__nv_bfloat16 *>(const_cast<void *>(ring)), state, heads, kv_heads, dim, vdim, taps,
                                          max_seqs, 0.f};
  const size_t slots = (size_t)axb::chunk_slots(rows - first, count);
  uint8_t *keys = static_cast<uint8_t *>(workspace);
  uint8_t *tiles = keys + slots * kv_heads * axb::key_bytes(dim);
  uint8_t *values = tiles + slots * heads * axb::kHeadTiles;
  const axb::ScanParams s{reinterpret_cast<const int4 *>(portions), first, keys, tiles, values, state, static_cast<__nv_bfloat16 *>(out),
                          heads, kv_heads, dim, vdim, max_seqs, axb::wait_limit_ns()};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return axb::padded_dim(dim) == 64 ? axb::run<64>(d, s, count, longest, keys, tiles, values, st)
                                    : axb::run<128>(d, s, count, longest, keys, tiles, values, st);
}

}  // extern "C"
