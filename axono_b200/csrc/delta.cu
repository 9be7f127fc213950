// The gated delta rule: a recurrent mixer whose state per sequence and head is a matrix S (dim x vdim) in fp32,
//     S <- g S,   u = beta (v - S^T k),   S <- S + k u^T,   o = S^T q,
// with q, k and v behind a short causal convolution over time and silu, q and k unit vectors (q also over sqrt(dim)), one
// decay g and one step beta per head; o is normed over vdim, weighted and gated.
//
//   delta_step_bulk_kernel  decoded tokens: convolution, norms, recurrence, norm and gate of one token in one launch, the
//                         state through shared memory by bulk copies; delta_step_kernel: the same through registers, for
//                         states that are too large or oddly sized
//   delta_prepare_kernel  portions: convolution, silu and unit norms of every row, decays and steps
//   delta_scan_kernel     portions, token by token with S in registers
//   delta_finish_kernel   portions: norm and gate of the outputs; the ring of inputs for the next step's convolution
//
// A sequence's first token (position 0) starts from a zero state whatever its slot held before.
#include <math.h>

#include "delta.cuh"

namespace axb {
namespace {

constexpr float kUnitEps = 1e-6f;

__device__ __forceinline__ bool bad_seq(int seq, int max_seqs, bool report) {
  if (seq >= 0 && seq < max_seqs) return false;
  if (report) atomicOr(&g_error_word, AXB200_ERR_CAPACITY);
  return true;
}

// ---- decoded tokens ----------------------------------------------------------------------------------
// One CTA per (row, head).  Warps split the rows of S, lanes its columns (kVec each, 32 * kVec per pass), so the state
// moves in whole 128-byte lines; a thread keeps its part in registers between the product with k and the update.  One
// reduction over the warps gives S^T k and S^T q together: o = g S^T q + (k . q) u.
constexpr int kStepThreads = 256, kStepWarps = kStepThreads / 32;

template <typename T, int kVec, int kRowsPerWarp>
__global__ void __launch_bounds__(kStepThreads)
delta_step_kernel(const DeltaParams<T> p, T *out) {
  extern __shared__ float sm[];
  __shared__ float scratch[32], part[2][kStepWarps][32 * kVec];
  float *q = sm, *k = q + p.dim, *v = k + p.dim, *o = v + p.vdim;
  const int64_t r = blockIdx.x;
  const int h = blockIdx.y, hk = h / (p.heads / p.kv_heads), warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  grid_dependency_wait();
  grid_dependency_launch();
  const int seq = p.row_seq[r], pos = p.row_pos[r];
  if (bad_seq(seq, p.max_seqs, threadIdx.x == 0)) return;
  const bool fresh = pos == 0;
  float *state = p.state + ((size_t)seq * p.heads + h) * p.dim * p.vdim;
  const int row0 = warp * kRowsPerWarp, row1 = min(row0 + kRowsPerWarp, p.dim);
  float s[kRowsPerWarp][kVec];
  auto load_state = [&](int col) {
#pragma unroll
    for (int i = 0; i < kRowsPerWarp; ++i) {
#pragma unroll
      for (int e = 0; e < kVec; ++e) s[i][e] = 0.f;
      if (!fresh && row0 + i < row1 && col < p.vdim) load_vec<kVec>(state + (size_t)(row0 + i) * p.vdim + col, s[i]);
    }
  };
  load_state(lane * kVec);  // on its way while the inputs are prepared

  // convolution and silu; the head that owns a channel files its input in the ring
  const int channels = p.channels(), slot = pos % p.taps;
  const T *x = p.proj + r * p.ld;
  T *ring = p.ring + (size_t)seq * p.taps * channels;
  const bool owns_qk = h % (p.heads / p.kv_heads) == 0;
  for (int i = threadIdx.x; i < 2 * p.dim + p.vdim; i += kStepThreads) {
    const int c = i < p.dim ? hk * p.dim + i : i < 2 * p.dim ? (p.kv_heads + hk) * p.dim + i - p.dim
                                                             : 2 * p.kv_heads * p.dim + h * p.vdim + i - 2 * p.dim;
    const T now = x[c];
    float acc = ldf(&now) * p.conv[(size_t)(p.taps - 1) * channels + c];
    for (int j = 1; j < p.taps && j <= pos; ++j)
      acc = fmaf(ldf(ring + (size_t)((pos - j) % p.taps) * channels + c), p.conv[(size_t)(p.taps - 1 - j) * channels + c], acc);
    if (owns_qk || i >= 2 * p.dim) ring[(size_t)slot * channels + c] = now;
    sm[i] = silu(acc);
  }
  __syncthreads();
  float qq = 0.f, kk = 0.f, kq = 0.f;
  for (int i = threadIdx.x; i < p.dim; i += kStepThreads) {
    qq = fmaf(q[i], q[i], qq);
    kk = fmaf(k[i], k[i], kk);
    kq = fmaf(k[i], q[i], kq);
  }
  qq = block_sum(qq, scratch);
  kk = block_sum(kk, scratch);
  kq = block_sum(kq, scratch);
  const float inv_q = 1.0f / (sqrtf(qq + kUnitEps) * sqrtf((float)p.dim)), inv_k = 1.0f / sqrtf(kk + kUnitEps);
  kq *= inv_q * inv_k;
  for (int i = threadIdx.x; i < p.dim; i += kStepThreads) {
    q[i] *= inv_q;
    k[i] *= inv_k;
  }
  const float g = expf(log_decay(ldf(x + p.a_at() + h), p.a_log[h], p.dt_bias[h])), beta = sigmoid(ldf(x + p.b_at() + h));
  __syncthreads();

  float sq = 0.f;
  for (int col0 = 0; col0 < p.vdim; col0 += 32 * kVec) {
    const int col = col0 + lane * kVec;
    if (col0 > 0) {
      load_state(col);
      __syncthreads();
    }
    float sk[kVec] = {}, so[kVec] = {};
#pragma unroll
    for (int i = 0; i < kRowsPerWarp; ++i) {
      if (row0 + i >= row1) break;
      const float ki = k[row0 + i], qi = q[row0 + i];
#pragma unroll
      for (int e = 0; e < kVec; ++e) {
        s[i][e] *= g;
        sk[e] = fmaf(s[i][e], ki, sk[e]);
        so[e] = fmaf(s[i][e], qi, so[e]);
      }
    }
#pragma unroll
    for (int e = 0; e < kVec; ++e) {
      part[0][warp][lane * kVec + e] = sk[e];
      part[1][warp][lane * kVec + e] = so[e];
    }
    __syncthreads();
    float u[kVec] = {};
    if (col < p.vdim) {
#pragma unroll
      for (int e = 0; e < kVec; ++e) {
        float a = 0.f, b = 0.f;
#pragma unroll
        for (int w = 0; w < kStepWarps; ++w) {
          a += part[0][w][lane * kVec + e];
          b += part[1][w][lane * kVec + e];
        }
        u[e] = beta * (v[col + e] - a);
        if (warp == 0) {
          const float y = fmaf(kq, u[e], b);
          o[col + e] = y;
          sq = fmaf(y, y, sq);
        }
      }
#pragma unroll
      for (int i = 0; i < kRowsPerWarp; ++i) {
        if (row0 + i >= row1) break;
        const float ki = k[row0 + i];
#pragma unroll
        for (int e = 0; e < kVec; ++e) s[i][e] = fmaf(ki, u[e], s[i][e]);
        store_vec<kVec>(state + (size_t)(row0 + i) * p.vdim + col, s[i]);
      }
    }
  }
  const float inv = 1.0f / sqrtf(block_sum(sq, scratch) / (float)p.vdim + p.eps);  // also: o is complete
  for (int i = threadIdx.x; i < p.vdim; i += kStepThreads)
    stf(out + (r * p.heads + h) * p.vdim + i, o[i] * inv * ldf(p.norm + i) * silu(ldf(x + p.gate_at() + h * p.vdim + i)));
}

// The same with the state in shared memory: one bulk copy fetches it while the inputs are prepared, one bulk copy puts it
// back, and with no registers tied up several CTAs per SM keep enough bytes on their way.  dim and vdim are multiples of 4.
template <typename T>
__global__ void __launch_bounds__(kStepThreads, 3) delta_step_bulk_kernel(const DeltaParams<T> p, T *out, unsigned long long wait_ns) {
  extern __shared__ __align__(128) float sm[];
  __shared__ float scratch[3][kStepWarps];
  __shared__ alignas(8) uint64_t bar;
  __shared__ int abort_flag;
  float *s = sm, *q = s + p.dim * p.vdim, *k = q + p.dim, *v = k + p.dim, *o = v + p.vdim, *part = o + p.vdim;
  const int64_t r = blockIdx.x;
  const int h = blockIdx.y, group = p.heads / p.kv_heads, hk = h / group, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x == 0) {
    mbar_init(&bar, 1);
    abort_flag = 0;
    mbar_fence_init();
  }
  __syncthreads();
  grid_dependency_wait();
  grid_dependency_launch();
  const int seq = p.row_seq[r], pos = p.row_pos[r];
  if (bad_seq(seq, p.max_seqs, threadIdx.x == 0)) return;
  const bool fresh = pos == 0;
  float *state = p.state + ((size_t)seq * p.heads + h) * p.dim * p.vdim;
  const uint32_t bytes = (uint32_t)(p.dim * p.vdim) * 4;
  if (threadIdx.x == 0 && !fresh) {
    mbar_arrive_expect_tx(&bar, bytes);
    bulk_load(s, state, bytes, &bar);
  }
  if (fresh)
    for (int i = threadIdx.x * 4; i < p.dim * p.vdim; i += kStepThreads * 4) *reinterpret_cast<float4 *>(s + i) = make_float4(0.f, 0.f, 0.f, 0.f);

  const int channels = p.channels(), slot = pos % p.taps;
  const T *x = p.proj + r * p.ld;
  T *ring = p.ring + (size_t)seq * p.taps * channels;
  const bool owns_qk = h % group == 0;
  const float a_in = ldf(x + p.a_at() + h), b_in = ldf(x + p.b_at() + h), a_log = p.a_log[h], dt_bias = p.dt_bias[h];
  // two neighbouring channels per thread; query and key elements stay with the threads whose sums they enter
  float sq[3] = {};  // q.q, k.k, k.q come out of one reduction each, k.q after the exchange
  for (int i = threadIdx.x * 2; i < 2 * p.dim + p.vdim; i += kStepThreads * 2) {
    const int c = i < p.dim ? hk * p.dim + i : i < 2 * p.dim ? (p.kv_heads + hk) * p.dim + i - p.dim
                                                             : 2 * p.kv_heads * p.dim + h * p.vdim + i - 2 * p.dim;
    float acc[2], in[2], w[2];
    load_vec<2>(x + c, in);
    load_vec<2>(p.conv + (size_t)(p.taps - 1) * channels + c, w);
    acc[0] = in[0] * w[0], acc[1] = in[1] * w[1];
    for (int j = 1; j < p.taps && j <= pos; ++j) {
      float old[2];
      load_vec<2>(ring + (size_t)((pos - j) % p.taps) * channels + c, old);
      load_vec<2>(p.conv + (size_t)(p.taps - 1 - j) * channels + c, w);
      acc[0] = fmaf(old[0], w[0], acc[0]), acc[1] = fmaf(old[1], w[1], acc[1]);
    }
    if (owns_qk || i >= 2 * p.dim) store_vec<2>(ring + (size_t)slot * channels + c, in);
    acc[0] = silu(acc[0]), acc[1] = silu(acc[1]);
    *reinterpret_cast<float2 *>(q + i) = make_float2(acc[0], acc[1]);
    const float both = fmaf(acc[0], acc[0], acc[1] * acc[1]);
    if (i < p.dim)
      sq[0] += both;
    else if (i < 2 * p.dim)
      sq[1] += both;
  }
  __syncthreads();
  for (int i = threadIdx.x; i < p.dim; i += kStepThreads) sq[2] = fmaf(q[i], k[i], sq[2]);
#pragma unroll
  for (int i = 0; i < 3; ++i) {
    sq[i] = warp_sum(sq[i]);
    if (lane == 0) scratch[i][warp] = sq[i];
  }
  const float g = expf(log_decay(a_in, a_log, dt_bias)), beta = sigmoid(b_in);
  __syncthreads();
#pragma unroll
  for (int i = 0; i < 3; ++i) {
    sq[i] = 0.f;
#pragma unroll
    for (int w = 0; w < kStepWarps; ++w) sq[i] += scratch[i][w];
  }
  const float inv_q = 1.0f / (sqrtf(sq[0] + kUnitEps) * sqrtf((float)p.dim)), inv_k = 1.0f / sqrtf(sq[1] + kUnitEps);
  const float kq = sq[2] * inv_q * inv_k;
  if (!fresh && !mbar_wait_bounded(&bar, 0, &abort_flag, wait_ns)) {  // no copy may still be on its way when the CTA leaves
    const unsigned long long t0 = global_timer_ns();
    while (!mbar_try_wait(&bar, 0) && global_timer_ns() - t0 < 100000000ull) {
    }
    return;
  }

  // g S^T k and g S^T q: a warp's rows, a lane's four columns
  const int rows = (p.dim + kStepWarps - 1) / kStepWarps, row0 = warp * rows, row1 = min(row0 + rows, p.dim);
  for (int col = lane * 4; col < p.vdim; col += 128) {
    float4 a = make_float4(0.f, 0.f, 0.f, 0.f), b = a;
#pragma unroll 8
    for (int i = row0; i < row1; ++i) {
      const float4 e = *reinterpret_cast<const float4 *>(s + i * p.vdim + col);
      const float ki = k[i], qi = q[i];
      a.x = fmaf(e.x, ki, a.x), a.y = fmaf(e.y, ki, a.y), a.z = fmaf(e.z, ki, a.z), a.w = fmaf(e.w, ki, a.w);
      b.x = fmaf(e.x, qi, b.x), b.y = fmaf(e.y, qi, b.y), b.z = fmaf(e.z, qi, b.z), b.w = fmaf(e.w, qi, b.w);
    }
    *reinterpret_cast<float4 *>(part + warp * 2 * p.vdim + col) = a;
    *reinterpret_cast<float4 *>(part + (warp * 2 + 1) * p.vdim + col) = b;
  }
  __syncthreads();
  float oo = 0.f;
  for (int c = threadIdx.x; c < p.vdim; c += kStepThreads) {
    float a = 0.f, b = 0.f;
#pragma unroll
    for (int w = 0; w < kStepWarps; ++w) {
      a += part[w * 2 * p.vdim + c];
      b += part[(w * 2 + 1) * p.vdim + c];
    }
    const float u = beta * (v[c] - g * inv_k * a), y = fmaf(kq, u, g * inv_q * b);
    v[c] = u * inv_k;  // what the rows of S are updated with, times k
    o[c] = y;
    oo = fmaf(y, y, oo);
  }
  oo = warp_sum(oo);
  if (lane == 0) scratch[0][warp] = oo;
  __syncthreads();
  for (int col = lane * 4; col < p.vdim; col += 128) {
    const float4 u = *reinterpret_cast<const float4 *>(v + col);
#pragma unroll 8
    for (int i = row0; i < row1; ++i) {
      float4 e = *reinterpret_cast<const float4 *>(s + i * p.vdim + col);
      const float ki = k[i];
      e.x = fmaf(ki, u.x, g * e.x), e.y = fmaf(ki, u.y, g * e.y), e.z = fmaf(ki, u.z, g * e.z), e.w = fmaf(ki, u.w, g * e.w);
      *reinterpret_cast<float4 *>(s + i * p.vdim + col) = e;
    }
  }
  asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
  __syncthreads();
  if (threadIdx.x == 0) bulk_store(state, s, bytes);
  oo = 0.f;
#pragma unroll
  for (int w = 0; w < kStepWarps; ++w) oo += scratch[0][w];
  const float inv = 1.0f / sqrtf(oo / (float)p.vdim + p.eps);
  for (int i = threadIdx.x; i < p.vdim; i += kStepThreads)
    stf(out + (r * p.heads + h) * p.vdim + i, o[i] * inv * ldf(p.norm + i) * silu(ldf(x + p.gate_at() + h * p.vdim + i)));
  if (threadIdx.x == 0) bulk_store_wait();
}

// ---- portions: convolution, unit norms, decays ----------------------------------------------------------
// A warp walks kPrepRows rows of one unit with the last taps inputs in registers: units are the query and the key heads
// (unit norms inside the warp), the value channels in runs of 32 * kVec, and one for the decays and steps.
constexpr int kPrepRows = 16, kPrepWarps = 4;

template <typename T, int kVec, int kRuns>
__global__ void __launch_bounds__(kPrepWarps * 32)
delta_prepare_kernel(const DeltaParams<T> p, int first, float *qk, T *v, float *log_g, float *beta) {
  const int lane = threadIdx.x & 31;
  const int unit = blockIdx.y * kPrepWarps + (threadIdx.x >> 5), run = 32 * kVec;
  const int v_units = (p.heads * p.vdim + run - 1) / run, qk_units = 2 * p.kv_heads;
  grid_dependency_wait();
  grid_dependency_launch();
  if (unit > qk_units + v_units) return;
  const int lo = first + blockIdx.x * kPrepRows, hi = min(lo + kPrepRows, p.rows);
  if (unit == qk_units + v_units) {
    for (int64_t r = lo; r < hi; ++r)
      for (int h = lane; h < p.heads; h += 32) {
        const T *x = p.proj + r * p.ld;
        log_g[(r - first) * p.heads + h] = log_decay(ldf(x + p.a_at() + h), p.a_log[h], p.dt_bias[h]);
        beta[(r - first) * p.heads + h] = sigmoid(ldf(x + p.b_at() + h));
      }
    return;
  }
  const bool is_v = unit >= qk_units;
  const int channels = p.channels(), qk_channels = 2 * p.kv_heads * p.dim;
  const int c0 = is_v ? qk_channels + (unit - qk_units) * run : unit * p.dim;  // the unit's first channel, and its width
  const int width = is_v ? min(run, channels - c0) : p.dim, runs = is_v ? 1 : (p.dim + run - 1) / run;
  const float gain = is_v || unit >= p.kv_heads ? 1.f : 1.0f / sqrtf((float)p.dim);
  float y[kRuns][kVec];
  for (int64_t r = lo; r < hi; ++r) {
    if (bad_seq(p.row_seq[r], p.max_seqs, lane == 0)) continue;
    float sq = 0.f;
#pragma unroll
    for (int n = 0; n < kRuns; ++n) {
      if (n >= runs) break;
      const int i = n * run + lane * kVec;
#pragma unroll
      for (int e = 0; e < kVec; ++e) y[n][e] = 0.f;
      if (i >= width) continue;
      for (int j = 0; j < p.taps; ++j) {
        float in[kVec], w[kVec];
        earlier_input<kVec>(p, r, j, c0 + i, in);
        load_vec<kVec>(p.conv + (size_t)(p.taps - 1 - j) * channels + c0 + i, w);
#pragma unroll
        for (int e = 0; e < kVec; ++e) y[n][e] = fmaf(in[e], w[e], y[n][e]);
      }
#pragma unroll
      for (int e = 0; e < kVec; ++e) {
        y[n][e] = silu(y[n][e]);
        sq = fmaf(y[n][e], y[n][e], sq);
      }
    }
    if (!is_v) sq = warp_sum(sq);
    const float inv = is_v ? 1.f : gain / sqrtf(sq + kUnitEps);
#pragma unroll
    for (int n = 0; n < kRuns; ++n) {
      const int i = n * run + lane * kVec;
      if (n >= runs || i >= width) continue;
#pragma unroll
      for (int e = 0; e < kVec; ++e) y[n][e] *= inv;
      if (is_v)
        store_vec<kVec>(v + (r - first) * (channels - qk_channels) + c0 - qk_channels + i, y[n]);
      else
        store_vec<kVec>(qk + (r - first) * qk_channels + c0 + i, y[n]);
    }
  }
}

// ---- portions, token by token -------------------------------------------------------------------------
// portion[i] = (sequence, first row, rows, start position).  A warp owns kScanCols columns of S, which are independent of
// the others; lane l holds rows l, l + 32, ... of them.
constexpr int kScanCols = 4, kScanWarps = 4;

template <typename T, int kRows>
__global__ void __launch_bounds__(kScanWarps * 32)
delta_scan_kernel(const DeltaParams<T> p, const int4 *portions, int first, const float *qk, const T *v, const float *log_g,
                  const float *beta, T *out) {
  const int lane = threadIdx.x & 31, h = blockIdx.y, hk = h / (p.heads / p.kv_heads);
  const int col0 = (blockIdx.z * kScanWarps + (threadIdx.x >> 5)) * kScanCols;
  grid_dependency_wait();
  grid_dependency_launch();
  if (col0 >= p.vdim) return;
  const int4 portion = portions[blockIdx.x];
  if (bad_seq(portion.x, p.max_seqs, lane == 0)) return;
  const int cols = min(kScanCols, p.vdim - col0);
  float *state = p.state + ((size_t)portion.x * p.heads + h) * p.dim * p.vdim + col0;
  float s[kRows][kScanCols];
#pragma unroll
  for (int i = 0; i < kRows; ++i)
#pragma unroll
    for (int c = 0; c < kScanCols; ++c) {
      const int row = lane + 32 * i;
      s[i][c] = portion.w > 0 && row < p.dim && c < cols ? state[(size_t)row * p.vdim + c] : 0.f;
    }
  const int qk_channels = 2 * p.kv_heads * p.dim;
  float kn[kRows], qn[kRows], vn[kScanCols], gn = 0.f, bn = 0.f;  // the next token's inputs
  auto fetch = [&](int t) {
    const int64_t r = portion.y - first + t;
    const float *q_row = qk + r * qk_channels + hk * p.dim;
#pragma unroll
    for (int i = 0; i < kRows; ++i) {
      const int row = lane + 32 * i;
      qn[i] = row < p.dim ? q_row[row] : 0.f;
      kn[i] = row < p.dim ? q_row[p.kv_heads * p.dim + row] : 0.f;
    }
#pragma unroll
    for (int c = 0; c < kScanCols; ++c) vn[c] = c < cols ? ldf(v + (r * p.heads + h) * p.vdim + col0 + c) : 0.f;
    gn = log_g[r * p.heads + h];
    bn = beta[r * p.heads + h];
  };
  fetch(0);
  for (int t = 0; t < portion.z; ++t) {
    float k[kRows], q[kRows], u[kScanCols], y[kScanCols];
    const float g = expf(gn), b = bn;
#pragma unroll
    for (int i = 0; i < kRows; ++i) k[i] = kn[i], q[i] = qn[i];
#pragma unroll
    for (int c = 0; c < kScanCols; ++c) u[c] = vn[c], y[c] = 0.f;
    if (t + 1 < portion.z) fetch(t + 1);
#pragma unroll
    for (int c = 0; c < kScanCols; ++c) {
      float a = 0.f;
#pragma unroll
      for (int i = 0; i < kRows; ++i) {
        s[i][c] *= g;
        a = fmaf(s[i][c], k[i], a);
      }
      u[c] = b * (u[c] - warp_sum(a));
    }
#pragma unroll
    for (int c = 0; c < kScanCols; ++c) {
#pragma unroll
      for (int i = 0; i < kRows; ++i) {
        s[i][c] = fmaf(k[i], u[c], s[i][c]);
        y[c] = fmaf(s[i][c], q[i], y[c]);
      }
      y[c] = warp_sum(y[c]);
    }
    if (lane < cols) {
      const float o = lane == 0 ? y[0] : lane == 1 ? y[1] : lane == 2 ? y[2] : y[3];
      stf(out + ((int64_t)(portion.y - first + t) * p.heads + h) * p.vdim + col0 + lane, o);
    }
  }
#pragma unroll
  for (int i = 0; i < kRows; ++i)
#pragma unroll
    for (int c = 0; c < kScanCols; ++c) {
      const int row = lane + 32 * i;
      if (row < p.dim && c < cols) state[(size_t)row * p.vdim + c] = s[i][c];
    }
}

// ---- portions: norm and gate; the ring ----------------------------------------------------------------
// o (rows - first, heads, vdim) may be the output itself.
constexpr int kFinishWarps = 8;

// The last `taps` rows of a portion are what the next step's convolution may look back at: filed by the threads of a CTA.
template <typename T, int kVec>
__device__ __forceinline__ void file_inputs(const DeltaParams<T> &p, int64_t r) {
  const bool last = r + p.taps >= p.rows || p.row_back[r + p.taps] < p.taps;
  const int seq = p.row_seq[r];
  if (!last || bad_seq(seq, p.max_seqs, false)) return;
  const int channels = p.channels();
  T *slot = p.ring + ((size_t)seq * p.taps + p.row_pos[r] % p.taps) * channels;
  for (int c = threadIdx.x * kVec; c < channels; c += blockDim.x * kVec) {
    float in[kVec];
    load_vec<kVec>(p.proj + r * p.ld + c, in);
    store_vec<kVec>(slot + c, in);
  }
}

// Heads of 8 * kLanes elements: kLanes lanes per head, eight elements each, kDeep heads of a lane on their way at a time.
template <typename T, int kLanes>
__global__ void __launch_bounds__(kFinishWarps * 32, 4)
delta_finish_lanes_kernel(const DeltaParams<T> p, int first, const T *o, T *out) {
  constexpr int kVdim = 8 * kLanes, kAtOnce = kFinishWarps * 32 / kLanes, kDeep = 4;
  const int at = threadIdx.x % kLanes * 8;
  const uint32_t items = (uint32_t)(p.rows - first) * p.heads, i0 = blockIdx.x * (kAtOnce * kDeep);
  grid_dependency_wait();
  grid_dependency_launch();
  uint4 y[kDeep], gate[kDeep];
#pragma unroll
  for (int d = 0; d < kDeep; ++d) {
    const uint32_t i = i0 + d * kAtOnce + threadIdx.x / kLanes;
    y[d] = gate[d] = make_uint4(0, 0, 0, 0);
    if (i < items) {
      const uint32_t r = i / (uint32_t)p.heads;
      y[d] = *reinterpret_cast<const uint4 *>(o + (size_t)i * kVdim + at);
      gate[d] = *reinterpret_cast<const uint4 *>(p.proj + (int64_t)(first + r) * p.ld + p.gate_at() + (size_t)(i - r * p.heads) * kVdim + at);
    }
  }
  // the rows whose first head is among this CTA's: which of them the next step may look back at
  const int r0 = first + (int)((i0 + p.heads - 1) / p.heads), r1 = min(p.rows, first + (int)((i0 + kAtOnce * kDeep + p.heads - 1) / p.heads));
  const int mine = r0 + (int)threadIdx.x;
  const bool files = __syncthreads_or(mine < r1 && (mine + p.taps >= p.rows || p.row_back[mine + p.taps] < p.taps));
  float w[8];
  load_vec<8>(p.norm + at, w);
#pragma unroll
  for (int d = 0; d < kDeep; ++d) {
    const uint32_t i = i0 + d * kAtOnce + threadIdx.x / kLanes;
    const T *ye = reinterpret_cast<const T *>(&y[d]), *ge = reinterpret_cast<const T *>(&gate[d]);
    float v[8], sq = 0.f;
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      v[e] = ldf(ye + e);
      sq = fmaf(v[e], v[e], sq);
    }
#pragma unroll
    for (int off = kLanes / 2; off > 0; off >>= 1) sq += __shfl_xor_sync(0xffffffffu, sq, off);
    const float inv = 1.0f / sqrtf(sq / (float)kVdim + p.eps);
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      const float z = ldf(ge + e);
      v[e] = v[e] * inv * w[e] * __fdividef(z, 1.0f + __expf(-z));
    }
    if (i < items) store_vec<8>(out + (size_t)i * kVdim + at, v);
  }
  if (files)
    for (int r = r0; r < r1; ++r) file_inputs<T, 8>(p, r);
}

// Any size: a warp per head.

template <typename T, int kVec>
__global__ void __launch_bounds__(kFinishWarps * 32)
delta_finish_kernel(const DeltaParams<T> p, int first, const T *o, T *out) {
  const int lane = threadIdx.x & 31;
  const int64_t r = first + (int64_t)blockIdx.x;
  grid_dependency_wait();
  grid_dependency_launch();
  const T *x = p.proj + r * p.ld;
  for (int h = threadIdx.x >> 5; h < p.heads; h += kFinishWarps) {
    const T *src = o + ((r - first) * p.heads + h) * p.vdim;
    float y[kVec], w[kVec], gate[kVec], sq = 0.f;
    for (int i = lane * kVec; i < p.vdim; i += 32 * kVec) {
      load_vec<kVec>(src + i, y);
#pragma unroll
      for (int e = 0; e < kVec; ++e) sq = fmaf(y[e], y[e], sq);
    }
    const float inv = 1.0f / sqrtf(warp_sum(sq) / (float)p.vdim + p.eps);
    for (int i = lane * kVec; i < p.vdim; i += 32 * kVec) {
      load_vec<kVec>(src + i, y);
      load_vec<kVec>(p.norm + i, w);
      load_vec<kVec>(x + p.gate_at() + h * p.vdim + i, gate);
#pragma unroll
      for (int e = 0; e < kVec; ++e) y[e] = y[e] * inv * w[e] * silu(gate[e]);
      store_vec<kVec>(out + ((r - first) * p.heads + h) * p.vdim + i, y);
    }
  }
  file_inputs<T, kVec>(p, r);
}

bool al16(const void *p) { return (reinterpret_cast<uintptr_t>(p) & 15u) == 0; }

template <typename T>
bool quads(const DeltaParams<T> &p) {
  return p.dim % 4 == 0 && p.vdim % 4 == 0 && p.ld % 4 == 0 && al16(p.proj) && al16(p.conv) && al16(p.norm) && al16(p.ring) &&
         al16(p.state);
}

template <typename T>
int step(const DeltaParams<T> &p, void *out, cudaStream_t st) {
  const size_t smem = (size_t)(2 * p.dim + 2 * p.vdim) * sizeof(float);
  auto go = [&](auto *kernel) {
    if (smem > 32 * 1024 && cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
      return (int)AXB200_DEVICE_ERROR;
    return launch_dependent(kernel, dim3(p.rows, p.heads), dim3(kStepThreads), smem, st, p, static_cast<T *>(out));
  };
  const bool vec = quads(p);
  const size_t bulk = ((size_t)p.dim * p.vdim + 2 * p.dim + (2 + 2 * kStepWarps) * p.vdim) * sizeof(float);
  if (vec && bulk <= 220 * 1024) {
    auto *kernel = delta_step_bulk_kernel<T>;
    if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bulk) != cudaSuccess)
      return (int)AXB200_DEVICE_ERROR;
    return launch_dependent(kernel, dim3(p.rows, p.heads), dim3(kStepThreads), bulk, st, p, static_cast<T *>(out), wait_limit_ns());
  }
  if (p.dim <= 8 * 4) return vec ? go(delta_step_kernel<T, 4, 4>) : go(delta_step_kernel<T, 1, 4>);
  if (p.dim <= 8 * 8) return vec ? go(delta_step_kernel<T, 4, 8>) : go(delta_step_kernel<T, 1, 8>);
  if (p.dim <= 8 * 16) return vec ? go(delta_step_kernel<T, 4, 16>) : go(delta_step_kernel<T, 1, 16>);
  return vec ? go(delta_step_kernel<T, 4, 32>) : go(delta_step_kernel<T, 1, 32>);
}

template <typename T>
int prepare(const DeltaParams<T> &p, int first, float *qk, void *v, float *log_g, float *beta, cudaStream_t st) {
  const bool vec = quads(p) && al16(qk) && al16(v);
  const int run = vec ? 128 : 32;
  const int units = 2 * p.kv_heads + (p.heads * p.vdim + run - 1) / run + 1;
  const dim3 grid((p.rows - first + kPrepRows - 1) / kPrepRows, (units + kPrepWarps - 1) / kPrepWarps);
  auto go = [&](auto *kernel) {
    return launch_dependent(kernel, grid, dim3(kPrepWarps * 32), 0, st, p, first, qk, static_cast<T *>(v), log_g, beta);
  };
  if (!vec) return go(delta_prepare_kernel<T, 1, 8>);
  return p.dim <= 128 ? go(delta_prepare_kernel<T, 4, 1>) : go(delta_prepare_kernel<T, 4, 2>);
}

template <typename T>
int scan(const DeltaParams<T> &p, const int32_t *portions, int count, int first, const float *qk, const void *v,
         const float *log_g, const float *beta, void *out, cudaStream_t st) {
  const int cols = kScanCols * kScanWarps;
  const dim3 grid(count, p.heads, (p.vdim + cols - 1) / cols);
  auto go = [&](auto *kernel) {
    return launch_dependent(kernel, grid, dim3(kScanWarps * 32), 0, st, p, reinterpret_cast<const int4 *>(portions), first, qk,
                            static_cast<const T *>(v), log_g, beta, static_cast<T *>(out));
  };
  if (p.dim <= 32) return go(delta_scan_kernel<T, 1>);
  if (p.dim <= 64) return go(delta_scan_kernel<T, 2>);
  if (p.dim <= 128) return go(delta_scan_kernel<T, 4>);
  return go(delta_scan_kernel<T, 8>);
}

template <typename T>
int finish(const DeltaParams<T> &p, int first, const void *o, void *out, cudaStream_t st) {
  const bool vec = quads(p) && al16(o) && al16(out);
  auto lanes = [&](auto *kernel) {
    const int64_t per = kFinishWarps * 32 / (p.vdim / 8) * 4, items = (int64_t)(p.rows - first) * p.heads;
    return launch_dependent(kernel, dim3((unsigned)((items + per - 1) / per)), dim3(kFinishWarps * 32), 0, st, p, first, static_cast<const T *>(o),
                            static_cast<T *>(out));
  };
  if constexpr (sizeof(T) == 2) {
    if (vec && p.ld % 8 == 0 && p.channels() % 8 == 0 && (int64_t)(p.rows - first) * p.heads < 0x7fff0000) {
      if (p.vdim == 64) return lanes(delta_finish_lanes_kernel<T, 8>);
      if (p.vdim == 128) return lanes(delta_finish_lanes_kernel<T, 16>);
      if (p.vdim == 256) return lanes(delta_finish_lanes_kernel<T, 32>);
    }
  }
  auto *kernel = vec ? delta_finish_kernel<T, 4> : delta_finish_kernel<T, 1>;
  return launch_dependent(kernel, dim3(p.rows - first), dim3(kFinishWarps * 32), 0, st, p, first, static_cast<const T *>(o),
                          static_cast<T *>(out));
}

// The arguments all entry points share.
struct Common {
  const void *proj;
  int64_t ld;
  const int32_t *row_seq, *row_pos, *row_back;
  int rows;
  const float *conv, *a_log, *dt_bias;
  const void *norm;
  void *ring;
  float *state;
  int heads, kv_heads, dim, vdim, taps, max_seqs;
  float eps;
  int dtype;

  int check() const {
    if (dtype != AXB200_FLOAT32 && dtype != AXB200_BFLOAT16) return AXB200_UNSUPPORTED_TYPE;
    if (!proj || !row_seq || !row_pos || !conv || !a_log || !dt_bias || !norm || !ring || !state) return AXB200_INVALID_PTR;
    if (rows < 0 || heads <= 0 || heads > 65535 || kv_heads <= 0 || heads % kv_heads != 0 || dim <= 0 || dim > 256 || vdim <= 0 ||
        vdim > 4096 || taps <= 0 || max_seqs <= 0)
      return AXB200_INVALID_ARGUMENT;
    if (ld < (int64_t)2 * kv_heads * dim + (int64_t)heads * (2 * vdim + 2)) return AXB200_SHAPE_MISMATCH;
    return AXB200_OK;
  }
  template <typename F>
  int dispatch(F f) const {
    auto go = [&](auto tag) {
      using T = decltype(tag);
      return f(DeltaParams<T>{static_cast<const T *>(proj), ld, row_seq, row_pos, row_back, rows, conv, a_log, dt_bias,
                              static_cast<const T *>(norm), static_cast<T *>(ring), state, heads, kv_heads, dim, vdim, taps,
                              max_seqs, eps});
    };
    return dtype == AXB200_FLOAT32 ? go(float{}) : go(__nv_bfloat16{});
  }
};

}  // namespace
}  // namespace axb

extern "C" {

int axb200_delta_step(const void *proj, int64_t ld, const int32_t *row_seq, const int32_t *row_pos, int rows, const float *conv,
                      const float *a_log, const float *dt_bias, const void *norm, void *ring, float *state, void *out, int heads,
                      int kv_heads, int dim, int vdim, int taps, int max_seqs, float eps, int dtype, void *stream) {
  const axb::Common c{proj, ld, row_seq, row_pos, nullptr, rows, conv, a_log, dt_bias, norm, ring, state, heads, kv_heads, dim,
                      vdim, taps, max_seqs, eps, dtype};
  if (int rc = c.check()) return rc;
  if (!out) return AXB200_INVALID_PTR;
  if (rows == 0) return AXB200_OK;
  return c.dispatch([&](const auto &p) { return axb::step(p, out, static_cast<cudaStream_t>(stream)); });
}

int axb200_delta_prepare(const void *proj, int64_t ld, const int32_t *row_seq, const int32_t *row_pos, const int32_t *row_back,
                         int first, int rows, const float *conv, const float *a_log, const float *dt_bias, const void *norm,
                         void *ring, float *state, float *qk, void *v, float *log_g, float *beta, int heads, int kv_heads,
                         int dim, int vdim, int taps, int max_seqs, float eps, int dtype, void *stream) {
  const axb::Common c{proj, ld, row_seq, row_pos, row_back, rows, conv, a_log, dt_bias, norm, ring, state, heads, kv_heads, dim,
                      vdim, taps, max_seqs, eps, dtype};
  if (int rc = c.check()) return rc;
  if (!row_back || !qk || !v || !log_g || !beta) return AXB200_INVALID_PTR;
  if (first < 0 || first > rows) return AXB200_INVALID_ARGUMENT;
  if (first == rows) return AXB200_OK;
  return c.dispatch([&](const auto &p) { return axb::prepare(p, first, qk, v, log_g, beta, static_cast<cudaStream_t>(stream)); });
}

int axb200_delta_scan(const int32_t *portions, int count, int first, const float *qk, const void *v, const float *log_g,
                      const float *beta, float *state, void *out, int heads, int kv_heads, int dim, int vdim, int max_seqs,
                      int dtype, void *stream) {
  if (dtype != AXB200_FLOAT32 && dtype != AXB200_BFLOAT16) return AXB200_UNSUPPORTED_TYPE;
  if (!portions || !qk || !v || !log_g || !beta || !state || !out) return AXB200_INVALID_PTR;
  if (count < 0 || count > 0x7fffffff || first < 0 || heads <= 0 || heads > 65535 || kv_heads <= 0 || heads % kv_heads != 0 ||
      dim <= 0 || dim > 256 || vdim <= 0 || vdim > 4096 || max_seqs <= 0 || (reinterpret_cast<uintptr_t>(portions) & 15u) != 0)
    return AXB200_INVALID_ARGUMENT;
  if (count == 0) return AXB200_OK;
  axb::Common c{};
  c.state = state;
  c.heads = heads, c.kv_heads = kv_heads, c.dim = dim, c.vdim = vdim, c.max_seqs = max_seqs, c.dtype = dtype;
  return c.dispatch([&](const auto &p) {
    return axb::scan(p, portions, count, first, qk, v, log_g, beta, out, static_cast<cudaStream_t>(stream));
  });
}

int axb200_delta_finish(const void *proj, int64_t ld, const int32_t *row_seq, const int32_t *row_pos, const int32_t *row_back,
                        int first, int rows, const float *conv, const float *a_log, const float *dt_bias, const void *norm,
                        void *ring, float *state, const void *o, void *out, int heads, int kv_heads, int dim, int vdim, int taps,
                        int max_seqs, float eps, int dtype, void *stream) {
  const axb::Common c{proj, ld, row_seq, row_pos, row_back, rows, conv, a_log, dt_bias, norm, ring, state, heads, kv_heads, dim,
                      vdim, taps, max_seqs, eps, dtype};
  if (int rc = c.check()) return rc;
  if (!row_back || !o || !out) return AXB200_INVALID_PTR;
  if (first < 0 || first > rows) return AXB200_INVALID_ARGUMENT;
  if (first == rows) return AXB200_OK;
  return c.dispatch([&](const auto &p) { return axb::finish(p, first, o, out, static_cast<cudaStream_t>(stream)); });
}

}  // extern "C"
