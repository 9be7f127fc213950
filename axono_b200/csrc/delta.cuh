// What the kernels of the gated delta rule share; see delta.cu.
#pragma once

#include "vec.cuh"

namespace axb {

// One mixer's weights and sizes, and the rows of a step.  Row r of proj holds [q | k | v | gate | a | b] (kv_heads * dim
// twice, heads * vdim twice, heads twice) and is a token of sequence row_seq[r] at position row_pos[r]; row_back[r] of the
// rows directly before it are the same sequence's tokens before it.
template <typename T>
struct DeltaParams {
  const T *proj;
  int64_t ld;
  const int32_t *row_seq, *row_pos, *row_back;
  int rows;
  const float *conv;     // (taps, channels): channels [q | k | v], the current token's tap last
  const float *a_log, *dt_bias;
  const T *norm;         // (vdim)
  T *ring;               // (max_seqs, taps, channels): the projections of position p stand in slot p % taps
  float *state;          // (max_seqs, heads, dim, vdim)
  int heads, kv_heads, dim, vdim, taps, max_seqs;
  float eps;

  __host__ __device__ int channels() const { return 2 * kv_heads * dim + heads * vdim; }
  __host__ __device__ int gate_at() const { return channels(); }
  __host__ __device__ int a_at() const { return channels() + heads * vdim; }
  __host__ __device__ int b_at() const { return a_at() + heads; }
};

__device__ __forceinline__ float silu(float z) { return z / (1.0f + expf(-z)); }

// Logarithm of the decay: -exp(A) * softplus(a + bias).
__device__ __forceinline__ float log_decay(float a, float a_log, float dt_bias) {
  const float z = a + dt_bias;
  return -expf(a_log) * (fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))));
}
__device__ __forceinline__ float sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }

// The projection of kVec channels from c on, `back` tokens before row r: a row of this step, the ring, or zero before
// the sequence's start.
template <int kVec, typename T>
__device__ __forceinline__ void earlier_input(const DeltaParams<T> &p, int64_t r, int back, int c, float (&v)[kVec]) {
  const int pos = p.row_pos[r] - back;
  if (back <= p.row_back[r]) {
    load_vec<kVec>(p.proj + (r - back) * p.ld + c, v);
  } else if (pos >= 0) {
    load_vec<kVec>(p.ring + ((size_t)p.row_seq[r] * p.taps + pos % p.taps) * p.channels() + c, v);
  } else {
#pragma unroll
    for (int i = 0; i < kVec; ++i) v[i] = 0.f;
  }
}

}  // namespace axb
