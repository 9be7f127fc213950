// Loads and stores of a few consecutive elements as floats; shared by the row-wise kernels.
#pragma once

#include "common.cuh"

namespace axb {

// kVec consecutive elements: 8 (16 or 32 bytes), 4 (8 or 16 bytes), 2 (4 or 8 bytes), or one.
template <int kVec, typename T>
__device__ __forceinline__ void load_vec(const T *p, float (&v)[kVec]) {
  if constexpr (kVec == 8 && sizeof(T) == 2) {
    const uint4 raw = *reinterpret_cast<const uint4 *>(p);
    const T *e = reinterpret_cast<const T *>(&raw);
#pragma unroll
    for (int i = 0; i < 8; ++i) v[i] = ldf(e + i);
  } else if constexpr (kVec == 4 && sizeof(T) == 2) {
    const uint2 raw = *reinterpret_cast<const uint2 *>(p);
    const T *e = reinterpret_cast<const T *>(&raw);
#pragma unroll
    for (int i = 0; i < 4; ++i) v[i] = ldf(e + i);
  } else if constexpr (kVec == 4) {
    const float4 a = reinterpret_cast<const float4 *>(p)[0];
    v[0] = a.x, v[1] = a.y, v[2] = a.z, v[3] = a.w;
  } else if constexpr (kVec == 8) {
    const float4 a = reinterpret_cast<const float4 *>(p)[0], b = reinterpret_cast<const float4 *>(p)[1];
    v[0] = a.x, v[1] = a.y, v[2] = a.z, v[3] = a.w, v[4] = b.x, v[5] = b.y, v[6] = b.z, v[7] = b.w;
  } else if constexpr (kVec == 2 && sizeof(T) == 2) {
    const uint32_t raw = *reinterpret_cast<const uint32_t *>(p);
    const T *e = reinterpret_cast<const T *>(&raw);
    v[0] = ldf(e), v[1] = ldf(e + 1);
  } else if constexpr (kVec == 2) {
    const float2 a = *reinterpret_cast<const float2 *>(p);
    v[0] = a.x, v[1] = a.y;
  } else {
    v[0] = ldf(p);
  }
}
template <int kVec, typename T>
__device__ __forceinline__ void store_vec(T *p, const float (&v)[kVec]) {
  if constexpr (kVec == 8 && sizeof(T) == 2) {
    uint4 raw;
    T *e = reinterpret_cast<T *>(&raw);
#pragma unroll
    for (int i = 0; i < 8; ++i) stf(e + i, v[i]);
    *reinterpret_cast<uint4 *>(p) = raw;
  } else if constexpr (kVec == 4 && sizeof(T) == 2) {
    uint2 raw;
    T *e = reinterpret_cast<T *>(&raw);
#pragma unroll
    for (int i = 0; i < 4; ++i) stf(e + i, v[i]);
    *reinterpret_cast<uint2 *>(p) = raw;
  } else if constexpr (kVec == 4) {
    reinterpret_cast<float4 *>(p)[0] = make_float4(v[0], v[1], v[2], v[3]);
  } else if constexpr (kVec == 8) {
    reinterpret_cast<float4 *>(p)[0] = make_float4(v[0], v[1], v[2], v[3]);
    reinterpret_cast<float4 *>(p)[1] = make_float4(v[4], v[5], v[6], v[7]);
  } else if constexpr (kVec == 2 && sizeof(T) == 2) {
    uint32_t raw;
    T *e = reinterpret_cast<T *>(&raw);
    stf(e, v[0]), stf(e + 1, v[1]);
    *reinterpret_cast<uint32_t *>(p) = raw;
  } else if constexpr (kVec == 2) {
    *reinterpret_cast<float2 *>(p) = make_float2(v[0], v[1]);
  } else {
    stf(p, v[0]);
  }
}

}  // namespace axb
