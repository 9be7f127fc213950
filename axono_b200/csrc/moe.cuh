// What the expert products of moe.cu and moe_umma.cu share.
#pragma once

#include "tcgen05.cuh"

namespace axb {

// Gated activation with clamps: g = min(gate, limit), u = clamp(up, -limit, limit),
// g * sigmoid(slope * g) * (u + offset).
struct ClampedGate {
  float limit, slope, offset;
};

// kExact: the accurate exponential and division (fp32 storage); otherwise their fast forms, whose error is far
// below a bf16 rounding.
template <bool kExact>
__device__ __forceinline__ float clamped_gate(float gate, float up, const ClampedGate &c) {
  const float g = fminf(gate, c.limit), u = fminf(fmaxf(up, -c.limit), c.limit);
  if constexpr (kExact) return g / (1.0f + expf(-c.slope * g)) * (u + c.offset);
  return __fdividef(g, 1.0f + __expf(-c.slope * g)) * (u + c.offset);
}

// One grouped product y[r] = w[expert of r] . x[r] (in -> out; for the gate/up form w holds 2 * out rows per
// expert and the activation joins the halves).  tiles: (expert, first row, rows, -), *n_tiles of them; null:
// one expert over all rows.
struct MoeProduct {
  const void *x, *w;
  void *y;
  const int4 *tiles;
  const int32_t *n_tiles;
  int rows, experts, in, out, tile_rows, max_tiles;
  ClampedGate act;
  unsigned long long wait_ns;
};

__device__ __forceinline__ bool moe_tile(const MoeProduct &p, int t, int tile_rows, int4 &tile) {
  if (p.tiles) {
    if (t >= *p.n_tiles) return false;
    tile = p.tiles[t];
    return true;
  }
  const int r0 = t * p.tile_rows;
  if (r0 >= p.rows) return false;
  tile = make_int4(0, r0, min(p.tile_rows, p.rows - r0), 0);
  return true;
}

// tcgen05 form (moe_umma.cu)
bool moe_umma_takes(int width, int ff);
int moe_umma_tile_rows(int64_t rows, int experts);
bool moe_umma_supported(const MoeProduct &p, bool gate_up);
// Both in one launch; shared.rows == 0: no shared expert.
int moe_umma(const MoeProduct &routed, const MoeProduct &shared, bool gate_up, cudaStream_t st);

}  // namespace axb
