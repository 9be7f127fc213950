#include "moe.cuh"
namespace axb {
bool moe_umma_takes(int, int) { return false; }
int moe_umma_tile_rows(int64_t, int) { return 32; }
bool moe_umma_supported(const MoeProduct &, bool) { return false; }
int moe_umma(const MoeProduct &, bool, cudaStream_t) { return AXB200_INTERNAL_ERROR; }
}  // namespace axb
