#include "tcgen05.cuh"
extern "C" {
int axb200_latent_prefill_supported(int, int, int, int, int) { return 0; }
int axb200_latent_prefill(const void *, int64_t, const void *, const void *, const void *, int64_t, void *, int, int64_t, int,
                          int, int, int, float, int, void *) { return AXB200_UNSUPPORTED_TYPE; }
}
