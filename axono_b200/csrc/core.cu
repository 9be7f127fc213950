// What every part of the library shares on the host side: the readers of the device error words, the limit
// of the bounded waits, the version string.
#include <atomic>

#include "common.cuh"

namespace axb {
namespace {
constexpr int kMaxErrorReaders = 32, kMaxTimeoutHooks = 8;
ErrorReader g_error_readers[kMaxErrorReaders];
int g_num_error_readers = 0;
TimeoutHook g_timeout_hooks[kMaxTimeoutHooks];
int g_num_timeout_hooks = 0;
std::atomic<unsigned long long> g_wait_limit_ns{kWaitNanos};
}  // namespace

void register_error_reader(ErrorReader fn) {
  if (g_num_error_readers < kMaxErrorReaders) g_error_readers[g_num_error_readers++] = fn;
}
void register_timeout_hook(TimeoutHook fn) {
  if (g_num_timeout_hooks < kMaxTimeoutHooks) g_timeout_hooks[g_num_timeout_hooks++] = fn;
}
unsigned long long wait_limit_ns() { return g_wait_limit_ns.load(); }
}  // namespace axb

extern "C" {

const char *axb200_version(void) { return "axono_b200 0.3 (sm_100a)"; }

int axb200_set_wait_limit_ns(uint64_t ns) {
  if (ns == 0) return AXB200_INVALID_ARGUMENT;
  axb::g_wait_limit_ns = ns;
  return AXB200_OK;
}

unsigned int axb200_last_error(void) {
  if (cudaDeviceSynchronize() != cudaSuccess) return 0x80000000u;
  unsigned int word = 0;
  for (int i = 0; i < axb::g_num_error_readers; ++i) word |= axb::g_error_readers[i]();
  if (word & AXB200_ERR_WAIT_TIMEOUT) {
    // a CTA that gave up never counted itself in: device-side counters go back to their rest values
    for (int i = 0; i < axb::g_num_timeout_hooks; ++i) axb::g_timeout_hooks[i]();
    cudaDeviceSynchronize();
  }
  return word;
}

}  // extern "C"
