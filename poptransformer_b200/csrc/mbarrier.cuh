// Shared-memory barriers and bulk copies that arrive on them.  Every wait is bounded.
#pragma once
#include "common.cuh"

namespace pt {

constexpr int WAIT_LIMIT = 1 << 22;
#ifndef PT_TC_HINT
#define PT_TC_HINT 1000   // suspend-time hint (ns) of the barrier waits; negative: plain polling with test_wait
#endif

__device__ __forceinline__ void mbar_init(uint32_t bar, int count) { asm volatile("mbarrier.init.shared::cta.b64 [%0], %1;" ::"r"(bar), "r"(count)); }
__device__ __forceinline__ void mbar_expect_tx(uint32_t bar, uint32_t bytes) {
  asm volatile("mbarrier.arrive.expect_tx.shared::cta.b64 _, [%0], %1;" ::"r"(bar), "r"(bytes) : "memory");
}
__device__ __forceinline__ void mbar_arrive(uint32_t bar) { asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(bar) : "memory"); }
// Bounded wait; gives up at once when the CTA has already recorded a failure.
__device__ __forceinline__ bool mbar_wait(uint32_t bar, uint32_t parity, volatile int *abort_flag) {
  for (int it = 0; it < WAIT_LIMIT; ++it) {
    uint32_t ok;
#if PT_TC_HINT < 0
    asm volatile("{\n\t.reg .pred p;\n\tmbarrier.test_wait.parity.shared::cta.b64 p, [%1], %2;\n\tselp.u32 %0, 1, 0, p;\n\t}"
                 : "=r"(ok)
                 : "r"(bar), "r"(parity)
                 : "memory");
#else
    asm volatile("{\n\t.reg .pred p;\n\tmbarrier.try_wait.parity.shared::cta.b64 p, [%1], %2, %3;\n\tselp.u32 %0, 1, 0, p;\n\t}"
                 : "=r"(ok)
                 : "r"(bar), "r"(parity), "r"((uint32_t)PT_TC_HINT)
                 : "memory");
#endif
    if (ok) return true;
    if (*abort_flag) return false;
  }
  return false;
}
// The same without a way to give up early: for what is still in flight when a block ends after a failure.
__device__ __forceinline__ void mbar_wait_all(uint32_t bar, uint32_t parity) {
  volatile int never = 0;
  mbar_wait(bar, parity, &never);
}
__device__ __forceinline__ void bulk_g2s(uint32_t dst, const void *src, uint32_t bytes, uint32_t bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(dst), "l"(src), "r"(bytes), "r"(bar)
               : "memory");
}

}  // namespace pt
