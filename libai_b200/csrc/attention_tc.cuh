// Shared pieces of the tcgen05 prompt-attention kernels: bounded mbarrier waits and the named barrier of a TMEM lane quadrant.
#pragma once
#include "common.cuh"

#include <type_traits>

namespace lb {

// false when the wait ran out (or another wait of the CTA had): *stop is set, and every later wait returns at once
constexpr uint32_t TC_WAIT_LIMIT = 1u << 22;
LB_DEVICE bool tc_wait(uint64_t* bar, uint32_t parity, volatile int* stop) {
  if (*stop) return false;
  for (uint32_t i = 0; i < TC_WAIT_LIMIT; ++i) {
    if (mbar_try_wait(bar, parity)) return true;
    if ((i & 1023u) == 1023u && *stop) return false;
  }
  *stop = 1;
  return false;
}
LB_DEVICE void tc_pair_sync(int quad) {       // the two warps that own the same TMEM lane quadrant
  if (quad == 0) asm volatile("bar.sync 1, 64;\n" ::: "memory");
  else if (quad == 1) asm volatile("bar.sync 2, 64;\n" ::: "memory");
  else if (quad == 2) asm volatile("bar.sync 3, 64;\n" ::: "memory");
  else asm volatile("bar.sync 4, 64;\n" ::: "memory");
}

}  // namespace lb
