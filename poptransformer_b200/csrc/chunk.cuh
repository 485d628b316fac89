// Pieces of the kernels that work on packed sequences in tiles: asynchronous copies, ldmatrix, and where the chunks of a recurrence live.
#pragma once
#include "elem.cuh"
#include "tile_math.cuh"

namespace pt {

__device__ __forceinline__ void ldsm4t(uint32_t addr, uint32_t &r0, uint32_t &r1, uint32_t &r2, uint32_t &r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void ldsm4(uint32_t addr, uint32_t &r0, uint32_t &r1, uint32_t &r2, uint32_t &r3) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
// 16-byte asynchronous copy; zeros instead of the source when !in (the source address is then not read).
__device__ __forceinline__ void cp16(void *dst, const void *src, bool in) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(smem_addr(dst)), "l"(src), "r"(in ? 16 : 0) : "memory");
}

// Recurrences in chunks of 64 tokens: chunk ci of sequence s uses slot cu[s] / 64 + s + ci of the scratch (distinct, below
// n_tok / 64 + n_seq).
constexpr int CHUNK = 64, CHUNK_THREADS = 256;
__device__ __forceinline__ int chunk_slot(const int *cu, int s) { return cu[s] / CHUNK + s; }
// Sequence and first token (within it) of a scratch slot; false for a slot that no chunk uses.
__device__ __forceinline__ bool chunk_of_slot(const int *cu, int n_seq, int slot, int &s, int &t0) {
  int lo = 0, hi = n_seq - 1;
  while (lo < hi) {
    const int mid = (lo + hi + 1) / 2;
    if (chunk_slot(cu, mid) <= slot) lo = mid;
    else hi = mid - 1;
  }
  s = lo;
  t0 = (slot - chunk_slot(cu, lo)) * CHUNK;
  return t0 < cu[lo + 1] - cu[lo];
}

}  // namespace pt
