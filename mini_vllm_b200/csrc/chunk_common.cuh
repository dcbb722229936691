// What the recurrent mixers share: sums over a warp, asynchronous copies, chunks of 16 tokens, and fp32 values as bf16 pairs
// (high part + what the rounding left over) for tensor-core products with 16 significant bits per factor.
#pragma once
#include "dtype.cuh"

namespace mvb {

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
  for (int off = 16; off > 0; off >>= 1) v += __shfl_xor_sync(0xffffffffu, v, off);
  return v;
}

__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// one thread: `bytes` (a multiple of 16, both sides 16-byte aligned) into shared memory, counted on an mbarrier
__device__ __forceinline__ void bulk_copy(uint32_t dst, const void* src, uint32_t bytes, uint32_t bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
               ::"r"(dst), "l"(src), "r"(bytes), "r"(bar) : "memory");
}

constexpr int kChunk = 16;

// sequence s owns chunk slots chunk_base(s) .. + ceil(n / 16): never overlapping, no prefix sum needed
__host__ __device__ __forceinline__ int chunk_base(int row, int s) { return row / kChunk + s; }

__device__ __forceinline__ float bf16_round(float x) { return __bfloat162float(__float2bfloat16_rn(x)); }
// (x, y) as packed bf16: the rounded values, and what the rounding left over
__device__ __forceinline__ void split_pair(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16(x, y);
  lo = pack_bf16(x - bf16_lo(hi), y - bf16_hi(hi));
}

// d += a * b with a, b given as high and low parts
struct Split { uint32_t hi[4], lo[4]; };
__device__ __forceinline__ void split_tile(const float (&x)[4], const float (&y)[4], Split& s) {   // two adjacent 8-column tiles
  split_pair(x[0], x[1], s.hi[0], s.lo[0]); split_pair(x[2], x[3], s.hi[1], s.lo[1]);
  split_pair(y[0], y[1], s.hi[2], s.lo[2]); split_pair(y[2], y[3], s.hi[3], s.lo[3]);
}

// the instance that holds a key size
static inline int chunk_ks(int dim) {
  const int need = (dim + 15) / 16;
  for (int ks : {1, 2, 3, 4, 6, 8, 12, 16})
    if (need <= ks) return ks;
  return 0;
}

}  // namespace mvb
