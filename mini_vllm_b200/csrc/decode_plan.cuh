// The work split of a paged decode-attention step: prefix sums of 16-token-multiple tiles over the sequences, cut into one
// contiguous range per persistent CTA.  Shared by the kernels that stream a paged context (decode_attn.cu, latent_attn.cu).
#pragma once
#include "common.cuh"
#include "host_util.cuh"
#include "scan.cuh"

namespace mvb {

constexpr int kMaxCtas = 160;          // workspace is sized for this many persistent CTAs
constexpr int kPlanThreads = 256;
constexpr int kMinTilesPerCta = 2;
constexpr int kMaxPartsPerSeq = 32;   // target bound on the partials one sequence is split into

struct DecodeHeader {                  // first 32 bytes of the workspace (device memory)
  int32_t total_tiles, per_cta, num_ctas, cta_tokens, num_seqs, window_left, aligned, pad1;
};

// What a CTA needs to start streaming, written by the plan kernel so that the attention kernel
// begins with ONE 32-byte load instead of a chain of dependent ones.
struct alignas(32) CtaDesc {
  int32_t t0, t1;             // this CTA's tile range [t0, t1) (t0 >= t1: no work)
  int32_t b;                  // sequence holding tile t0
  int32_t tp0, tp1;           // that sequence's tile range
  int32_t n;                  // its context length
  int32_t per;                // tiles per CTA
  int32_t blk0;               // block id holding tile t0 (-1: read it from the block table)
};

struct DecodeLayout {                  // byte offsets inside the workspace
  size_t descs, lse, o, tile_prefix, total;       // arrival counters follow tile_prefix[num_seqs + 1]
};

static inline size_t align_up(size_t x, size_t a) { return (x + a - 1) / a * a; }

static DecodeLayout decode_layout(int max_seqs, int hq, int d) {
  DecodeLayout l;
  l.descs = sizeof(DecodeHeader);
  l.lse = align_up(l.descs + sizeof(CtaDesc) * kMaxCtas, 256);
  l.o = align_up(l.lse + sizeof(float) * kMaxCtas * 2 * hq, 256);
  l.tile_prefix = align_up(l.o + sizeof(float) * kMaxCtas * 2 * static_cast<size_t>(hq) * d, 256);
  l.total = align_up(l.tile_prefix + sizeof(int32_t) * (static_cast<size_t>(max_seqs) + 1) +
                         sizeof(int32_t) * static_cast<size_t>(max_seqs) * hq, 256);
  return l;
}

__device__ __forceinline__ int visible_start(int n, int window_left) {
  return window_left >= 0 ? max(0, n - 1 - window_left) : 0;
}

// A window with kept first tokens: a sequence's tiles are numbered without the gap between the kept ones and the window's.
// tiles left out, and the token a tile starts with
__device__ __forceinline__ int skipped_tiles(int start, int keep_first, int cta_tokens) {
  return max(0, start / cta_tokens - (keep_first + cta_tokens - 1) / cta_tokens);
}
__device__ __forceinline__ int tile_token(int tile, int skip, int keep_first, int cta_tokens) {
  return (tile < (keep_first + cta_tokens - 1) / cta_tokens ? tile : tile + skip) * cta_tokens;
}

static __global__ void __launch_bounds__(kPlanThreads) decode_plan_kernel(const int32_t* __restrict__ cache_seqlens,
                                                                   int num_seqs, int window_left, int keep_first, int cta_tokens,
                                                                   int merge_tiles,
                                                                   int num_ctas, int num_counters,
                                                                   const int32_t* __restrict__ block_table,
                                                                   int64_t table_stride, int block_size,
                                                                   DecodeHeader* hdr, CtaDesc* descs,
                                                                   int32_t* tile_prefix) {
  __shared__ int max_tiles_s, max_load_s;
  if (threadIdx.x == 0) { max_tiles_s = 0; max_load_s = 0; }
  for (int i = threadIdx.x; i < num_counters; i += kPlanThreads) tile_prefix[num_seqs + 1 + i] = 0;
  __syncthreads();
  block_exclusive_scan<kPlanThreads>(
      [&](int b) {
        const int n = cache_seqlens[b];
        if (n <= 0) return 0;
        const int tiles = (n + cta_tokens - 1) / cta_tokens - skipped_tiles(visible_start(n, window_left), keep_first, cta_tokens);
        atomicMax(&max_tiles_s, tiles);
        return tiles;
      },
      num_seqs, tile_prefix);
  const int total = tile_prefix[num_seqs];
  int per = (total + num_ctas - 1) / num_ctas;
  per = per < kMinTilesPerCta ? kMinTilesPerCta : per;
  // one CTA merges all partials of a sequence: keep that bounded (a few-sequence batch would
  // otherwise be cut into a hundred slivers whose merge costs more than the streaming)
  const int per_for_merge = (max_tiles_s + kMaxPartsPerSeq - 1) / kMaxPartsPerSeq;
  per = per < per_for_merge ? per_for_merge : per;
  auto seq_of_tile = [&](int t) -> int {   // last b with tile_prefix[b] <= t (the sequence holding tile t < total)
    int lo = 0, hi = num_seqs;
    while (hi - lo > 1) {
      const int mid = (lo + hi) >> 1;
      if (tile_prefix[mid] <= t) lo = mid; else hi = mid;
    }
    return lo;
  };
  // the aligned cut: boundary c sits on the sequence boundary nearest to c * total / num_ctas
  auto aligned_start = [&](int c) -> int {
    if (c <= 0 || total == 0) return 0;
    if (c >= num_ctas) return total;
    const int ideal = static_cast<int>(static_cast<int64_t>(c) * total / num_ctas);
    const int b = seq_of_tile(ideal);
    const int below = tile_prefix[b], above = tile_prefix[b + 1];
    return ideal - below <= above - ideal ? below : above;
  };
  for (int c = threadIdx.x; c < num_ctas; c += kPlanThreads)
    atomicMax(&max_load_s, aligned_start(c + 1) - aligned_start(c));
  __syncthreads();
  const bool aligned = total > 0 && max_load_s <= per + merge_tiles;
  if (threadIdx.x == 0) {
    hdr->total_tiles = total; hdr->per_cta = per; hdr->num_ctas = num_ctas; hdr->cta_tokens = cta_tokens;
    hdr->num_seqs = num_seqs; hdr->window_left = window_left; hdr->aligned = aligned ? 1 : 0; hdr->pad1 = 0;
  }
  for (int c = threadIdx.x; c < num_ctas; c += kPlanThreads) {
    const int64_t even0 = static_cast<int64_t>(c) * per;
    const int64_t t = aligned ? aligned_start(c) : even0;
    CtaDesc d;
    d.t0 = t < total ? static_cast<int32_t>(t) : total;
    d.t1 = aligned ? aligned_start(c + 1) : (even0 + per < total ? static_cast<int32_t>(even0 + per) : total);
    d.b = num_seqs; d.tp0 = d.tp1 = d.n = 0; d.per = per; d.blk0 = -1;
    if (d.t0 < d.t1) {
      const int lo = seq_of_tile(d.t0);
      d.b = lo; d.tp0 = tile_prefix[lo]; d.tp1 = tile_prefix[lo + 1]; d.n = cache_seqlens[lo];
      if (block_table != nullptr) {      // spare the attention kernel one dependent load before its first TMA
        const int skip = skipped_tiles(visible_start(d.n, window_left), keep_first, cta_tokens);
        const int token0 = tile_token(static_cast<int>(t) - d.tp0, skip, keep_first, cta_tokens);
        d.blk0 = block_table[lo * table_stride + token0 / block_size];
      }
    }
    descs[c] = d;
  }
}

}  // namespace mvb
