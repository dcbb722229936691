// Mixture of experts: each token goes through the `top` experts that score highest, small gated feed-forwards with weights of their own.
//
//   route    z = router logits (fp32): a warp per token picks the largest scores, keeps them as weights (times a factor), and counts.  A
//            score is sigmoid(z), or the softmax of z over all outputs; a correction per output may be added for the choice alone.  The
//            outputs behind the experts are identity experts: they give a token its own row back, so their weights are only added up.
//            Counts meet in shared memory first, one atomic per block and expert after that; the block that finishes last turns them
//            into the sorted layout (first row of every expert) and into row tiles (expert, first row, rows) of at most `block_rows`.
//   gather   rows of h in the sorted order
//   gemm 1   [gate; up] of an expert times its rows, with the gated unit in the epilogue and the weight on the expert's input, or on its
//            output: y = g sigmoid(alpha g) (u + offset), g = min(w gate, limit), u = clamp(w up, -limit, limit), or w times that with
//            the plain gate and up
//   gemm 2   down projection.  The sum over a token's experts is taken by whoever reads the rows (residual_ops.cu), in a fixed order.
//
// The sizes of the groups never reach the host, so a step with experts is one CUDA graph whatever the tokens are.
//
// moe_gemm_kernel (bf16, tcgen05): the expert's weights are the 128 rows of a tile (A), its tokens the columns (B) - so a few tokens
// per expert cost a narrow tile and not a mostly empty one - and a tile has two such row blocks over the same tokens: gate and up, or two
// blocks of the down projection.  Work items are (row tile, weight block), persistent CTAs take them in turn:
//   producer warp    TMA (128-byte swizzle): two weight blocks [128 x 64] and the tokens [BN x 64] per K block, ring of 4 to 6 stages
//   MMA warp         one thread issues both products, M = 128, N = BN, fp32 accumulators in tensor memory, two accumulator stages
//   epilogue warps   eight, a thread per weight row and half of the tokens; a warp stores 32 neighbouring columns of an output row
// Rows past a tile's end belong to another expert (or to nobody) and only reach columns that are not stored.  Every wait is bounded.
//
// Roofline: tensor-bound for hundreds of rows per expert, HBM-bound on the weights for a few.
#include "dtype.cuh"
#include "host_util.cuh"
#include "mini_vllm_b200.h"
#include "scan.cuh"

#include <type_traits>

namespace mvb {

// ---- routing ----------------------------------------------------------------------------------------------------
constexpr int kRouteThreads = 256;
constexpr int kMaxExperts = 1024;

struct RouteParams {
  const float* logits; int64_t logits_stride;
  int tokens, experts, top, block_rows, max_tiles;
  int32_t* counters;            // [experts + 1], zero between calls: rows per expert, blocks finished
  int32_t* ids;                 // [tokens, top]
  float* weights;               // [tokens, top]
  int32_t* ranks;               // [tokens, top]: the row's number among its expert's
  int32_t* offsets;             // [experts + 1]: first sorted row of an expert
  int32_t* tile_offsets;        // [experts + 1]: first tile of an expert; the last entry is the number of tiles
  int4* tiles;                  // [max_tiles] (expert, first row, rows, 0)
  int outputs;                  // router outputs: experts + identity experts
  int softmax;
  const float* correction;      // [outputs] or nullptr
  float scale;                  // factor of the weights
  float* identity;              // [tokens]: sum of a token's identity weights; nullptr: there are none
};

template <int EPL>              // router outputs per lane
__global__ void __launch_bounds__(kRouteThreads) moe_route_kernel(const RouteParams p) {
  __shared__ int local[kMaxExperts];
  __shared__ int is_last;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, warps = kRouteThreads / 32;
  for (int e = tid; e < p.experts; e += kRouteThreads) local[e] = 0;
  __syncthreads();
  for (int t = blockIdx.x * warps + warp; t < p.tokens; t += gridDim.x * warps) {
    const float* row = p.logits + t * p.logits_stride;
    float z[EPL], own = 0.f;                                 // z: what is compared
#pragma unroll
    for (int i = 0; i < EPL; ++i) z[i] = i * 32 + lane < p.outputs ? row[i * 32 + lane] : -INFINITY;
    float top_z = 0.f, inv = 1.f;                            // softmax: e^(z - top_z) inv
    if (p.softmax) {
      top_z = z[0];
#pragma unroll
      for (int i = 1; i < EPL; ++i) top_z = fmaxf(top_z, z[i]);
#pragma unroll
      for (int off = 16; off > 0; off >>= 1) top_z = fmaxf(top_z, __shfl_xor_sync(0xffffffffu, top_z, off));
      float sum = 0.f;
#pragma unroll
      for (int i = 0; i < EPL; ++i) sum += expf(z[i] - top_z);
#pragma unroll
      for (int off = 16; off > 0; off >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, off);
      inv = 1.f / sum;
    }
    auto score = [&](float x) { return p.softmax ? expf(x - top_z) * inv : sigmoid_f(x); };
    if (p.correction != nullptr) {                           // (without one the logits' order is the scores')
#pragma unroll
      for (int i = 0; i < EPL; ++i)
        if (i * 32 + lane < p.outputs) z[i] = score(z[i]) + p.correction[i * 32 + lane];
    }
    uint32_t taken = 0;
    for (int k = 0; k < p.top; ++k) {
      float best = -INFINITY;
      int who = 0x7fffffff;
#pragma unroll
      for (int i = 0; i < EPL; ++i) {
        const int e = i * 32 + lane;
        if (e < p.outputs && !((taken >> i) & 1u) && (who == 0x7fffffff || z[i] > best)) { best = z[i]; who = e; }
      }
#pragma unroll
      for (int off = 16; off > 0; off >>= 1) {
        const float b = __shfl_xor_sync(0xffffffffu, best, off);
        const int w = __shfl_xor_sync(0xffffffffu, who, off);
        if (w != 0x7fffffff && (who == 0x7fffffff || b > best || (b == best && w < who))) { best = b; who = w; }
      }
      if ((who & 31) == lane) taken |= 1u << (who >> 5);
      if (lane == 0) {
        const int64_t at = static_cast<int64_t>(t) * p.top + k;
        const float w = score(row[who]) * p.scale;
        p.ids[at] = who;
        p.weights[at] = w;
        if (who < p.experts) p.ranks[at] = atomicAdd(&local[who], 1);
        else own += w;
      }
    }
    if (p.identity != nullptr && lane == 0) p.identity[t] = own;
  }
  __syncthreads();
  for (int e = tid; e < p.experts; e += kRouteThreads)
    if (local[e] > 0) local[e] = atomicAdd(p.counters + e, local[e]);
  __syncthreads();
  for (int t = blockIdx.x * warps + warp; t < p.tokens; t += gridDim.x * warps)
    for (int k = lane; k < p.top; k += 32) {
      const int64_t at = static_cast<int64_t>(t) * p.top + k;
      const int e = p.ids[at];
      p.ranks[at] = e < p.experts ? p.ranks[at] + local[e] : -1;
    }
  __threadfence();
  __syncthreads();
  if (tid == 0) is_last = atomicAdd(p.counters + p.experts, 1) == static_cast<int>(gridDim.x) - 1;
  __syncthreads();
  if (!is_last) return;
  __threadfence();
  auto count = [&](int e) { return *reinterpret_cast<volatile int32_t*>(p.counters + e); };
  block_exclusive_scan<kRouteThreads>(count, p.experts, p.offsets);
  block_exclusive_scan<kRouteThreads>([&](int e) { return (count(e) + p.block_rows - 1) / p.block_rows; }, p.experts, p.tile_offsets);
  __syncthreads();
  for (int e = tid; e < p.experts; e += kRouteThreads) {
    const int n = count(e), first = p.tile_offsets[e], row0 = p.offsets[e];
    for (int i = 0; i * p.block_rows < n && first + i < p.max_tiles; ++i)
      p.tiles[first + i] = make_int4(e, row0 + i * p.block_rows, min(p.block_rows, n - i * p.block_rows), 0);
    p.counters[e] = 0;                                       // ready for the next call
  }
  if (tid == 0) p.counters[p.experts] = 0;
}

// A warp per token and part of its row: read once, written to every expert's place.
constexpr int kGatherPart = 128;                             // 16-byte vectors of a row that a warp takes

template <class T>
__global__ void __launch_bounds__(256) moe_gather_kernel(const T* __restrict__ h, int64_t h_stride, const int32_t* __restrict__ ids,
                                                         const float* __restrict__ weights, const int32_t* __restrict__ ranks,
                                                         const int32_t* __restrict__ offsets, T* __restrict__ out, int64_t out_stride,
                                                         int32_t* __restrict__ slots, float* __restrict__ row_weights, int tokens, int top,
                                                         int width, int parts, int vec) {
  const int w = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31, t = w / parts, part = w % parts;
  if (t >= tokens) return;
  const int64_t at = static_cast<int64_t>(t) * top;
  constexpr int V = kVec<T>, N = kGatherPart / 32;
  const T* src = h + t * h_stride;
  const int first = part * kGatherPart, last = min(first + kGatherPart, width / V);
  uint4 row[N];
  if (vec) {
#pragma unroll
    for (int i = 0; i < N; ++i)
      if (first + i * 32 + lane < last) row[i] = reinterpret_cast<const uint4*>(src)[first + i * 32 + lane];
  }
  for (int j0 = 0; j0 < top; j0 += 32) {
    const int n = min(32, top - j0);
    const int rank = lane < n ? ranks[at + j0 + lane] : -1, slot = rank < 0 ? -1 : offsets[ids[at + j0 + lane]] + rank;
    if (part == 0 && lane < n) {
      slots[at + j0 + lane] = slot;
      if (slot >= 0) row_weights[slot] = weights[at + j0 + lane];
    }
    for (int j = 0; j < n; ++j) {
      const int to = __shfl_sync(0xffffffffu, slot, j);
      if (to < 0) continue;                                  // an identity expert
      T* dst = out + static_cast<int64_t>(to) * out_stride;
      if (vec) {
#pragma unroll
        for (int i = 0; i < N; ++i)
          if (first + i * 32 + lane < last) reinterpret_cast<uint4*>(dst)[first + i * 32 + lane] = row[i];
      } else {
        for (int i = lane; i < width; i += 32) dst[i] = src[i];
      }
    }
  }
}

// ---- grouped products --------------------------------------------------------------------------------------------
struct GroupParams {
  const int32_t* num_tiles;
  const int4* tiles;
  int max_tiles;
  const float* row_weights;     // [sorted rows] or nullptr (gated form)
  bool weigh_output;
  void* out; int64_t out_stride;
  int m, blocks, k;             // rows of a weight block, items per row tile, inner size
  float limit, neg_alpha_log2e, offset;
  const float* x32; int64_t x_stride; const float* w32;      // fp32 form
  int* dev_status;
};

__device__ __forceinline__ float gated_unit(float gate, float up, float w, const GroupParams& p) {
  const float in = p.weigh_output ? 1.f : w, g = fminf(gate * in, p.limit), u = fminf(fmaxf(up * in, -p.limit), p.limit);
  const float y = g * fast_rcp(1.f + fast_exp2(p.neg_alpha_log2e * g)) * (u + p.offset);      // g -> -inf: 0
  return p.weigh_output ? y * w : y;
}

constexpr int kMoeThreads = 10 * 32;                          // producer, MMA, eight epilogue warps
constexpr int kMoeBlockBytes = 128 * 128;                     // 128 weight rows x 64 columns

template <int BN>
struct MoeCfg {
  static constexpr int TOK_BYTES = BN * 128, STAGE = 2 * kMoeBlockBytes + TOK_BYTES;
  static constexpr int FIT = (226 * 1024 - 1024 - 256) / STAGE, STAGES = FIT > 6 ? 6 : FIT;
  static constexpr int SMEM = STAGES * STAGE + 1024 /*align*/ + 256 /*barriers*/;
  static constexpr int TMEM_COLS = 4 * BN;                    // two blocks, two accumulator stages
  static constexpr int FULL = 0, EMPTY = STAGES, ACC_FULL = 2 * STAGES, ACC_EMPTY = 2 * STAGES + 2, COUNT = 2 * STAGES + 4;
};

template <int BN, bool GATED>
__global__ void __launch_bounds__(kMoeThreads, 1)
moe_gemm_kernel(const __grid_constant__ CUtensorMap w_map, const __grid_constant__ CUtensorMap x_map, const GroupParams p) {
  using C = MoeCfg<BN>;
  constexpr uint32_t IDESC = umma_idesc_bf16(128, BN, false, false);
  extern __shared__ uint8_t smem_raw[];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const uint32_t base = (smem_u32(smem_raw) + 1023u) & ~1023u;
  uint8_t* base_ptr = smem_raw + (base - smem_u32(smem_raw));
  uint64_t* bars = reinterpret_cast<uint64_t*>(base_ptr + C::STAGES * C::STAGE);
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + C::COUNT);
  volatile uint32_t* fail_flag = tmem_slot + 1;
  const int num_items = min(*p.num_tiles, p.max_tiles) * p.blocks;
  if (static_cast<int>(blockIdx.x) >= num_items) return;      // CTA-uniform

  if (tid == 0) {
    for (int i = 0; i < C::COUNT; ++i) mbar_init(&bars[i], i >= C::ACC_EMPTY ? 8u : 1u);
    *fail_flag = 0;
    fence_mbar_init();
  }
  if (warp == 1) {
    tmem_alloc(tmem_slot, C::TMEM_COLS);
    tmem_relinquish();
  }
  tc_fence_before();
  __syncthreads();
  tc_fence_after();
  const uint32_t tmem = *tmem_slot;
  auto wait = [&](int slot, uint32_t parity, int where) -> bool {
    if (mbar_try_wait(&bars[slot], parity)) return true;
    return mbar_wait_or_fail(&bars[slot], parity, fail_flag, p.dev_status, where);
  };
  const int kblocks = (p.k + 63) / 64;

  if (warp == 0) {
    // ============================ producer ==========================================================
    if (lane == 0) {
      tma_prefetch_desc(&w_map);
      tma_prefetch_desc(&x_map);
      uint32_t g = 0;
      bool ok = true;
      auto load = [&](uint32_t dst, const CUtensorMap* map, uint64_t* bar, int x, int y, int z) {
        asm volatile(
            "cp.async.bulk.tensor.3d.shared::cta.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4, %5}], [%2];"
            ::"r"(dst), "l"(reinterpret_cast<uint64_t>(map)), "r"(smem_u32(bar)), "r"(x), "r"(y), "r"(z) : "memory");
      };
      for (int item = blockIdx.x; item < num_items && ok; item += gridDim.x) {
        const int4 tile = p.tiles[item / p.blocks];
        const int mb = item % p.blocks;
        for (int kb = 0; kb < kblocks && ok; ++kb, ++g) {
          const int st = g % C::STAGES;
          if (g >= C::STAGES) ok = wait(C::EMPTY + st, ((g / C::STAGES) - 1) & 1, 100);
          if (!ok) break;
          const uint32_t dst = base + st * C::STAGE;
          uint64_t* bar = &bars[C::FULL + st];
          mbar_arrive_expect_tx(bar, C::STAGE);
          if (GATED) {                                        // weights viewed as [2 experts, m, k]: gate, then up
            load(dst, &w_map, bar, kb * 64, mb * 128, 2 * tile.x);
            load(dst + kMoeBlockBytes, &w_map, bar, kb * 64, mb * 128, 2 * tile.x + 1);
          } else {
            load(dst, &w_map, bar, kb * 64, mb * 256, tile.x);
            load(dst + kMoeBlockBytes, &w_map, bar, kb * 64, mb * 256 + 128, tile.x);
          }
          load(dst + 2 * kMoeBlockBytes, &x_map, bar, kb * 64, tile.y, 0);
        }
      }
      if (!ok) {                                              // nothing may still be writing this CTA's shared memory when it ends
        for (uint32_t back = 1; back <= C::STAGES && back <= g; ++back)
          mbar_wait(&bars[C::FULL + ((g - back) % C::STAGES)], ((g - back) / C::STAGES) & 1);
      }
    }
  } else if (warp == 1) {
    // ============================ MMA issuer ========================================================
    if (lane == 0) {
      uint32_t g = 0, n = 0;
      bool ok = true;
      for (int item = blockIdx.x; item < num_items && ok; item += gridDim.x, ++n) {
        const uint32_t acc = n & 1;
        if (n >= 2) ok = wait(C::ACC_EMPTY + acc, ((n >> 1) - 1) & 1, 200);
        if (!ok) break;
        tc_fence_after();
        const uint32_t d = tmem + acc * 2 * BN;
        for (int kb = 0; kb < kblocks && ok; ++kb, ++g) {
          const int st = g % C::STAGES;
          ok = wait(C::FULL + st, (g / C::STAGES) & 1, 210);
          if (!ok) break;
          tc_fence_after();
          const uint64_t a0 = umma_desc_sw128(base + st * C::STAGE, 16, 1024);
          const uint64_t a1 = umma_desc_sw128(base + st * C::STAGE + kMoeBlockBytes, 16, 1024);
          const uint64_t b = umma_desc_sw128(base + st * C::STAGE + 2 * kMoeBlockBytes, 16, 1024);
#pragma unroll
          for (int ks = 0; ks < 4; ++ks) {
            const uint32_t o = (ks * 32) >> 4, more = (kb > 0 || ks > 0) ? 1u : 0u;
            umma_bf16_ss(d, a0 + o, b + o, IDESC, more);
            umma_bf16_ss(d + BN, a1 + o, b + o, IDESC, more);
          }
          umma_commit(&bars[C::EMPTY + st]);
        }
        if (ok) umma_commit(&bars[C::ACC_FULL + acc]);
      }
    }
    __syncwarp();
  } else {
    // ============================ epilogue ============================================================
    const int quad = warp & 3, half = (warp - 2) >> 2;        // a warp reads the 32 tensor-memory lanes of its rank mod 4
    const uint32_t lane_addr = tmem + (static_cast<uint32_t>(quad * 32) << 16);
    __nv_bfloat16* out = static_cast<__nv_bfloat16*>(p.out);
    bool ok = true;
    uint32_t n = 0;
    for (int item = blockIdx.x; item < num_items && ok; item += gridDim.x, ++n) {
      const int4 tile = p.tiles[item / p.blocks];
      const int m0 = (item % p.blocks) * (GATED ? 128 : 256) + quad * 32 + lane;
      const uint32_t acc = n & 1;
      ok = wait(C::ACC_FULL + acc, (n >> 1) & 1, 300);
      if (!ok) break;
      tc_fence_after();
#pragma unroll 1
      for (int c = half * (BN / 2); c < (half + 1) * (BN / 2) && c < tile.z; c += 16) {
        uint32_t r0[16], r1[16];
        tmem_ld_32x16(lane_addr + acc * 2 * BN + c, r0);
        tmem_ld_32x16(lane_addr + acc * 2 * BN + BN + c, r1);
        float w = 1.f;
        if (GATED && p.row_weights != nullptr && lane < 16 && c + lane < tile.z) w = p.row_weights[tile.y + c + lane];
        tmem_wait_ld();
#pragma unroll
        for (int i = 0; i < 16; ++i) {
          const float a = __uint_as_float(r0[i]), b = __uint_as_float(r1[i]);
          __nv_bfloat16* o = out + static_cast<int64_t>(tile.y + c + i) * p.out_stride + m0;
          if constexpr (GATED) {
            const float y = gated_unit(a, b, __shfl_sync(0xffffffffu, w, i), p);
            if (c + i < tile.z && m0 < p.m) *o = __float2bfloat16_rn(y);
          } else {
            if (c + i < tile.z && m0 < p.m) *o = __float2bfloat16_rn(a);
            if (c + i < tile.z && m0 + 128 < p.m) o[128] = __float2bfloat16_rn(b);
          }
        }
      }
      tc_fence_before();
      __syncwarp();
      if (lane == 0) mbar_arrive(&bars[C::ACC_EMPTY + acc]);
    }
  }
  tc_fence_before();
  __syncthreads();
  if (warp == 1) tmem_dealloc(tmem, C::TMEM_COLS);
}

// fp32: 64 rows x 64 columns per block on the fp32 pipe
template <bool GATED>
__global__ void __launch_bounds__(256) moe_gemm_f32_kernel(const GroupParams p) {
  __shared__ float xs[16][68], ws[GATED ? 2 : 1][16][68];
  if (static_cast<int>(blockIdx.y) >= min(*p.num_tiles, p.max_tiles)) return;
  const int4 tile = p.tiles[blockIdx.y];
  const int m0 = blockIdx.x * 64, tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  float acc[GATED ? 2 : 1][4][4] = {};
  for (int k0 = 0; k0 < p.k; k0 += 16) {
    for (int i = threadIdx.x; i < 64 * 16; i += 256) {
      const int r = i >> 4, c = i & 15;
      xs[c][r] = r < tile.z && k0 + c < p.k ? p.x32[static_cast<int64_t>(tile.y + r) * p.x_stride + k0 + c] : 0.f;
#pragma unroll
      for (int g = 0; g < (GATED ? 2 : 1); ++g) {
        const int64_t block = GATED ? 2 * static_cast<int64_t>(tile.x) + g : tile.x;
        ws[g][c][r] = m0 + r < p.m && k0 + c < p.k ? p.w32[(block * p.m + m0 + r) * p.k + k0 + c] : 0.f;
      }
    }
    __syncthreads();
#pragma unroll
    for (int c = 0; c < 16; ++c) {
      float a[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) a[i] = xs[c][ty * 4 + i];
#pragma unroll
      for (int g = 0; g < (GATED ? 2 : 1); ++g)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float b = ws[g][c][tx + 16 * j];
#pragma unroll
          for (int i = 0; i < 4; ++i) acc[g][i][j] = fmaf(a[i], b, acc[g][i][j]);
        }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int r = ty * 4 + i;
    if (r >= tile.z) continue;
    const float w = GATED && p.row_weights != nullptr ? p.row_weights[tile.y + r] : 1.f;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int m = m0 + tx + 16 * j;
      if (m >= p.m) continue;
      float y = acc[0][i][j];
      if constexpr (GATED) y = gated_unit(y, acc[1][i][j], w, p);
      static_cast<float*>(p.out)[static_cast<int64_t>(tile.y + r) * p.out_stride + m] = y;
    }
  }
}

// [z, rows, k] bf16, k innermost; box = 64 columns x box_rows rows, 128-byte swizzle; what lies outside reads as zeros
static int make_group_map(CUtensorMap* map, const void* base, int64_t k, int64_t rows, int64_t z, int64_t row_stride, int box_rows) {
  EncodeTiledFn fn = encode_tiled_fn();
  if (fn == nullptr) return kNoDriverEntry;
  if (!is_aligned(base, 16) || row_stride % 8 != 0) return kMisaligned;
  cuuint64_t dims[3] = {static_cast<cuuint64_t>(k), static_cast<cuuint64_t>(rows), static_cast<cuuint64_t>(z)};
  cuuint64_t strides[2] = {static_cast<cuuint64_t>(row_stride) * 2, static_cast<cuuint64_t>(row_stride) * 2 * static_cast<cuuint64_t>(rows)};
  cuuint32_t box[3] = {64, static_cast<cuuint32_t>(box_rows), 1}, estr[3] = {1, 1, 1};
  const CUresult r = fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(base), dims, strides, box, estr,
                        CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                        CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  return r == CUDA_SUCCESS ? kOk : kTensorMapFailed;
}

template <int BN, bool GATED>
static int launch_moe_gemm(const CUtensorMap& wm, const CUtensorMap& xm, const GroupParams& p, cudaStream_t st) {
  using C = MoeCfg<BN>;
  struct Tag {};
  const int rc = opt_in_dynamic_smem<Tag>(reinterpret_cast<const void*>(&moe_gemm_kernel<BN, GATED>), C::SMEM);
  if (rc != kOk) return rc;
  const int64_t items = static_cast<int64_t>(p.max_tiles) * p.blocks;
  int grid = sm_count();
  if (grid > items) grid = static_cast<int>(items);
  moe_gemm_kernel<BN, GATED><<<grid, kMoeThreads, C::SMEM, st>>>(wm, xm, p);
  return cudaGetLastError() == cudaSuccess ? kOk : kLaunchFailed;
}

}  // namespace mvb

extern "C" int mvb_moe_route_ext(const float* logits, int64_t logits_row_stride, int num_tokens, int num_experts, int num_identity, int top,
                                 int softmax, const float* correction, float weight_scale, int block_rows, int max_tiles,
                                 int32_t* counters, int32_t* ids, float* weights, int32_t* ranks, int32_t* offsets, int32_t* tile_offsets,
                                 int32_t* tiles, float* identity_weights, void* stream) {
  using namespace mvb;
  if (!logits || !counters || !ids || !weights || !ranks || !offsets || !tile_offsets || !tiles) return kInvalidArgument;
  if (num_tokens <= 0 || num_experts <= 0 || num_identity < 0 || top <= 0 || top > num_experts + num_identity || block_rows <= 0)
    return kInvalidArgument;
  if (num_identity > 0 && identity_weights == nullptr) return kInvalidArgument;
  if (num_experts + num_identity > kMaxExperts || static_cast<int64_t>(num_tokens) * top > 0x7fffffffLL) return kUnsupportedShape;
  const int64_t rows = static_cast<int64_t>(num_tokens) * top, part = rows < num_experts ? rows : num_experts;
  if (max_tiles < rows / block_rows + part || !is_aligned(tiles, 16)) return kInvalidArgument;
  const int outputs = num_experts + num_identity;
  const RouteParams p{logits, logits_row_stride, num_tokens, num_experts, top, block_rows, max_tiles, counters, ids, weights, ranks, offsets,
                      tile_offsets, reinterpret_cast<int4*>(tiles), outputs, softmax, correction, weight_scale, identity_weights};
  const int warps = kRouteThreads / 32;
  int grid = (num_tokens + warps - 1) / warps;
  if (grid > 4 * sm_count()) grid = 4 * sm_count();
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (outputs <= 32) moe_route_kernel<1><<<grid, kRouteThreads, 0, st>>>(p);
  else if (outputs <= 64) moe_route_kernel<2><<<grid, kRouteThreads, 0, st>>>(p);
  else if (outputs <= 128) moe_route_kernel<4><<<grid, kRouteThreads, 0, st>>>(p);
  else if (outputs <= 256) moe_route_kernel<8><<<grid, kRouteThreads, 0, st>>>(p);
  else moe_route_kernel<32><<<grid, kRouteThreads, 0, st>>>(p);
  return cudaGetLastError() == cudaSuccess ? kOk : kLaunchFailed;
}

extern "C" int mvb_moe_route(const float* logits, int64_t logits_row_stride, int num_tokens, int num_experts, int top, int block_rows,
                             int max_tiles, int32_t* counters, int32_t* ids, float* weights, int32_t* ranks, int32_t* offsets,
                             int32_t* tile_offsets, int32_t* tiles, void* stream) {
  return mvb_moe_route_ext(logits, logits_row_stride, num_tokens, num_experts, 0, top, 0, nullptr, 1.f, block_rows, max_tiles, counters,
                           ids, weights, ranks, offsets, tile_offsets, tiles, nullptr, stream);
}

extern "C" int mvb_moe_gather(int dtype, const void* h, int64_t h_row_stride, const int32_t* ids, const float* weights,
                              const int32_t* ranks, const int32_t* offsets, void* out, int64_t out_row_stride, int32_t* slots,
                              float* row_weights, int num_tokens, int top, int width, void* stream) {
  using namespace mvb;
  if (!h || !ids || !weights || !ranks || !offsets || !out || !slots || !row_weights || num_tokens < 0 || top <= 0 || width <= 0 ||
      (dtype != kBf16 && dtype != kF32))
    return kInvalidArgument;
  if (num_tokens == 0) return kOk;
  const int v = dtype == kBf16 ? 8 : 4;
  const int vec = width % v == 0 && h_row_stride % v == 0 && out_row_stride % v == 0 && is_aligned(h, 16) && is_aligned(out, 16);
  const int parts = vec ? (width / v + kGatherPart - 1) / kGatherPart : 1;
  const int64_t blocks = (static_cast<int64_t>(num_tokens) * parts + 7) / 8;
  if (blocks > 0x7fffffffLL / 8) return kUnsupportedShape;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const unsigned grid = static_cast<unsigned>(blocks);
  if (dtype == kBf16)
    moe_gather_kernel<<<grid, 256, 0, st>>>(static_cast<const __nv_bfloat16*>(h), h_row_stride, ids, weights, ranks, offsets,
                                            static_cast<__nv_bfloat16*>(out), out_row_stride, slots, row_weights, num_tokens, top, width,
                                            parts, vec);
  else
    moe_gather_kernel<<<grid, 256, 0, st>>>(static_cast<const float*>(h), h_row_stride, ids, weights, ranks, offsets,
                                            static_cast<float*>(out), out_row_stride, slots, row_weights, num_tokens, top, width, parts, vec);
  return cudaGetLastError() == cudaSuccess ? kOk : kLaunchFailed;
}

extern "C" int mvb_moe_gemm(int dtype, const void* x, int64_t x_row_stride, int64_t num_rows, const void* weight, int64_t w_row_stride,
                            int num_experts, int m, int k, int gated, float limit, float alpha, float offset, const float* row_weights,
                            const int32_t* num_tiles, const int32_t* tiles, int max_tiles, int block_rows, void* out,
                            int64_t out_row_stride, int32_t* dev_status, void* stream) {
  using namespace mvb;
  if (!x || !weight || !num_tiles || !tiles || !out || num_rows < 0 || num_experts <= 0 || m <= 0 || k <= 0 || max_tiles < 0)
    return kInvalidArgument;
  if (dtype != kBf16 && dtype != kF32) return kInvalidArgument;
  if (num_rows == 0 || max_tiles == 0) return kOk;
  if (num_rows > 0x7fffffffLL || max_tiles > 65535 || !is_aligned(tiles, 16)) return kUnsupportedShape;
  GroupParams p{num_tiles, reinterpret_cast<const int4*>(tiles), max_tiles, row_weights, gated == 2, out, out_row_stride, m, 0, k, limit,
                -alpha * 1.4426950408889634f, offset, nullptr, 0, nullptr, dev_status};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (dtype == kF32) {
    if (block_rows != 64 || w_row_stride != k) return kUnsupportedShape;
    p.x32 = static_cast<const float*>(x); p.x_stride = x_row_stride; p.w32 = static_cast<const float*>(weight);
    const dim3 grid((m + 63) / 64, max_tiles);
    if (gated) moe_gemm_f32_kernel<true><<<grid, 256, 0, st>>>(p);
    else moe_gemm_f32_kernel<false><<<grid, 256, 0, st>>>(p);
    return cudaGetLastError() == cudaSuccess ? kOk : kLaunchFailed;
  }
  if (block_rows != 32 && block_rows != 64 && block_rows != 128) return kUnsupportedShape;
  p.blocks = gated ? (m + 127) / 128 : (m + 255) / 256;
  CUtensorMap wm, xm;
  int rc = make_group_map(&wm, weight, k, m, static_cast<int64_t>(num_experts) * (gated ? 2 : 1), w_row_stride, 128);
  if (rc != kOk) return rc;
  rc = make_group_map(&xm, x, k, num_rows, 1, x_row_stride, block_rows);
  if (rc != kOk) return rc;
  auto launch = [&](auto gated_tag) {
    constexpr bool G = decltype(gated_tag)::value;
    if (block_rows == 32) return launch_moe_gemm<32, G>(wm, xm, p, st);
    if (block_rows == 64) return launch_moe_gemm<64, G>(wm, xm, p, st);
    return launch_moe_gemm<128, G>(wm, xm, p, st);
  };
  return gated ? launch(std::true_type{}) : launch(std::false_type{});
}
