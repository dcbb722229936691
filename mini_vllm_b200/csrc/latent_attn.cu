// Attention over a latent: keys and values of all heads are projections of one vector c per token, and only c is cached
// (pool [blocks, block_size, width], one "head").
//
//   latent_norm_kernel      RMS norms of the query latent and of c, c also into its cache slot
//   gather_latents_kernel   the contexts of a ragged step as dense rows (keys and values are then two matrix products away, and the
//                           prefill attention kernel takes them)
//   latent_decode_kernel    one query token per sequence in the absorbed form: with q' = q W_uk per head a score is q' . c, and the
//                           softmax-weighted sum of c (times W_uv afterwards) is the output.  Every head reads the same c, so a row of the
//                           cache is loaded once for all of them: the roofline is HBM, sum_b context(b) * width * 2 bytes
//   gate_mul_kernel         o * sigmoid(gate)
//
// latent_decode_kernel: persistent CTAs over the tile ranges of decode_plan.cuh.  A tile = 32 tokens x width in 128-byte-swizzled shared
// memory, brought by TMA through the block table, up to six tiles deep.  Two groups of eight warps take the tiles in turn, so that one
// group's barriers and latencies lie under the other's arithmetic; each keeps its own running softmax, and they meet at the end of a
// sequence.  Per tile and group, three barriers of 256 threads:
//   scores   S[heads x 32] = Q' C^T     warp = 16 tokens x a quarter of the width (mma.sync, heads in M); the quarters meet in shared memory
//   softmax  a few threads per head, running maximum and sum in registers, P as bf16 through shared memory
//   output   O[heads x width] += P C    warp = an eighth of the width (C again, as transposed fragments), O in registers
// A stage is filled again by the group that has just read it, so the groups never wait for each other inside a sequence.
// A sequence that is split between CTAs is merged by the CTA that arrives last, as in decode_attn.cu; nothing waits on another CTA.
#include "chunk_common.cuh"
#include "decode_plan.cuh"
#include "mini_vllm_b200.h"

namespace mvb {

// ---- norms + cache write -------------------------------------------------------------------------------------
struct LatentNormParams {
  const void* q; int64_t q_stride; const void* q_weight; void* q_out; int q_cols, q_pad;
  const void* c; int64_t c_stride; const void* c_weight; void* c_out; int c_cols, c_pad;     // c == nullptr: no latent of its own
  void* cache; const int32_t* slot_mapping; int64_t num_slots;                               // cache == nullptr: not written
  int tokens;
  float eps;
  int* dev_status;
};

template <class T, int V>
__device__ __forceinline__ void norm_row(const T* src, const T* weight, int cols, int pad, float eps, T* out, T* out2, int lane) {
  float ss = 0.f;
  for (int i = lane * V; i < cols; i += 32 * V) {
    float x[V];
    load_vec<T, V>(src + i, x);
#pragma unroll
    for (int j = 0; j < V; ++j) ss += x[j] * x[j];
  }
  const float r = 1.f / sqrtf(warp_sum(ss) / static_cast<float>(cols) + eps);
  for (int i = lane * V; i < cols; i += 32 * V) {
    float x[V], w[V];
    load_vec<T, V>(src + i, x);
    load_vec<T, V>(weight + i, w);
#pragma unroll
    for (int j = 0; j < V; ++j) x[j] = x[j] * r * w[j];
    store_vec<T, V>(out + i, x);
    if (out2 != nullptr) store_vec<T, V>(out2 + i, x);
  }
  for (int i = cols + lane; i < pad; i += 32) {
    out[i] = from_f<T>(0.f);
    if (out2 != nullptr) out2[i] = from_f<T>(0.f);
  }
}

// a warp per row: query latents first, then the cached ones
template <class T, int V>
__global__ void __launch_bounds__(128) latent_norm_kernel(const LatentNormParams p) {
  int w = static_cast<int>((static_cast<int64_t>(blockIdx.x) * 128 + threadIdx.x) >> 5);
  const int lane = threadIdx.x & 31;
  if (w < p.tokens) {
    norm_row<T, V>(static_cast<const T*>(p.q) + w * p.q_stride, static_cast<const T*>(p.q_weight), p.q_cols, p.q_pad, p.eps,
                   static_cast<T*>(p.q_out) + static_cast<int64_t>(w) * p.q_pad, nullptr, lane);
    return;
  }
  w -= p.tokens;
  if (p.c == nullptr || w >= p.tokens) return;
  T* cached = nullptr;
  if (p.cache != nullptr) {
    const int64_t slot = p.slot_mapping[w];
    if (slot >= p.num_slots) {
      if (lane == 0) report(p.dev_status, kDevBadSlot, w);
    } else if (slot >= 0) {
      cached = static_cast<T*>(p.cache) + slot * p.c_pad;
    }
  }
  norm_row<T, V>(static_cast<const T*>(p.c) + w * p.c_stride, static_cast<const T*>(p.c_weight), p.c_cols, p.c_pad, p.eps,
                 static_cast<T*>(p.c_out) + static_cast<int64_t>(w) * p.c_pad, cached, lane);
}

template <class T>
static int launch_latent_norm(const LatentNormParams& p, cudaStream_t st) {
  constexpr int V = kVec<T>;
  const bool vec = p.q_cols % V == 0 && p.q_pad % V == 0 && p.q_stride % V == 0 && is_aligned(p.q, 16) && is_aligned(p.q_weight, 16) &&
                   is_aligned(p.q_out, 16) && (p.c == nullptr || (p.c_cols % V == 0 && p.c_pad % V == 0 && p.c_stride % V == 0 &&
                   is_aligned(p.c, 16) && is_aligned(p.c_weight, 16) && is_aligned(p.c_out, 16) && is_aligned(p.cache, 16)));
  const int64_t warps = static_cast<int64_t>(p.tokens) * (p.c == nullptr ? 1 : 2);
  const unsigned blocks = static_cast<unsigned>((warps + 3) / 4);
  if (vec) latent_norm_kernel<T, V><<<blocks, 128, 0, st>>>(p);
  else latent_norm_kernel<T, 1><<<blocks, 128, 0, st>>>(p);
  return cudaGetLastError() == cudaSuccess ? kOk : kLaunchFailed;
}

// ---- contexts as dense rows -----------------------------------------------------------------------------------
__global__ void __launch_bounds__(256) gather_latents_kernel(const uint4* __restrict__ cache, int64_t num_slots, int row_vecs,
                                                             const int32_t* __restrict__ block_table, int64_t table_stride, int table_width,
                                                             int block_size, const int32_t* __restrict__ cu_k, int num_seqs, int rows,
                                                             uint4* __restrict__ out, int* dev_status) {
  const int warp = static_cast<int>((static_cast<int64_t>(blockIdx.x) * 256 + threadIdx.x) >> 5), lane = threadIdx.x & 31;
  if (warp >= rows) return;
  const int s = seq_of_row(cu_k, num_seqs, warp), j = warp - cu_k[s], col = j / block_size;
  const int64_t blk = col < table_width ? block_table[s * table_stride + col] : -1;
  const int64_t slot = blk * block_size + j % block_size;
  const bool ok = blk >= 0 && slot < num_slots;
  if (!ok && lane == 0) report(dev_status, kDevBadBlock, s);
  for (int i = lane; i < row_vecs; i += 32)
    out[static_cast<int64_t>(warp) * row_vecs + i] = ok ? cache[slot * row_vecs + i] : make_uint4(0u, 0u, 0u, 0u);
}

// ---- output gate ------------------------------------------------------------------------------------------------
template <class T, int V>
__global__ void __launch_bounds__(128) gate_mul_kernel(const T* __restrict__ o, int64_t o_stride, const T* __restrict__ g, int64_t g_stride,
                                                       T* __restrict__ out, int64_t out_stride, int rows, int cols) {
  const int c = (blockIdx.x * 128 + threadIdx.x) * V;
  if (c >= cols) return;
  for (int t = blockIdx.y; t < rows; t += gridDim.y) {
    float x[V], z[V];
    load_vec<T, V>(o + t * o_stride + c, x);
    load_vec<T, V>(g + t * g_stride + c, z);
#pragma unroll
    for (int i = 0; i < V; ++i)
      x[i] *= sizeof(T) == 2 ? fast_rcp(1.f + fast_exp2(z[i] * -1.4426950408889634f)) : sigmoid_f(z[i]);
    store_vec<T, V>(out + t * out_stride + c, x);
  }
}

template <class T>
static int launch_gate(const void* o, int64_t os, const void* g, int64_t gs, void* out, int64_t outs, int rows, int cols, cudaStream_t st) {
  constexpr int V = kVec<T>;
  const bool vec = cols % V == 0 && os % V == 0 && gs % V == 0 && outs % V == 0 && is_aligned(o, 16) && is_aligned(g, 16) && is_aligned(out, 16);
  const int v = vec ? V : 1, bx = (cols + 128 * v - 1) / (128 * v);
  int by = rows, cap = (sm_count() * 16 + bx - 1) / bx;
  if (by > cap) by = cap;
  if (by > 65535) by = 65535;
  auto to = static_cast<const T*>(o); auto tg = static_cast<const T*>(g); auto tout = static_cast<T*>(out);
  if (vec) gate_mul_kernel<T, V><<<dim3(bx, by), 128, 0, st>>>(to, os, tg, gs, tout, outs, rows, cols);
  else gate_mul_kernel<T, 1><<<dim3(bx, by), 128, 0, st>>>(to, os, tg, gs, tout, outs, rows, cols);
  return cudaGetLastError() == cudaSuccess ? kOk : kLaunchFailed;
}

// ---- decode -----------------------------------------------------------------------------------------------------
constexpr int kLatentTile = 32;

template <int RH, int MT>                       // width = 64 RH, 16 MT heads per CTA
struct LatentCfg {
  static constexpr int W = 64 * RH, HEADS = 16 * MT, TOK = kLatentTile;
  static constexpr int HALF = TOK * 128, STAGE = RH * HALF;             // 32 tokens x 64 columns
  static constexpr int QROW = W * 2 + 16, SROW = TOK + 4, PROW = TOK * 2 + 16;
  static constexpr int Q = HEADS * QROW, SB = 4 * HEADS * SROW * 4, P = HEADS * PROW, ROWS = 3 * HEADS * 4;     // (the last three per group)
  static constexpr int FIXED = Q + 2 * (SB + P + ROWS) + 64;
  static constexpr int FIT = (226 * 1024 - 1024 - FIXED) / STAGE;
  static constexpr int NST = FIT > 6 ? 6 : FIT;
  static constexpr int SMEM = 1024 + NST * STAGE + FIXED;
  static_assert(NST >= 3, "a tile per group and one in flight at least");
  static_assert(HEADS * (W / 2) * 4 <= 2 * SB, "half of O fits the score buffers");
};

struct LatentDecodeParams {
  const __nv_bfloat16* q; int64_t q_stride, q_head_stride;
  __nv_bfloat16* out; int64_t out_stride, out_head_stride;
  const int32_t* cache_seqlens;
  const int32_t* block_table; int64_t table_stride; int table_width;
  int num_seqs, heads, block_size;
  int64_t num_blocks;
  float scale_log2;
  const CtaDesc* descs;
  const int32_t* tile_prefix;
  float *part_lse, *part_o;
  int32_t* arrivals;
  int* dev_status;
};

struct SeqSpan { int b, tp0, tp1, n; };          // a sequence, its tile range, its length

__device__ __forceinline__ void group_sync(int group) { asm volatile("barrier.cta.sync.aligned %0, 256;" ::"r"(group + 1) : "memory"); }
__device__ __forceinline__ bool group_all(int group, bool ok) {
  uint32_t r;
  asm volatile(
      "{\n\t.reg .pred p, q;\n\t"
      "setp.ne.u32 q, %1, 0;\n\t"
      "barrier.cta.red.and.aligned.pred p, %2, 256, q;\n\t"
      "selp.u32 %0, 1, 0, p;\n\t}"
      : "=r"(r) : "r"(static_cast<uint32_t>(ok)), "r"(group + 1) : "memory");
  return r != 0;
}

template <int RH, int MT>
__global__ void __launch_bounds__(512, 1) latent_decode_kernel(const __grid_constant__ CUtensorMap map, const LatentDecodeParams p) {
  using C = LatentCfg<RH, MT>;
  constexpr int TOK = C::TOK, NST = C::NST, W = C::W, HEADS = C::HEADS;
  constexpr uint32_t FULL = 0xffffffffu;
  extern __shared__ uint8_t smem_raw[];
  const int tid = threadIdx.x, group = tid >> 8, gt = tid & 255, warp = gt >> 5, lane = tid & 31, c = blockIdx.x;
  const int head0 = blockIdx.y * HEADS, nheads = min(HEADS, p.heads - head0);
  const CtaDesc desc = p.descs[c];
  auto zero_empty_rows = [&]() {
    for (int b = c; b < p.num_seqs; b += gridDim.x)
      if (p.cache_seqlens[b] <= 0)
        for (int e = tid; e < nheads * W; e += 512)
          p.out[b * p.out_stride + (head0 + e / W) * p.out_head_stride + e % W] = __float2bfloat16_rn(0.f);
  };
  if (desc.t0 >= desc.t1) { zero_empty_rows(); return; }

  const uint32_t base = (smem_u32(smem_raw) + 1023u) & ~1023u;
  uint8_t* base_ptr = smem_raw + (base - smem_u32(smem_raw));
  uint8_t* q_s = base_ptr + NST * C::STAGE;
  float* scores = reinterpret_cast<float*>(q_s + C::Q);                 // [group][quarter][HEADS][SROW]; also O and weights in a merge
  uint8_t* p_all = q_s + C::Q + 2 * C::SB;                              // [group][HEADS][PROW bytes]
  float* rows_s = reinterpret_cast<float*>(p_all + 2 * C::P);           // [group][alpha | l | m][HEADS]
  uint64_t* full = reinterpret_cast<uint64_t*>(rows_s + 6 * HEADS);
  float* s_s = scores + group * (C::SB / 4);
  uint8_t* p_s = p_all + group * C::P;
  float *alpha_s = rows_s + group * 3 * HEADS, *l_s = alpha_s + HEADS, *m_s = l_s + HEADS;
  const uint32_t q_base = smem_u32(q_s), p_base = smem_u32(p_s);
  if (tid == 0) {
    tma_prefetch_desc(&map);
    for (int i = 0; i < NST; ++i) mbar_init(&full[i], 1);
    fence_mbar_init();
  }
  __syncthreads();

  // ---- producer: warp 0 of a group; tiles are counted from desc.t0, tile i lives in stage i % NST ----
  const int total = desc.t1 - desc.t0;
  SeqSpan fs{desc.b, desc.tp0, desc.tp1, desc.n}, cs = fs;
  auto next_seq = [&](SeqSpan& v) {
    ++v.b; v.tp0 = p.tile_prefix[v.b]; v.tp1 = p.tile_prefix[v.b + 1]; v.n = p.cache_seqlens[v.b];
  };
  int blk_base = -1, blk_reg = -1, blk_n = 0, fetched = -1;
  if (desc.blk0 >= 0) { blk_base = (desc.t0 - desc.tp0) * TOK / p.block_size; blk_reg = desc.blk0; blk_n = 1; }
  auto fetch = [&](int i) {                                             // all lanes; i only grows
    if (i >= total) return;
    const int t = desc.t0 + i;
    while (t >= fs.tp1 && fs.b + 1 < p.num_seqs) { next_seq(fs); blk_base = -1; blk_n = 0; }
    const int token0 = (t - fs.tp0) * TOK, bi = token0 / p.block_size;
    if (blk_base < 0 || bi < blk_base || bi >= blk_base + blk_n) {
      blk_base = bi; blk_n = 32;
      const int col = bi + lane;
      blk_reg = col < p.table_width ? p.block_table[fs.b * p.table_stride + col] : -1;
    }
    const int blk = __shfl_sync(FULL, blk_reg, bi - blk_base);
    int slot0 = -TOK;                                                   // out of range: TMA fills zeros
    if (blk >= 0 && blk < p.num_blocks) slot0 = blk * p.block_size + (token0 - bi * p.block_size);
    else if (lane == 0) report(p.dev_status, kDevBadBlock, fs.b);
    if (lane == 0) {
      const int st = i % NST;
      fence_proxy_async();
      mbar_arrive_expect_tx(&full[st], C::STAGE);
#pragma unroll
      for (int h = 0; h < RH; ++h) tma_load_3d(base_ptr + st * C::STAGE + h * C::HALF, &map, &full[st], h * 64, 0, slot0);
    }
    fetched = i;
  };
  if (group == 0 && warp == 0)
    for (int i = 0; i < NST; ++i) fetch(i);

  const int first_b = cs.b;
  int seg = 0, i = group;                                               // first tile of the segment; this group's next tile
  bool dead = false;
  const int tg = warp & 1, kq = warp >> 1;                              // scores: 16-token group, quarter of the width
  constexpr int TPR = 256 / HEADS, TPT = TOK / TPR;                     // softmax: threads per head, tokens per thread
  const int srow = gt / TPR, ssub = gt % TPR, mi = lane >> 3;
  while (seg < total) {
    while (desc.t0 + seg >= cs.tp1 && cs.b + 1 < p.num_seqs) next_seq(cs);
    const int seg_end = min(desc.t1, cs.tp1) - desc.t0, b = cs.b;
    const bool whole = desc.t0 + seg == cs.tp0 && desc.t0 + seg_end == cs.tp1;
    __syncthreads();                                                    // the queries of the sequence before have been read
    for (int e = tid; e < HEADS * (W / 8); e += 512) {
      const int h = e / (W / 8), v = e % (W / 8);
      uint4 x = make_uint4(0u, 0u, 0u, 0u);
      if (h < nheads) x = *reinterpret_cast<const uint4*>(p.q + b * p.q_stride + (head0 + h) * p.q_head_stride + v * 8);
      *reinterpret_cast<uint4*>(q_s + h * C::QROW + v * 16) = x;
    }
    __syncthreads();
    const uint32_t qrow = q_base + ((lane & 7) + (mi & 1) * 8) * C::QROW + (lane >> 4) * 16 + kq * RH * 32;
    uint32_t qa[MT == 1 ? RH : 1][4];                                   // one head tile: its query fragments stay in registers
    if constexpr (MT == 1) {
#pragma unroll
      for (int k = 0; k < RH; ++k) ldmatrix_x4(qa[k], qrow + k * 32);
    }
    float o[MT][RH][4];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
      for (int n = 0; n < RH; ++n) o[m][n][0] = o[m][n][1] = o[m][n][2] = o[m][n][3] = 0.f;
    float m_run = -INFINITY, l_run = 0.f;

    for (; i < seg_end; i += 2) {
      if (dead) continue;
      const int st = i % NST;
      const bool ok = mbar_wait(&full[st], (i / NST) & 1);
      if (!group_all(group, ok)) {                                      // (also: the group is done with its tile before)
        if (!ok) report(p.dev_status, kDevWaitTimeout, i);
        dead = true;
        continue;
      }
      if (warp == 0 && i >= 2) fetch(i - 2 + NST);                      // into the stage that tile has left
      const uint32_t stage = base + st * C::STAGE;
      const int token0 = (desc.t0 + i - cs.tp0) * TOK, valid = cs.n - token0;
      if (valid < TOK) {                                                // rows behind the end may hold anything: zero them
        for (int e = gt; e < (TOK - valid) * RH * 8; e += 256) {
          const int r = valid + e / (RH * 8), k = e % (RH * 8);
          *reinterpret_cast<uint4*>(base_ptr + st * C::STAGE + (k >> 3) * C::HALF + r * 128 + (k & 7) * 16) = make_uint4(0u, 0u, 0u, 0u);
        }
        group_sync(group);
      }
      {                                                                 // scores
        float s[MT][2][4];
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
          for (int n = 0; n < 2; ++n) s[m][n][0] = s[m][n][1] = s[m][n][2] = s[m][n][3] = 0.f;
        const int tok = tg * 16 + (lane & 7) + (mi >> 1) * 8;
        const uint32_t trow = stage + tok * 128;
#pragma unroll
        for (int k = 0; k < RH; ++k) {
          const int chunk = (kq * RH + k) * 2 + (mi & 1);
          uint32_t cb[4];
          ldmatrix_x4(cb, trow + (chunk >> 3) * C::HALF + (((chunk & 7) ^ (tok & 7)) << 4));
#pragma unroll
          for (int m = 0; m < MT; ++m) {
            if constexpr (MT == 1) {
              mma_bf16_16816(s[0][0], qa[k], cb[0], cb[1]);
              mma_bf16_16816(s[0][1], qa[k], cb[2], cb[3]);
            } else {
              uint32_t a[4];
              ldmatrix_x4(a, qrow + m * 16 * C::QROW + k * 32);
              mma_bf16_16816(s[m][0], a, cb[0], cb[1]);
              mma_bf16_16816(s[m][1], a, cb[2], cb[3]);
            }
          }
        }
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
          for (int n = 0; n < 2; ++n) {
            float* d = s_s + (kq * HEADS + m * 16 + (lane >> 2)) * C::SROW + tg * 16 + n * 8 + (lane & 3) * 2;
            *reinterpret_cast<float2*>(d) = make_float2(s[m][n][0], s[m][n][1]);
            *reinterpret_cast<float2*>(d + 8 * C::SROW) = make_float2(s[m][n][2], s[m][n][3]);
          }
      }
      group_sync(group);
      {                                                                 // softmax
        float x[TPT], top = -INFINITY;
        const float* r0 = s_s + srow * C::SROW + ssub * TPT;
#pragma unroll
        for (int j = 0; j < TPT; j += 2) {
          float2 a = *reinterpret_cast<const float2*>(r0 + j);
#pragma unroll
          for (int k = 1; k < 4; ++k) {
            const float2 d = *reinterpret_cast<const float2*>(r0 + k * HEADS * C::SROW + j);
            a.x += d.x; a.y += d.y;
          }
          x[j] = a.x; x[j + 1] = a.y;
        }
#pragma unroll
        for (int j = 0; j < TPT; ++j) {
          x[j] = ssub * TPT + j < valid ? x[j] * p.scale_log2 : -INFINITY;
          top = fmaxf(top, x[j]);
        }
#pragma unroll
        for (int off = 1; off < TPR; off <<= 1) top = fmaxf(top, __shfl_xor_sync(FULL, top, off));
        const float m_new = fmaxf(m_run, top), alpha = fast_exp2(m_run - m_new);      // (a tile has a visible token: m_new is finite)
        float sum = 0.f;
#pragma unroll
        for (int j = 0; j < TPT; ++j) { x[j] = fast_exp2(x[j] - m_new); sum += x[j]; }
#pragma unroll
        for (int off = 1; off < TPR; off <<= 1) sum += __shfl_xor_sync(FULL, sum, off);
        l_run = l_run * alpha + sum;
        m_run = m_new;
#pragma unroll
        for (int j = 0; j < TPT; j += 2)
          *reinterpret_cast<uint32_t*>(p_s + srow * C::PROW + (ssub * TPT + j) * 2) = pack_bf16(x[j], x[j + 1]);
        if (ssub == 0) alpha_s[srow] = alpha;
      }
      group_sync(group);
      {                                                                 // output
        uint32_t pa[MT][2][4];
        const uint32_t prow = p_base + ((lane & 7) + (mi & 1) * 8) * C::PROW + (lane >> 4) * 16;
#pragma unroll
        for (int m = 0; m < MT; ++m) {
          const float a0 = alpha_s[m * 16 + (lane >> 2)], a1 = alpha_s[m * 16 + (lane >> 2) + 8];
#pragma unroll
          for (int k = 0; k < 2; ++k) ldmatrix_x4(pa[m][k], prow + m * 16 * C::PROW + k * 32);
#pragma unroll
          for (int n = 0; n < RH; ++n) { o[m][n][0] *= a0; o[m][n][1] *= a0; o[m][n][2] *= a1; o[m][n][3] *= a1; }
        }
        const uint32_t trow = stage + lane * 128;                       // a lane addresses its token: two 16-token steps
#pragma unroll
        for (int n = 0; n < RH; ++n) {
          const int chunk = warp * RH + n;
          uint32_t cb[4];
          ldmatrix_x4_trans(cb, trow + (chunk >> 3) * C::HALF + (((chunk & 7) ^ (lane & 7)) << 4));
#pragma unroll
          for (int m = 0; m < MT; ++m) {
            mma_bf16_16816(o[m][n], pa[m][0], cb[0], cb[1]);
            mma_bf16_16816(o[m][n], pa[m][1], cb[2], cb[3]);
          }
        }
      }
    }
    // ---- end of the segment: the groups meet (half of the columns at a time), then output or a partial result ----
    if (ssub == 0) { l_s[srow] = l_run; m_s[srow] = m_run; }
    __syncthreads();
    const int part = b == first_b ? 0 : 1;
    auto row_weights = [&](int h, float& w0, float& w1, float& m, float& l) {          // of the groups' O in the result
      const float m0 = rows_s[2 * HEADS + h], m1 = rows_s[5 * HEADS + h];
      m = fmaxf(m0, m1);
      w0 = m0 == -INFINITY ? 0.f : fast_exp2(m0 - m);
      w1 = m1 == -INFINITY ? 0.f : fast_exp2(m1 - m);
      l = rows_s[HEADS + h] * w0 + rows_s[4 * HEADS + h] * w1;
      const float inv = l > 0.f ? 1.f / l : 0.f;
      w0 *= inv; w1 *= inv;
    };
#pragma unroll 1
    for (int half = 0; half < 2; ++half) {
      const int wl = warp - half * 4;
      const bool mine = wl >= 0 && wl < 4;
      if (group == 1 && mine) {
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
          for (int r = 0; r < 2; ++r)
#pragma unroll
            for (int n = 0; n < RH; ++n)
              *reinterpret_cast<float2*>(scores + (m * 16 + (lane >> 2) + r * 8) * (W / 2) + (wl * RH + n) * 8 + (lane & 3) * 2) =
                  make_float2(o[m][n][2 * r], o[m][n][2 * r + 1]);
      }
      __syncthreads();
      if (group == 0 && mine) {
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
          for (int r = 0; r < 2; ++r) {
            const int h = m * 16 + (lane >> 2) + r * 8;
            if (h >= nheads) continue;
            float w0, w1, mm, ll;
            row_weights(h, w0, w1, mm, ll);
#pragma unroll
            for (int n = 0; n < RH; ++n) {
              const float2 other = *reinterpret_cast<const float2*>(scores + h * (W / 2) + (wl * RH + n) * 8 + (lane & 3) * 2);
              const int col = (warp * RH + n) * 8 + (lane & 3) * 2;
              const float x = o[m][n][2 * r] * w0 + other.x * w1, y = o[m][n][2 * r + 1] * w0 + other.y * w1;
              if (whole) *reinterpret_cast<uint32_t*>(p.out + b * p.out_stride + (head0 + h) * p.out_head_stride + col) = pack_bf16(x, y);
              else *reinterpret_cast<float2*>(p.part_o + ((static_cast<int64_t>(c) * 2 + part) * p.heads + head0 + h) * W + col) = make_float2(x, y);
            }
          }
      }
      __syncthreads();
    }
    if (!whole) {
      __shared__ int is_last;
      if (tid < nheads) {
        float w0, w1, m, l;
        row_weights(tid, w0, w1, m, l);
        p.part_lse[(static_cast<int64_t>(c) * 2 + part) * p.heads + head0 + tid] = l > 0.f ? m + log2f(l) : -INFINITY;
      }
      const int per = desc.per, c1 = cs.tp0 / per, c2 = (cs.tp1 - 1) / per, nparts = c2 - c1 + 1;
      // the CTA barrier orders every thread's partial stores before thread 0's release; the last arriver's acquire plus its CTA
      // barrier order them before every merging thread's loads
      __syncthreads();
      if (tid == 0) {
        int32_t* cnt = p.arrivals + static_cast<int64_t>(b) * gridDim.y + blockIdx.y;
        int prev;
        asm volatile("atom.acq_rel.gpu.global.add.s32 %0, [%1], 1;" : "=r"(prev) : "l"(cnt) : "memory");
        is_last = prev == nparts - 1;
        if (is_last) *cnt = 0;                                          // re-arm for the next launch
      }
      __syncthreads();
      if (is_last) {
        const bool first_is_head = cs.tp0 % per == 0;                   // does CTA c1's range start at this sequence?
        auto part_index = [&](int j, int h) -> int64_t {
          return ((static_cast<int64_t>(c1 + j) * 2 + (j > 0 || first_is_head ? 0 : 1)) * p.heads) + head0 + h;
        };
        constexpr int PC = 32;                                          // parts weighted per pass, in the score buffers
        float *top_s = rows_s, *inv_s = rows_s + HEADS;
        for (int e = tid; e < nheads; e += 512) {
          float top = -INFINITY, sum = 0.f;
          for (int j = 0; j < nparts; ++j) top = fmaxf(top, __ldcg(p.part_lse + part_index(j, e)));
          for (int j = 0; j < nparts; ++j) sum += top == -INFINITY ? 0.f : fast_exp2(__ldcg(p.part_lse + part_index(j, e)) - top);
          top_s[e] = top;
          inv_s[e] = sum > 0.f ? 1.f / sum : 0.f;
        }
        __syncthreads();
        constexpr int ITEMS = (HEADS * W / 4 + 511) / 512;
        float4 acc[ITEMS];
#pragma unroll
        for (int k = 0; k < ITEMS; ++k) acc[k] = make_float4(0.f, 0.f, 0.f, 0.f);
        for (int p0 = 0; p0 < nparts; p0 += PC) {
          const int pn = min(PC, nparts - p0);
          for (int e = tid; e < pn * nheads; e += 512) {
            const int h = e % nheads;
            scores[e] = inv_s[h] == 0.f ? 0.f : fast_exp2(__ldcg(p.part_lse + part_index(p0 + e / nheads, h)) - top_s[h]) * inv_s[h];
          }
          __syncthreads();
#pragma unroll
          for (int k = 0; k < ITEMS; ++k) {
            const int it = tid + k * 512, h = it * 4 / W, col = it * 4 % W;
            if (h >= nheads) continue;
#pragma unroll 4
            for (int j = 0; j < pn; ++j) {
              const float w = scores[j * nheads + h];
              const float4 v = __ldcg(reinterpret_cast<const float4*>(p.part_o + part_index(p0 + j, h) * W + col));
              acc[k].x = fmaf(w, v.x, acc[k].x); acc[k].y = fmaf(w, v.y, acc[k].y);
              acc[k].z = fmaf(w, v.z, acc[k].z); acc[k].w = fmaf(w, v.w, acc[k].w);
            }
          }
          __syncthreads();
        }
#pragma unroll
        for (int k = 0; k < ITEMS; ++k) {
          const int it = tid + k * 512, h = it * 4 / W, col = it * 4 % W;
          if (h < nheads)
            *reinterpret_cast<uint2*>(p.out + b * p.out_stride + (head0 + h) * p.out_head_stride + col) =
                make_uint2(pack_bf16(acc[k].x, acc[k].y), pack_bf16(acc[k].z, acc[k].w));
        }
      }
    }
    seg = seg_end;
  }
  if (dead && warp == 0) {                                              // a wait gave up: let the copies in flight land, within bounds
    for (int k = max(0, fetched - NST + 1); k <= fetched; ++k) mbar_wait(&full[k % NST], (k / NST) & 1, 1u << 16);
  }
  zero_empty_rows();
}

template <int RH, int MT>
static int launch_latent_decode(const CUtensorMap& map, const LatentDecodeParams& p, int num_ctas, cudaStream_t st) {
  using C = LatentCfg<RH, MT>;
  struct Tag {};
  const int rc = opt_in_dynamic_smem<Tag>(reinterpret_cast<const void*>(&latent_decode_kernel<RH, MT>), C::SMEM);
  if (rc != kOk) return rc;
  latent_decode_kernel<RH, MT><<<dim3(num_ctas, (p.heads + C::HEADS - 1) / C::HEADS), 512, C::SMEM, st>>>(map, p);
  return cudaGetLastError() == cudaSuccess ? kOk : kLaunchFailed;
}
template <int RH>
static int launch_latent_width(const CUtensorMap& map, const LatentDecodeParams& p, int num_ctas, cudaStream_t st) {
  return p.heads <= 16 ? launch_latent_decode<RH, 1>(map, p, num_ctas, st) : launch_latent_decode<RH, 2>(map, p, num_ctas, st);
}

static bool latent_width_ok(int width) {                                 // the instances there are
  for (int w : {64, 128, 192, 256, 384, 512})
    if (width == w) return true;
  return false;
}

static int plan_ctas() { return sm_count() < kMaxCtas ? sm_count() : kMaxCtas; }

}  // namespace mvb

extern "C" int mvb_latent_norm(int dtype, const void* q, int64_t q_row_stride, const void* q_weight, void* q_out, int q_cols, int q_pad,
                               const void* c, int64_t c_row_stride, const void* c_weight, void* c_out, int c_cols, int c_pad, void* cache,
                               const int32_t* slot_mapping, int64_t num_slots, int num_tokens, float eps, int32_t* dev_status,
                               void* stream) {
  using namespace mvb;
  if (!q || !q_weight || !q_out || num_tokens < 0 || q_cols <= 0 || q_pad < q_cols || (dtype != kBf16 && dtype != kF32)) return kInvalidArgument;
  if (c != nullptr && (!c_weight || !c_out || c_cols <= 0 || c_pad < c_cols)) return kInvalidArgument;
  if (cache != nullptr && (c == nullptr || !slot_mapping || num_slots <= 0)) return kInvalidArgument;
  if (num_tokens == 0) return kOk;
  const LatentNormParams p{q, q_row_stride, q_weight, q_out, q_cols, q_pad, c, c_row_stride, c_weight, c_out, c_cols, c_pad,
                           cache, slot_mapping, num_slots, num_tokens, eps, dev_status};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return dtype == kBf16 ? launch_latent_norm<__nv_bfloat16>(p, st) : launch_latent_norm<float>(p, st);
}

extern "C" int mvb_gather_latents(const void* cache, int64_t num_slots, int row_bytes, const int32_t* block_table, int64_t table_stride,
                                  int table_width, int block_size, const int32_t* cu_seqlens_k, int num_seqs, int num_rows, void* out,
                                  int32_t* dev_status, void* stream) {
  using namespace mvb;
  if (!cache || !block_table || !cu_seqlens_k || !out || num_slots <= 0 || row_bytes <= 0 || table_width <= 0 || block_size <= 0 ||
      num_seqs <= 0 || num_rows < 0)
    return kInvalidArgument;
  if (row_bytes % 16 != 0 || !is_aligned(cache, 16) || !is_aligned(out, 16)) return kMisaligned;
  if (num_rows == 0) return kOk;
  const int64_t blocks = (static_cast<int64_t>(num_rows) * 32 + 255) / 256;
  gather_latents_kernel<<<static_cast<unsigned>(blocks), 256, 0, static_cast<cudaStream_t>(stream)>>>(
      static_cast<const uint4*>(cache), num_slots, row_bytes / 16, block_table, table_stride, table_width, block_size, cu_seqlens_k, num_seqs,
      num_rows, static_cast<uint4*>(out), dev_status);
  return cudaGetLastError() == cudaSuccess ? kOk : kLaunchFailed;
}

extern "C" int mvb_gate_mul(int dtype, const void* o, int64_t o_row_stride, const void* gate, int64_t gate_row_stride, void* out,
                            int64_t out_row_stride, int rows, int cols, void* stream) {
  using namespace mvb;
  if (!o || !gate || !out || rows < 0 || cols <= 0 || (dtype != kBf16 && dtype != kF32)) return kInvalidArgument;
  if (rows == 0) return kOk;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return dtype == kBf16 ? launch_gate<__nv_bfloat16>(o, o_row_stride, gate, gate_row_stride, out, out_row_stride, rows, cols, st)
                        : launch_gate<float>(o, o_row_stride, gate, gate_row_stride, out, out_row_stride, rows, cols, st);
}

extern "C" int mvb_latent_decode_plan(const int32_t* cache_seqlens, const int32_t* block_table, int64_t table_stride, int block_size,
                                      int num_seqs, int num_heads, int width, void* workspace, size_t workspace_bytes, void* stream) {
  using namespace mvb;
  if (!cache_seqlens || !block_table || !workspace || num_seqs <= 0 || num_heads <= 0 || block_size <= 0 || table_stride <= 0) return kInvalidArgument;
  const DecodeLayout l = decode_layout(num_seqs, num_heads, width);
  if (workspace_bytes < l.total || !is_aligned(workspace, 256)) return kInvalidArgument;
  uint8_t* ws = static_cast<uint8_t*>(workspace);
  decode_plan_kernel<<<1, kPlanThreads, 0, static_cast<cudaStream_t>(stream)>>>(
      cache_seqlens, num_seqs, -1, kLatentTile, plan_ctas(), num_seqs * num_heads, block_table, table_stride, block_size,
      reinterpret_cast<DecodeHeader*>(ws), reinterpret_cast<CtaDesc*>(ws + l.descs), reinterpret_cast<int32_t*>(ws + l.tile_prefix));
  return cudaGetLastError() == cudaSuccess ? kOk : kLaunchFailed;
}

extern "C" int mvb_latent_decode(const void* q, int64_t q_row_stride, int64_t q_head_stride, const void* cache, int64_t num_blocks,
                                 int block_size, const int32_t* cache_seqlens, const int32_t* block_table, int64_t table_stride,
                                 int table_width, int num_seqs, int num_heads, int width, float scale, void* out, int64_t out_row_stride,
                                 int64_t out_head_stride, void* workspace, size_t workspace_bytes, int32_t* dev_status, void* stream) {
  using namespace mvb;
  if (!q || !cache || !cache_seqlens || !block_table || !out || !workspace) return kInvalidArgument;
  if (num_seqs <= 0 || num_heads <= 0 || num_blocks <= 0 || block_size <= 0 || table_width <= 0 || table_stride < table_width) return kInvalidArgument;
  if (!latent_width_ok(width) || block_size % kLatentTile != 0 || num_blocks * block_size > 0x7fffffffLL) return kUnsupportedShape;
  if (q_row_stride % 8 || q_head_stride % 8 || out_row_stride % 4 || out_head_stride % 4 || !is_aligned(q, 16) || !is_aligned(out, 8) || !is_aligned(cache, 16))
    return kMisaligned;
  const DecodeLayout l = decode_layout(num_seqs, num_heads, width);
  if (workspace_bytes < l.total || !is_aligned(workspace, 256)) return kInvalidArgument;
  CUtensorMap map;
  const int rc = make_kv_tensor_map(&map, cache, num_blocks * block_size, 1, width, width, kLatentTile);
  if (rc != kOk) return rc;
  uint8_t* ws = static_cast<uint8_t*>(workspace);
  LatentDecodeParams p{};
  p.q = static_cast<const __nv_bfloat16*>(q); p.q_stride = q_row_stride; p.q_head_stride = q_head_stride;
  p.out = static_cast<__nv_bfloat16*>(out); p.out_stride = out_row_stride; p.out_head_stride = out_head_stride;
  p.cache_seqlens = cache_seqlens; p.block_table = block_table; p.table_stride = table_stride; p.table_width = table_width;
  p.num_seqs = num_seqs; p.heads = num_heads; p.block_size = block_size; p.num_blocks = num_blocks;
  p.scale_log2 = scale * 1.4426950408889634f;
  p.descs = reinterpret_cast<const CtaDesc*>(ws + l.descs);
  p.tile_prefix = reinterpret_cast<const int32_t*>(ws + l.tile_prefix);
  p.part_lse = reinterpret_cast<float*>(ws + l.lse); p.part_o = reinterpret_cast<float*>(ws + l.o);
  p.arrivals = reinterpret_cast<int32_t*>(ws + l.tile_prefix) + num_seqs + 1;
  p.dev_status = dev_status;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const int n = plan_ctas();
  switch (width / 64) {
    case 1: return launch_latent_width<1>(map, p, n, st);
    case 2: return launch_latent_width<2>(map, p, n, st);
    case 3: return launch_latent_width<3>(map, p, n, st);
    case 4: return launch_latent_width<4>(map, p, n, st);
    case 6: return launch_latent_width<6>(map, p, n, st);
    default: return launch_latent_width<8>(map, p, n, st);
  }
}
