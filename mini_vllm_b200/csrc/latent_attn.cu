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
// latent_decode_kernel: persistent CTAs over the tile ranges of decode_plan.cuh, eight working warps and one that fetches.  A tile = 64
// tokens x width in two halves of 32 tokens, 128-byte-swizzled in shared memory; a half is one TMA copy through the block table (its
// tensor map has the 64-column blocks of a row as a dimension), and the ring holds NH of them.  Per tile, three barriers of the
// working warps:
//   scores   S[heads x 64] = Q' C^T     warp = 32 tokens x a quarter of the width (mma.sync, heads in M; the queries stay in registers);
//                                       the quarters meet in shared memory
//   softmax  a few threads per head, running maximum and sum in registers, P as bf16 through shared memory
//   output   O[heads x width] += P C    warp = an eighth of the width (C again, as transposed fragments), O in registers
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
constexpr int kLatentTile = 64, kLatentHalf = 32;
constexpr int kLatentMergeTiles = 12;           // what a partial + arrival + merge costs a CTA, in tiles of streaming (decode_plan.cuh)

constexpr int kLatentHeads = 16;                // heads per CTA

template <int RH>                               // width = 64 RH
struct LatentCfg {
  static constexpr int W = 64 * RH, HEADS = kLatentHeads, TOK = kLatentTile;
  static constexpr int COLS = kLatentHalf * 128, HALF = RH * COLS;      // 32 tokens x 64 columns; 32 tokens
  static constexpr int SROW = TOK + 4, PROW = TOK * 2 + 16;
  static constexpr int SB = 4 * HEADS * SROW * 4, P = HEADS * PROW, ROWS = 3 * HEADS * 4;
  static constexpr int FIXED = SB + P + ROWS + 128;                     // (eight full and eight empty barriers at most)
  static constexpr int FIT = (226 * 1024 - 1024 - FIXED) / HALF;
  static constexpr int NH = FIT > 8 ? 8 : FIT;
  static constexpr int SMEM = 1024 + NH * HALF + FIXED;
  static_assert(NH >= 5, "a tile in use and more than one in flight");
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

// barriers of the working warps
__device__ __forceinline__ void workers_sync() { asm volatile("barrier.cta.sync.aligned 1, 256;" ::: "memory"); }
__device__ __forceinline__ bool workers_all(bool ok) {
  uint32_t r;
  asm volatile(
      "{\n\t.reg .pred p, q;\n\t"
      "setp.ne.u32 q, %1, 0;\n\t"
      "barrier.cta.red.and.aligned.pred p, 1, 256, q;\n\t"
      "selp.u32 %0, 1, 0, p;\n\t}"
      : "=r"(r) : "r"(static_cast<uint32_t>(ok)) : "memory");
  return r != 0;
}

template <int RH>
__global__ void __launch_bounds__(288, 1) latent_decode_kernel(const __grid_constant__ CUtensorMap map, const LatentDecodeParams p) {
  using C = LatentCfg<RH>;
  constexpr int TOK = C::TOK, NH = C::NH, W = C::W, HEADS = C::HEADS;
  constexpr uint32_t FULL = 0xffffffffu;
  extern __shared__ uint8_t smem_raw[];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, c = blockIdx.x;
  const int head0 = blockIdx.y * HEADS, nheads = min(HEADS, p.heads - head0);
  const CtaDesc desc = p.descs[c];
  auto zero_empty_rows = [&]() {                                        // one warp
    for (int b = c; b < p.num_seqs; b += gridDim.x)
      if (p.cache_seqlens[b] <= 0)
        for (int e = lane; e < nheads * W; e += 32)
          p.out[b * p.out_stride + (head0 + e / W) * p.out_head_stride + e % W] = __float2bfloat16_rn(0.f);
  };
  if (desc.t0 >= desc.t1) {
    if (warp == 0) zero_empty_rows();
    return;
  }

  const uint32_t base = (smem_u32(smem_raw) + 1023u) & ~1023u;
  uint8_t* base_ptr = smem_raw + (base - smem_u32(smem_raw));
  float* s_s = reinterpret_cast<float*>(base_ptr + NH * C::HALF);       // [quarter][HEADS][SROW]; weights of the parts in a merge
  uint8_t* p_s = base_ptr + NH * C::HALF + C::SB;                       // [HEADS][PROW bytes]
  float* alpha_s = reinterpret_cast<float*>(p_s + C::P);                // [HEADS]; behind it the final l and m
  float *l_s = alpha_s + HEADS, *m_s = l_s + HEADS;
  uint64_t *full = reinterpret_cast<uint64_t*>(m_s + HEADS), *empty = full + 8;
  const uint32_t p_base = smem_u32(p_s);
  if (tid == 0) {
    tma_prefetch_desc(&map);
    for (int i = 0; i < NH; ++i) { mbar_init(&full[i], 1); mbar_init(&empty[i], 8); }
    fence_mbar_init();
  }
  __syncthreads();

  SeqSpan cs{desc.b, desc.tp0, desc.tp1, desc.n};
  auto next_seq = [&](SeqSpan& v) {
    ++v.b; v.tp0 = p.tile_prefix[v.b]; v.tp1 = p.tile_prefix[v.b + 1]; v.n = p.cache_seqlens[v.b];
  };
  // ---- the fetching warp: halves are counted from desc.t0, half i lives in place i % NH ----
  const int total = 2 * (desc.t1 - desc.t0);
  if (warp == 8) {
    int blk_base = -1, blk_reg = -1, blk_n = 0, i = 0;
    if (desc.blk0 >= 0) { blk_base = (desc.t0 - desc.tp0) * TOK / p.block_size; blk_reg = desc.blk0; blk_n = 1; }
    for (; i < total; ++i) {
      const int t = desc.t0 + (i >> 1);
      while (t >= cs.tp1 && cs.b + 1 < p.num_seqs) { next_seq(cs); blk_base = -1; blk_n = 0; }
      const int token0 = (t - cs.tp0) * TOK + (i & 1) * kLatentHalf, bi = token0 / p.block_size;
      if (blk_base < 0 || bi < blk_base || bi >= blk_base + blk_n) {
        blk_base = bi; blk_n = 32;
        const int col = bi + lane;
        blk_reg = col < p.table_width ? p.block_table[cs.b * p.table_stride + col] : -1;
      }
      const int blk = __shfl_sync(FULL, blk_reg, bi - blk_base), st = i % NH;
      int slot0 = -kLatentHalf;                                         // out of range: TMA fills zeros
      if (blk >= 0 && blk < p.num_blocks) slot0 = blk * p.block_size + (token0 - bi * p.block_size);
      else if (lane == 0) report(p.dev_status, kDevBadBlock, cs.b);
      if (i >= NH && !__all_sync(FULL, mbar_wait(&empty[st], (i / NH - 1) & 1))) {      // the working warps have given up
        if (lane == 0) report(p.dev_status, kDevWaitTimeout, i);
        break;
      }
      if (lane == 0) {
        mbar_arrive_expect_tx(&full[st], C::HALF);
        tma_load_3d(base_ptr + st * C::HALF, &map, &full[st], 0, slot0, 0);
      }
    }
    if (i < total)                                                      // let the copies in flight land, within bounds
      for (int k = max(0, i - NH); k < i; ++k) mbar_wait(&full[k % NH], (k / NH) & 1, 1u << 16);
    zero_empty_rows();
    return;
  }

  const int first_b = cs.b;
  int t = 0;                                                            // tile, from desc.t0
  bool ok = true;
  const int tg = warp & 1, kq = warp >> 1, mi = lane >> 3;              // scores: half of the tile, quarter of the width
  constexpr int TPR = 256 / HEADS, TPT = TOK / TPR;                     // softmax: threads per head, tokens per thread
  const int srow = tid / TPR, ssub = tid % TPR, ntiles = total / 2;
  while (t < ntiles && ok) {
    while (desc.t0 + t >= cs.tp1 && cs.b + 1 < p.num_seqs) next_seq(cs);
    const int seg_end = min(desc.t1, cs.tp1) - desc.t0, b = cs.b;
    const bool whole = desc.t0 + t == cs.tp0 && desc.t0 + seg_end == cs.tp1;
    uint32_t qa[RH][4];                                             // this warp's quarter of the queries, as first operand
    {
      const __nv_bfloat16* q = p.q + b * p.q_stride + static_cast<int64_t>(head0) * p.q_head_stride + kq * RH * 16 + (lane & 3) * 2;
#pragma unroll
      for (int k = 0; k < RH; ++k)
#pragma unroll
        for (int r = 0; r < 4; ++r) {
          const int h = (lane >> 2) + (r & 1) * 8;
          qa[k][r] = h < nheads ? *reinterpret_cast<const uint32_t*>(q + h * p.q_head_stride + k * 16 + (r >> 1) * 8) : 0u;
        }
    }
    float o[RH][4];
#pragma unroll
    for (int n = 0; n < RH; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
    float m_run = -INFINITY, l_run = 0.f;
    // scores of tile u into s_s; false: its half did not arrive
    auto scores = [&](int u) -> bool {
      const int i = 2 * u + tg;
      const bool here = mbar_wait(&full[i % NH], (i / NH) & 1);
      const uint32_t half = base + (i % NH) * C::HALF;
      float s[4][4];
#pragma unroll
      for (int n = 0; n < 4; ++n) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f;
      const int tok = (lane & 7) + (mi >> 1) * 8;
      const uint32_t trow = half + tok * 128;
#pragma unroll
      for (int k = 0; k < RH; ++k) {
        const int chunk = (kq * RH + k) * 2 + (mi & 1);
        const uint32_t at = trow + (chunk >> 3) * C::COLS + (((chunk & 7) ^ (tok & 7)) << 4);
        uint32_t c0[4], c1[4];
        ldmatrix_x4(c0, at);
        ldmatrix_x4(c1, at + 16 * 128);
        mma_bf16_16816(s[0], qa[k], c0[0], c0[1]);
        mma_bf16_16816(s[1], qa[k], c0[2], c0[3]);
        mma_bf16_16816(s[2], qa[k], c1[0], c1[1]);
        mma_bf16_16816(s[3], qa[k], c1[2], c1[3]);
      }
#pragma unroll
      for (int n = 0; n < 4; ++n) {
        float* d = s_s + (kq * HEADS + (lane >> 2)) * C::SROW + tg * 32 + n * 8 + (lane & 3) * 2;
        *reinterpret_cast<float2*>(d) = make_float2(s[n][0], s[n][1]);
        *reinterpret_cast<float2*>(d + 8 * C::SROW) = make_float2(s[n][2], s[n][3]);
      }
      return here;
    };
    for (; t < seg_end; ++t) {
      const bool here = scores(t);
      ok = workers_all(here);
      if (!ok) {
        if (!here) report(p.dev_status, kDevWaitTimeout, t);
        break;
      }
      const int valid = cs.n - (desc.t0 + t - cs.tp0) * TOK;
      if (valid < TOK) {                                                // rows behind the end may hold anything: zero them for P C
        for (int e = tid; e < (TOK - valid) * RH * 8; e += 256) {
          const int r = valid + e / (RH * 8), k = e % (RH * 8);
          *reinterpret_cast<uint4*>(base_ptr + (2 * t + (r >> 5)) % NH * C::HALF + (k >> 3) * C::COLS + (r & 31) * 128 + (k & 7) * 16) = make_uint4(0u, 0u, 0u, 0u);
        }
        fence_proxy_async();                                            // (a copy will go over them)
      }
      {                                                                 // softmax
        float x[TPT], top = -INFINITY;
        const float* r0 = s_s + srow * C::SROW + ssub * TPT;
#pragma unroll
        for (int j = 0; j < TPT; j += 4) {
          float4 a = *reinterpret_cast<const float4*>(r0 + j);
#pragma unroll
          for (int k = 1; k < 4; ++k) {
            const float4 d = *reinterpret_cast<const float4*>(r0 + k * HEADS * C::SROW + j);
            a.x += d.x; a.y += d.y; a.z += d.z; a.w += d.w;
          }
          x[j] = a.x; x[j + 1] = a.y; x[j + 2] = a.z; x[j + 3] = a.w;
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
        l_run = l_run * alpha + sum;                                    // (of this thread's tokens; the row meets at the end)
        m_run = m_new;
#pragma unroll
        for (int j = 0; j < TPT; j += 4)
          *reinterpret_cast<uint2*>(p_s + srow * C::PROW + (ssub * TPT + j) * 2) = make_uint2(pack_bf16(x[j], x[j + 1]), pack_bf16(x[j + 2], x[j + 3]));
        if (ssub == 0) alpha_s[srow] = alpha;
      }
      workers_sync();
      {                                                                 // output
        const uint32_t prow = p_base + ((lane & 7) + (mi & 1) * 8) * C::PROW + (lane >> 4) * 16;
        const float a0 = alpha_s[lane >> 2], a1 = alpha_s[(lane >> 2) + 8];
#pragma unroll
        for (int n = 0; n < RH; ++n) { o[n][0] *= a0; o[n][1] *= a0; o[n][2] *= a1; o[n][3] *= a1; }
#pragma unroll
        for (int k = 0; k < 2; ++k) {
          uint32_t pa[2][4];
          ldmatrix_x4(pa[0], prow + k * 64);
          ldmatrix_x4(pa[1], prow + k * 64 + 32);
          const uint32_t trow = base + (2 * t + k) % NH * C::HALF + lane * 128;        // a lane addresses its token: two 16-token steps
#pragma unroll
          for (int n = 0; n < RH; ++n) {
            const int chunk = warp * RH + n;
            uint32_t cb[4];
            ldmatrix_x4_trans(cb, trow + (chunk >> 3) * C::COLS + (((chunk & 7) ^ (lane & 7)) << 4));
            mma_bf16_16816(o[n], pa[0], cb[0], cb[1]);
            mma_bf16_16816(o[n], pa[1], cb[2], cb[3]);
          }
        }
      }
      __syncwarp();
      if (lane == 0) { mbar_arrive(&empty[2 * t % NH]); mbar_arrive(&empty[(2 * t + 1) % NH]); }
    }
    if (!ok) break;
    // ---- end of the segment: output, or a partial result ----
#pragma unroll
    for (int off = 1; off < TPR; off <<= 1) l_run += __shfl_xor_sync(FULL, l_run, off);
    if (ssub == 0) { l_s[srow] = l_run; m_s[srow] = m_run; }
    workers_sync();
    const int part = b == first_b ? 0 : 1;
#pragma unroll
    for (int r = 0; r < 2; ++r) {
      const int h = (lane >> 2) + r * 8;
      if (h >= nheads) continue;
      const float inv = l_s[h] > 0.f ? 1.f / l_s[h] : 0.f;
#pragma unroll
      for (int n = 0; n < RH; ++n) {
        const int col = (warp * RH + n) * 8 + (lane & 3) * 2;
        const float x = o[n][2 * r] * inv, y = o[n][2 * r + 1] * inv;
        if (whole) *reinterpret_cast<uint32_t*>(p.out + b * p.out_stride + (head0 + h) * p.out_head_stride + col) = pack_bf16(x, y);
        else *reinterpret_cast<float2*>(p.part_o + ((static_cast<int64_t>(c) * 2 + part) * p.heads + head0 + h) * W + col) = make_float2(x, y);
      }
    }
    if (!whole) {
      __shared__ int is_last;
      if (tid < nheads) p.part_lse[(static_cast<int64_t>(c) * 2 + part) * p.heads + head0 + tid] = m_s[tid] + log2f(l_s[tid]);
      const int per = desc.per, c1 = cs.tp0 / per, c2 = (cs.tp1 - 1) / per, nparts = c2 - c1 + 1;
      // the CTA barrier orders every thread's partial stores before thread 0's release; the last arriver's acquire plus its CTA
      // barrier order them before every merging thread's loads
      workers_sync();
      if (tid == 0) {
        int32_t* cnt = p.arrivals + static_cast<int64_t>(b) * gridDim.y + blockIdx.y;
        int prev;
        asm volatile("atom.acq_rel.gpu.global.add.s32 %0, [%1], 1;" : "=r"(prev) : "l"(cnt) : "memory");
        is_last = prev == nparts - 1;
        if (is_last) *cnt = 0;                                          // re-arm for the next launch
      }
      workers_sync();
      if (is_last) {
        const bool first_is_head = cs.tp0 % per == 0;                   // does CTA c1's range start at this sequence?
        auto part_index = [&](int j, int h) -> int64_t {
          return ((static_cast<int64_t>(c1 + j) * 2 + (j > 0 || first_is_head ? 0 : 1)) * p.heads) + head0 + h;
        };
        static_assert((kMaxPartsPerSeq + 2) * HEADS <= C::SB / 4, "a weight per part and head fits the score buffer");
        for (int e = tid; e < nparts * nheads; e += 256) s_s[e] = __ldcg(p.part_lse + part_index(e / nheads, e % nheads));
        workers_sync();
        if (tid < nheads) {
          float top = -INFINITY, sum = 0.f;
          for (int j = 0; j < nparts; ++j) top = fmaxf(top, s_s[j * nheads + tid]);
          for (int j = 0; j < nparts; ++j) { const float w = fast_exp2(s_s[j * nheads + tid] - top); s_s[j * nheads + tid] = w; sum += w; }
          l_s[tid] = 1.f / sum;
        }
        workers_sync();
        constexpr int ITEMS = (HEADS * W / 4 + 255) / 256, GROUP = ITEMS < 8 ? ITEMS : 8;
#pragma unroll 1
        for (int k0 = 0; k0 < ITEMS; k0 += GROUP) {
          float4 acc[GROUP];
#pragma unroll
          for (int k = 0; k < GROUP; ++k) acc[k] = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 2
          for (int j = 0; j < nparts; ++j) {                            // a part's loads are independent: they pipeline
            const float* src = p.part_o + part_index(j, 0) * W;
#pragma unroll
            for (int k = 0; k < GROUP; ++k) {
              const int e = (tid + (k0 + k) * 256) * 4, h = e / W;
              if (h >= nheads) continue;
              const float w = s_s[j * nheads + h];
              const float4 v = __ldcg(reinterpret_cast<const float4*>(src + e));
              acc[k].x = fmaf(w, v.x, acc[k].x); acc[k].y = fmaf(w, v.y, acc[k].y);
              acc[k].z = fmaf(w, v.z, acc[k].z); acc[k].w = fmaf(w, v.w, acc[k].w);
            }
          }
#pragma unroll
          for (int k = 0; k < GROUP; ++k) {
            const int e = (tid + (k0 + k) * 256) * 4, h = e / W;
            if (h >= nheads) continue;
            const float w = l_s[h];
            *reinterpret_cast<uint2*>(p.out + b * p.out_stride + (head0 + h) * p.out_head_stride + e % W) =
                make_uint2(pack_bf16(acc[k].x * w, acc[k].y * w), pack_bf16(acc[k].z * w, acc[k].w * w));
          }
        }
      }
    }
    workers_sync();                                                    // l, m and the score buffer are about to be written again
  }
}

static int head_groups(int heads) { return (heads + kLatentHeads - 1) / kLatentHeads; }

template <int RH>
static int launch_latent_decode(const CUtensorMap& map, const LatentDecodeParams& p, int num_ctas, cudaStream_t st) {
  using C = LatentCfg<RH>;
  struct Tag {};
  const int rc = opt_in_dynamic_smem<Tag>(reinterpret_cast<const void*>(&latent_decode_kernel<RH>), C::SMEM);
  if (rc != kOk) return rc;
  latent_decode_kernel<RH><<<dim3(num_ctas, head_groups(p.heads)), 288, C::SMEM, st>>>(map, p);
  return cudaGetLastError() == cudaSuccess ? kOk : kLaunchFailed;
}
// the pool as [64-column blocks, slots, 64 columns], so that one box is 32 tokens with all their columns, block after block
static int make_latent_map(CUtensorMap* map, const void* base, int64_t rows, int width) {
  EncodeTiledFn fn = encode_tiled_fn();
  if (fn == nullptr) return kNoDriverEntry;
  const cuuint64_t dims[3] = {64, static_cast<cuuint64_t>(rows), static_cast<cuuint64_t>(width / 64)};
  const cuuint64_t strides[2] = {static_cast<cuuint64_t>(width) * 2, 128};
  const cuuint32_t box[3] = {64, kLatentHalf, static_cast<cuuint32_t>(width / 64)}, estr[3] = {1, 1, 1};
  const CUresult r = fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(base), dims, strides, box, estr,
                        CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                        CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  return r == CUDA_SUCCESS ? kOk : kTensorMapFailed;
}

static bool latent_width_ok(int width) {                                 // the instances there are
  for (int w : {64, 128, 192, 256, 384, 512})
    if (width == w) return true;
  return false;
}

// the groups of heads share the SMs, so that all of them stream the same ranges at the same time and meet in L2
static int latent_ctas(int heads) {
  const int n = (sm_count() < kMaxCtas ? sm_count() : kMaxCtas) / head_groups(heads);
  return n > 1 ? n : 1;
}

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
      cache_seqlens, num_seqs, -1, 0, kLatentTile, kLatentMergeTiles, latent_ctas(num_heads), num_seqs * num_heads, block_table, table_stride, block_size,
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
  const int rc = make_latent_map(&map, cache, num_blocks * block_size, width);
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
  const int n = latent_ctas(num_heads);
  switch (width / 64) {
    case 1: return launch_latent_decode<1>(map, p, n, st);
    case 2: return launch_latent_decode<2>(map, p, n, st);
    case 3: return launch_latent_decode<3>(map, p, n, st);
    case 4: return launch_latent_decode<4>(map, p, n, st);
    case 6: return launch_latent_decode<6>(map, p, n, st);
    default: return launch_latent_decode<8>(map, p, n, st);
  }
}
