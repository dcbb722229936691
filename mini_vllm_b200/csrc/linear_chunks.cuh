// Linear attention with decay over chunks of 16 tokens on the tensor cores (ragged steps with bf16 activations).
//
// Channel decay: with A_ts = a_{s+1} .. a_t (per key channel) inside a chunk, and the chunk's initial S0:
//   o_t = (q_t A_t0) S0 + sum_{s <= t} B_ts v_s             B_ts = sum_d q_t k_s A_ts
//   S  <- A_{16,0} S0 + sum_s (k_s A_{16,s}) v_s^T
// Exponential gates: F_t = sum_{s <= t} f_s (a scalar per head), M_t = max_{s <= t} (F_t - F_s + i_s), m_t = max(F_t + m_0, M_t):
//   o_t = e^{F_t + m_0 - m_t} q_t S0 + e^{M_t - m_t} sum_{s <= t} B_ts v_s          B_ts = (q_t . k_s) e^{F_t - F_s + i_s - M_t}
//   S  <- e^{F_16 + m_0 - m_16} S0 + e^{M_16 - m_16} sum_s (k_s e^{F_16 - F_s + i_s - M_16}) v_s^T,    n likewise with v = 1
// B, M and the scaled keys do not depend on what came before the chunk; only the row factors do, through the one scalar m_0.
// All factors are <= 1, whatever the gates are.
//
// The prep kernels (parallel over chunks and heads) leave one contiguous record per (chunk, head) with everything the recurrence
// needs, already in the register order of mma.sync operands.  linear_chunk_scan (sequential over the chunks of a sequence, parallel
// over heads and 16-column tiles) keeps S^T in the fp32 accumulator registers of one warp per 16 columns, whose fragments are operand
// fragments of the next product as they stand; records arrive by bulk copies, several chunks ahead.  With exponential gates one more warp
// carries the normaliser and the maximum, in plain fp32.
// v (and, with exponential gates, q) is a bf16 projection and enters exactly; every other operand enters as bf16 high + low part:
// 16 significant bits per factor with fp32 accumulation.  The state itself is never rounded below fp32.
#pragma once
#include "chunk_common.cuh"

namespace mvb {

struct LinearLayout {             // bytes inside a record
  int k, b, extra, v, total;      // q at 0; extra: decay of the chunk per key channel, or F, M, row sums of B, and sums of scaled keys
};
__host__ __device__ inline LinearLayout linear_layout(int ks, int vtp, bool exp_gates) {
  LinearLayout l;
  l.k = ks * (exp_gates ? 512 : 1024);
  l.b = l.k + ks * 1024;
  l.extra = l.b + 1024;
  l.v = l.extra + (exp_gates ? 192 : 0) + ks * 64;
  l.total = l.v + vtp * 512;
  return l;
}

static inline int linear_warps(const LinearParams& p) {       // 16-column tiles per CTA
  const int tiles = (p.vdim + 15) / 16;
  // few (sequence, head) pairs: one warp per CTA, so that they spread over the SMs
  if (static_cast<int64_t>(tiles) * p.heads * p.num_seqs <= sm_count() * 2) return 1;
  int best = 4;
  for (int w = 4; w >= 2; --w)
    if ((tiles + w - 1) / w * w < (tiles + best - 1) / best * best) best = w;
  return tiles == 1 ? 1 : best;
}
static inline int linear_tiles(const LinearParams& p) {
  const int tiles = (p.vdim + 15) / 16, w = linear_warps(p);
  return (tiles + w - 1) / w * w;
}

struct ChunkSite { int seq, row, n; };        // the sequence, first row and token count of a chunk slot; n = 0: an unused slot
__device__ __forceinline__ ChunkSite chunk_site(const LinearParams& p, int slot) {
  int lo = 0, hi = p.num_seqs;
  while (hi - lo > 1) {
    const int mid = (lo + hi) >> 1;
    if (chunk_base(p.cu[mid], mid) <= slot) lo = mid; else hi = mid;
  }
  const int begin = p.cu[lo], t0 = (slot - chunk_base(begin, lo)) * kChunk;
  return {lo, begin + t0, min(kChunk, p.cu[lo + 1] - begin - t0)};
}

__device__ __forceinline__ float bf_at(const void* base, int64_t i) { return __bfloat162float(static_cast<const __nv_bfloat16*>(base)[i]); }

// v of a chunk as [16][cols] bf16 in shared memory: zeros behind the tokens and columns there are
__device__ __forceinline__ void stage_values(const LinearParams& p, const ChunkSite& c, int h, int cols, __nv_bfloat16* v_s) {
  const __nv_bfloat16* v = static_cast<const __nv_bfloat16*>(p.v) + c.row * p.qkv_stride + static_cast<int64_t>(h) * p.vdim;
  if (p.vdim % 8 == 0 && p.qkv_stride % 8 == 0 && (reinterpret_cast<uintptr_t>(p.v) & 15) == 0) {
    const int vec = cols / 8;
    for (int e = threadIdx.x; e < kChunk * vec; e += blockDim.x) {
      const int t = e / vec, col = (e % vec) * 8;
      uint4 w = make_uint4(0u, 0u, 0u, 0u);
      if (t < c.n && col < p.vdim) w = *reinterpret_cast<const uint4*>(v + t * p.qkv_stride + col);
      *reinterpret_cast<uint4*>(v_s + t * cols + col) = w;
    }
  } else {
    for (int e = threadIdx.x; e < kChunk * cols; e += blockDim.x) {
      const int t = e / cols, col = e % cols;
      v_s[e] = t < c.n && col < p.vdim ? v[t * p.qkv_stride + col] : __float2bfloat16_rn(0.f);
    }
  }
}
// the values as first operand of V^T (.): rows = columns of v, k = tokens
__device__ __forceinline__ void write_values(const __nv_bfloat16* v_s, int cols, uint8_t* dst) {
  const uint16_t* v = reinterpret_cast<const uint16_t*>(v_s);
  auto two = [&](int t, int c) { return static_cast<uint32_t>(v[t * cols + c]) | static_cast<uint32_t>(v[(t + 1) * cols + c]) << 16; };
  for (int i = threadIdx.x; i < cols / 16 * 32; i += blockDim.x) {
    const int ln = i & 31, t = (ln & 3) * 2, c = (i >> 5) * 16 + (ln >> 2);
    reinterpret_cast<uint4*>(dst)[i] = make_uint4(two(t, c), two(t, c + 8), two(t + 8, c), two(t + 8, c + 8));
  }
}
// B as second operand of (.) B^T; at(t, s) for s <= t, one warp
template <class F>
__device__ __forceinline__ void write_triangle(F at, int lane, uint8_t* dst) {
#pragma unroll
  for (int n = 0; n < 2; ++n) {
    const int t = n * 8 + (lane >> 2), s = (lane & 3) * 2;
    auto below = [&](int c) { return c <= t ? at(t, c) : 0.f; };
    uint4 w;
    split_pair(below(s), below(s + 1), w.x, w.z);
    split_pair(below(s + 8), below(s + 9), w.y, w.w);
    reinterpret_cast<uint4*>(dst)[n * 32 + lane] = w;
  }
}
// scaled keys k_s [16][row] (fp32) as second operand of V^T K: 8-channel tiles
__device__ __forceinline__ void write_keys(const float* k_s, int row, int ks, uint8_t* dst) {
  for (int i = threadIdx.x; i < ks * 64; i += blockDim.x) {
    const int ln = i & 31, d = (i >> 5) * 8 + (ln >> 2), t = (ln & 3) * 2;
    uint4 o;
    split_pair(k_s[t * row + d], k_s[(t + 1) * row + d], o.x, o.z);
    split_pair(k_s[(t + 8) * row + d], k_s[(t + 9) * row + d], o.y, o.w);
    reinterpret_cast<uint4*>(dst)[i] = o;
  }
}

// ---- channel decay ----------------------------------------------------------------------------------------
template <int KS>
__global__ void __launch_bounds__(128, KS <= 8 ? 7 : 3) decay_chunk_prep(const LinearParams p) {
  constexpr int D32 = (16 * KS + 31) / 32 * 32, ROW = D32 + 4, NI = D32 / 32;
  extern __shared__ __align__(16) float sm[];
  float* q_s = sm;                               // [16][ROW]
  float* k_s = q_s + kChunk * ROW;
  float* a_s = k_s + kChunk * ROW;               // decay factors
  __nv_bfloat16* v_s = reinterpret_cast<__nv_bfloat16*>(a_s + kChunk * ROW);
  __shared__ float bm[kChunk][kChunk + 1];
  const int h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const ChunkSite c = chunk_site(p, blockIdx.x);
  if (c.n <= 0) return;
  const LinearLayout lay = linear_layout(KS, p.vtp, false);
  uint8_t* rec = p.records + (static_cast<int64_t>(blockIdx.x) * p.heads + h) * lay.total;

  // a warp takes every fourth token; the raw operands of U tokens are requested before any is worked on
  constexpr int U = 2;
  const float to_log2 = p.inv_tau * kLog2e;
  float bias[NI];
#pragma unroll
  for (int i = 0; i < NI; ++i) bias[i] = i * 32 + lane < p.dim ? p.decay_bias[h * p.dim + i * 32 + lane] : 0.f;
  stage_values(p, c, h, p.vtp * 16, v_s);
#pragma unroll 1
  for (int tb = warp; tb < kChunk; tb += 4 * U) {
    float rq[U][NI], rk[U][NI], ra[U][NI];
#pragma unroll
    for (int m = 0; m < U; ++m) {
      const int t = tb + 4 * m;
      const int64_t qk = (c.row + t) * p.qkv_stride + h * p.dim, a = (c.row + t) * p.decay_stride + h * p.dim;
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        const int d = i * 32 + lane;
        const bool in = t < c.n && d < p.dim;
        rq[m][i] = in ? bf_at(p.q, qk + d) : 0.f;
        rk[m][i] = in ? bf_at(p.k, qk + d) : 0.f;
        ra[m][i] = in ? bf_at(p.decay, a + d) : 0.f;
      }
    }
#pragma unroll
    for (int m = 0; m < U; ++m) {
      const int t = tb + 4 * m;
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        const int d = i * 32 + lane, x = t * ROW + d;
        a_s[x] = t < c.n && d < p.dim ? fast_exp2(to_log2 * log_sigmoid_of<__nv_bfloat16>(ra[m][i] + bias[i])) : 1.f;
        q_s[x] = rq[m][i] * p.q_scale;
        k_s[x] = rk[m][i];
      }
    }
  }
  __syncthreads();
  // B below and on the diagonal: a warp takes every fourth column s and walks down the rows with w = k_s a_{s+1} .. a_t in registers,
  // two rows at a time
  {
    float w[4][NI];
#pragma unroll
    for (int j = 0; j < 4; ++j)
#pragma unroll
      for (int i = 0; i < NI; ++i) w[j][i] = 0.f;
#pragma unroll 1
    for (int t0 = 0; t0 < kChunk; t0 += 2) {
      float v[8];
#pragma unroll
      for (int r = 0; r < 2; ++r) {
        const int t = t0 + r, x = t * ROW + lane;
        float q[NI], a[NI];
#pragma unroll
        for (int i = 0; i < NI; ++i) { q[i] = q_s[x + i * 32]; a[i] = a_s[x + i * 32]; }
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int col = warp + 4 * j;          // (the same for the whole warp)
          if (col == t) {
#pragma unroll
            for (int i = 0; i < NI; ++i) w[j][i] = k_s[x + i * 32];
          } else if (col < t) {
#pragma unroll
            for (int i = 0; i < NI; ++i) w[j][i] *= a[i];
          }
          float b = 0.f;
#pragma unroll
          for (int i = 0; i < NI; ++i) b = fmaf(q[i], w[j][i], b);
          v[r * 4 + j] = b;
        }
      }
      // halving exchanges leave lane groups of four with one sum each
      const bool up16 = lane & 16, up8 = lane & 8, up4 = lane & 4;
#pragma unroll
      for (int m = 0; m < 4; ++m) {
        const float send = up16 ? v[m] : v[4 + m];
        v[m] = (up16 ? v[4 + m] : v[m]) + __shfl_xor_sync(0xffffffffu, send, 16);
      }
#pragma unroll
      for (int m = 0; m < 2; ++m) {
        const float send = up8 ? v[m] : v[2 + m];
        v[m] = (up8 ? v[2 + m] : v[m]) + __shfl_xor_sync(0xffffffffu, send, 8);
      }
      {
        const float send = up4 ? v[0] : v[1];
        v[0] = (up4 ? v[1] : v[0]) + __shfl_xor_sync(0xffffffffu, send, 4);
      }
      v[0] += __shfl_xor_sync(0xffffffffu, v[0], 2);
      v[0] += __shfl_xor_sync(0xffffffffu, v[0], 1);
      if ((lane & 3) == 0) bm[t0 + (up16 ? 1 : 0)][warp + (up8 ? 8 : 0) + (up4 ? 4 : 0)] = v[0];      // (above the diagonal: not read)
    }
  }
  __syncthreads();
  if (warp == 0) write_triangle([&](int t, int s) { return bm[t][s]; }, lane, rec + lay.b);
  for (int d = tid; d < D32; d += 128) {         // a thread owns a key channel: q times the decay so far, k times what is still to come
    float a[kChunk], run = 1.f;
#pragma unroll
    for (int t = 0; t < kChunk; ++t) {
      a[t] = a_s[t * ROW + d];
      run *= a[t];
      q_s[t * ROW + d] *= run;
    }
    if (d < 16 * KS) reinterpret_cast<float*>(rec + lay.extra)[d] = run;
    run = 1.f;
#pragma unroll
    for (int t = kChunk - 1; t >= 0; --t) {
      k_s[t * ROW + d] *= run;
      run *= a[t];
    }
  }
  __syncthreads();
  for (int i = tid; i < KS * 64; i += 128) {
    const int ln = i & 31, n = (i >> 5) & 1, ks = i >> 6;
    const float* src = q_s + (n * 8 + (ln >> 2)) * ROW + ks * 16 + (ln & 3) * 2;
    const float2 x = *reinterpret_cast<const float2*>(src), y = *reinterpret_cast<const float2*>(src + 8);
    uint4 o;
    split_pair(x.x, x.y, o.x, o.z);
    split_pair(y.x, y.y, o.y, o.w);
    reinterpret_cast<uint4*>(rec)[i] = o;
  }
  write_keys(k_s, ROW, KS, rec + lay.k);
  write_values(v_s, p.vtp * 16, rec + lay.v);
}

// ---- exponential gates -------------------------------------------------------------------------------------
template <int KS>
__global__ void __launch_bounds__(128) exp_chunk_prep(const LinearParams p) {
  constexpr int DP = 16 * KS, ROW = DP + 2;
  extern __shared__ __align__(16) float sm[];
  float* k_s = sm;                               // [16][ROW], scaled
  __nv_bfloat16* v_s = reinterpret_cast<__nv_bfloat16*>(k_s + kChunk * ROW);
  __shared__ float part[4][kChunk][kChunk + 1], bm[kChunk][kChunk + 1], e_s[kChunk], top_s[kChunk];
  const int h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const ChunkSite c = chunk_site(p, blockIdx.x);
  if (c.n <= 0) return;
  const LinearLayout lay = linear_layout(KS, p.vtp, true);
  uint8_t* rec = p.records + (static_cast<int64_t>(blockIdx.x) * p.heads + h) * lay.total;
  if (tid == 0 && c.row == p.cu[c.seq]) stash_maximum(p, c.seq, h);
  stage_values(p, c, h, p.vtp * 16, v_s);
  // gates, every warp for itself (lanes 0..15): F, the running maximum of i - F, and with them M, all in log2 units
  float f = 0.f, i = -INFINITY;
  if (lane < c.n) {
    f = log_forget<__nv_bfloat16>(p, c.row + lane, h) * kLog2e;
    i = log_input<__nv_bfloat16>(p, c.row + lane, h) * kLog2e;
  }
#pragma unroll
  for (int off = 1; off < kChunk; off <<= 1) {
    const float x = __shfl_up_sync(0xffffffffu, f, off);
    if (lane >= off) f += x;
  }
  const float e = i - f;                         // -inf behind the last token
  float top = e;
#pragma unroll
  for (int off = 1; off < kChunk; off <<= 1) {
    const float x = __shfl_up_sync(0xffffffffu, top, off);
    if (lane >= off) top = fmaxf(top, x);
  }
  if (warp == 0 && lane < kChunk) {
    e_s[lane] = e; top_s[lane] = top;
    reinterpret_cast<float*>(rec + lay.extra)[lane] = f;
    reinterpret_cast<float*>(rec + lay.extra)[kChunk + lane] = f + top;
  }
  const float key_w = fast_exp2(e - __shfl_sync(0xffffffffu, top, kChunk - 1));      // lane s: e^{F_16 - F_s + i_s - M_16}
  // q . k: a warp takes every fourth 16-channel step.  The second operand of (.) q^T is the first operand of q k^T with its
  // middle registers exchanged
  float acc[2][4];
#pragma unroll
  for (int n = 0; n < 2; ++n)
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[n][j] = 0.f;
  const bool pairs = p.dim % 2 == 0 && p.qkv_stride % 2 == 0 && ((reinterpret_cast<uintptr_t>(p.q) | reinterpret_cast<uintptr_t>(p.k)) & 3) == 0;
  auto two = [&](const void* base, int t, int d) -> uint32_t {
    if (t >= c.n || d >= p.dim) return 0u;
    const uint16_t* x = static_cast<const uint16_t*>(base) + (c.row + t) * p.qkv_stride + static_cast<int64_t>(h) * p.dim + d;
    if (pairs) return *reinterpret_cast<const uint32_t*>(x);
    return static_cast<uint32_t>(x[0]) | (d + 1 < p.dim ? static_cast<uint32_t>(x[1]) << 16 : 0u);
  };
  const float w0 = __shfl_sync(0xffffffffu, key_w, lane >> 2), w1 = __shfl_sync(0xffffffffu, key_w, (lane >> 2) + 8);
#pragma unroll
  for (int ks = warp; ks < KS; ks += 4) {
    const int t = lane >> 2, d = ks * 16 + (lane & 3) * 2;
    const uint2 q0 = make_uint2(two(p.q, t, d), two(p.q, t, d + 8)), q1 = make_uint2(two(p.q, t + 8, d), two(p.q, t + 8, d + 8));
    const uint2 k0 = make_uint2(two(p.k, t, d), two(p.k, t, d + 8)), k1 = make_uint2(two(p.k, t + 8, d), two(p.k, t + 8, d + 8));
    reinterpret_cast<uint2*>(rec)[(ks * 2) * 32 + lane] = q0;
    reinterpret_cast<uint2*>(rec)[(ks * 2 + 1) * 32 + lane] = q1;
    const uint32_t a[4] = {q0.x, q1.x, q0.y, q1.y};
    mma_bf16_16816(acc[0], a, k0.x, k0.y);
    mma_bf16_16816(acc[1], a, k1.x, k1.y);
    float* row0 = k_s + t * ROW + d;
    float* row1 = row0 + 8 * ROW;
    *reinterpret_cast<float2*>(row0) = make_float2(bf16_lo(k0.x) * w0, bf16_hi(k0.x) * w0);
    *reinterpret_cast<float2*>(row0 + 8) = make_float2(bf16_lo(k0.y) * w0, bf16_hi(k0.y) * w0);
    *reinterpret_cast<float2*>(row1) = make_float2(bf16_lo(k1.x) * w1, bf16_hi(k1.x) * w1);
    *reinterpret_cast<float2*>(row1 + 8) = make_float2(bf16_lo(k1.y) * w1, bf16_hi(k1.y) * w1);
  }
#pragma unroll
  for (int n = 0; n < 2; ++n)
#pragma unroll
    for (int j = 0; j < 4; ++j) part[warp][(lane >> 2) + (j >> 1) * 8][n * 8 + (lane & 3) * 2 + (j & 1)] = acc[n][j];
  __syncthreads();
#pragma unroll
  for (int x = tid; x < kChunk * kChunk; x += 128) {
    const int t = x / kChunk, s = x % kChunk;
    const float dot = (part[0][t][s] + part[1][t][s]) + (part[2][t][s] + part[3][t][s]);
    bm[t][s] = s <= t ? dot * p.q_scale * fast_exp2(e_s[s] - top_s[t]) : 0.f;
  }
  float* extra = reinterpret_cast<float*>(rec + lay.extra);
  for (int d = tid; d < DP; d += 128) {
    float sum = 0.f;
#pragma unroll
    for (int t = 0; t < kChunk; ++t) sum += k_s[t * ROW + d];
    extra[3 * kChunk + d] = sum;
  }
  __syncthreads();
  if (warp == 0) {
    write_triangle([&](int t, int s) { return bm[t][s]; }, lane, rec + lay.b);
  } else if (warp == 1 && lane < kChunk) {
    float sum = 0.f;
#pragma unroll
    for (int s = 0; s < kChunk; ++s) sum += bm[lane][s];
    extra[2 * kChunk + lane] = sum;
  }
  write_keys(k_s, ROW, KS, rec + lay.k);
  write_values(v_s, p.vtp * 16, rec + lay.v);
}

// ---- the recurrence over chunks ------------------------------------------------------------------------------
// SPLIT warps share a 16-column tile: each keeps the state of its part of the key channels, and the first adds their outputs up one
// chunk later than they are left in shared memory
template <bool EXP, int KS, int WARPS, int SPLIT>
struct LinearScanCfg {
  static constexpr int SHARED = KS * (EXP ? 512 : 1024) + KS * 1024 + 1024 + (EXP ? 192 : 0) + KS * 64;
  static constexpr int THREADS = (WARPS * SPLIT + (EXP ? 1 : 0)) * 32;
  static constexpr int STAGE = SHARED + WARPS * 512;           // common part + a tile of values per tile
  static constexpr int SUMS = 2 * WARPS * (SPLIT - 1) * 1024;
  // deep enough for the latency of a record: two CTAs per SM, or one where a CTA is a single tile (few heads and sequences)
  static constexpr int FIT = ((WARPS == 1 ? 200 : 100) * 1024 - SUMS) / STAGE;
  static constexpr int STAGES = FIT < 3 ? 3 : FIT > 10 ? 10 : FIT;
  static constexpr int SMEM = STAGES * STAGE + SUMS + STAGES * 8;
  static_assert(STAGE % 16 == 0 && KS % SPLIT == 0, "stages start at multiples of 16 bytes; parts are equal");
};

template <bool EXP, int KS, int WARPS, int SPLIT>
__global__ void __launch_bounds__(LinearScanCfg<EXP, KS, WARPS, SPLIT>::THREADS) linear_chunk_scan(const LinearParams p) {
  using C = LinearScanCfg<EXP, KS, WARPS, SPLIT>;
  constexpr int KP = KS / SPLIT;
  extern __shared__ __align__(128) uint8_t smem[];
  float* sums = reinterpret_cast<float*>(smem + C::STAGES * C::STAGE);
  uint64_t* full = reinterpret_cast<uint64_t*>(smem + C::STAGES * C::STAGE + C::SUMS);
  __shared__ int dead_s;                          // a copy did not arrive: nobody waits any more, nothing is kept
  const int s = blockIdx.z, h = blockIdx.y, tid = threadIdx.x, lane = tid & 31;
  const int tile = (tid >> 5) % WARPS, part = (tid >> 5) / WARPS;
  const int begin = p.cu[s], n_tok = p.cu[s + 1] - begin;
  if (n_tok <= 0) return;
  const int n_chunks = (n_tok + kChunk - 1) / kChunk, vt = blockIdx.x * WARPS + tile;
  const LinearLayout lay = linear_layout(KS, p.vtp, EXP);
  const uint8_t* rec = p.records + (static_cast<int64_t>(chunk_base(begin, s)) * p.heads + h) * lay.total;
  const int64_t rec_step = static_cast<int64_t>(p.heads) * lay.total;
  if (tid == 0) {
    for (int i = 0; i < C::STAGES; ++i) mbar_init(&full[i], 1);
    dead_s = 0;
    fence_mbar_init();
  }
  __syncthreads();
  auto fetch = [&](int c) {                       // one thread
    const int st = c % C::STAGES;
    const uint8_t* src = rec + c * rec_step;
    const uint32_t dst = smem_u32(smem + st * C::STAGE), bar = smem_u32(&full[st]);
    mbar_arrive_expect_tx(&full[st], C::STAGE);
    bulk_copy(dst, src, C::SHARED, bar);
    bulk_copy(dst + C::SHARED, src + lay.v + blockIdx.x * (WARPS * 512), WARPS * 512, bar);
  };
  if (tid == 0)
    for (int c = 0; c < min(C::STAGES, n_chunks); ++c) fetch(c);

  const int64_t slot = linear_slot(p, s), hbase = (slot * p.heads + h) * static_cast<int64_t>(p.dim);
  const bool fresh = slot < 0 || p.positions[begin] == 0;
  const int v0 = vt * 16 + (lane >> 2), dq = (lane & 3) * 2, d0 = part * KP * 16 + dq;
  const bool normaliser = EXP && part == SPLIT;   // the warp behind the tiles
  float S[2 * KP][4];                             // S^T: rows v0, v0 + 8; columns 8 j + d0, + 1
  auto state_at = [&](int j, int i) { return p.S + (hbase + 8 * j + d0 + (i & 1)) * p.vp + v0 + (i & 2) * 4; };
  auto in_state = [&](int j, int i) { return 8 * j + d0 + (i & 1) < p.dim && v0 + (i & 2) * 4 < p.vdim; };
  float m = EXP ? p.m0[s * p.heads + h] * kLog2e : 0.f;
  volatile int* dead = &dead_s;
  auto arrived = [&](int c) {
    if (!*dead && !mbar_wait(&full[c % C::STAGES], (c / C::STAGES) & 1)) {
      *dead = 1;
      report(p.dev_status, kDevWaitTimeout, c);
    }
    __syncwarp();
  };
  if (normaliser) {
    // n at the channels of this lane's query fragments: 16 ks + dq, + 1, + 8, + 9.  The CTA of the first columns has it; the others'
    // warp keeps step with the barriers
    const bool works = blockIdx.x == 0;
    auto channel = [&](int ks, int i) { return ks * 16 + dq + (i & 1) + (i & 2) * 4; };
    float n[KS][4];
#pragma unroll
    for (int ks = 0; ks < KS; ++ks)
#pragma unroll
      for (int i = 0; i < 4; ++i) n[ks][i] = works && !fresh && channel(ks, i) < p.dim ? p.n[hbase + channel(ks, i)] : 0.f;
    for (int c = 0; c < n_chunks; ++c) {
      if (works) {
        arrived(c);
        const uint8_t* base = smem + c % C::STAGES * C::STAGE;
        const float* extra = reinterpret_cast<const float*>(base + lay.extra);
        const uint2* q_r = reinterpret_cast<const uint2*>(base);
        const float from0 = extra[kChunk - 1] + m, local = extra[2 * kChunk - 1], m_end = fmaxf(from0, local);
        const float alpha = fast_exp2(from0 - m_end), beta = fast_exp2(local - m_end);
        float dot[2] = {0.f, 0.f};                // tokens lane / 4 and lane / 4 + 8
#pragma unroll
        for (int ks = 0; ks < KS; ++ks) {
#pragma unroll
          for (int r = 0; r < 2; ++r) {
            const uint2 q = q_r[(ks * 2 + r) * 32 + lane];
            dot[r] = fmaf(bf16_lo(q.x), n[ks][0], dot[r]); dot[r] = fmaf(bf16_hi(q.x), n[ks][1], dot[r]);
            dot[r] = fmaf(bf16_lo(q.y), n[ks][2], dot[r]); dot[r] = fmaf(bf16_hi(q.y), n[ks][3], dot[r]);
          }
          const float* sum = extra + 3 * kChunk + ks * 16 + dq;
          const float2 lo = *reinterpret_cast<const float2*>(sum), hi = *reinterpret_cast<const float2*>(sum + 8);
          n[ks][0] = fmaf(beta, lo.x, alpha * n[ks][0]); n[ks][1] = fmaf(beta, lo.y, alpha * n[ks][1]);
          n[ks][2] = fmaf(beta, hi.x, alpha * n[ks][2]); n[ks][3] = fmaf(beta, hi.y, alpha * n[ks][3]);
        }
#pragma unroll
        for (int r = 0; r < 2; ++r) {
          dot[r] += __shfl_xor_sync(0xffffffffu, dot[r], 1);
          dot[r] += __shfl_xor_sync(0xffffffffu, dot[r], 2);
          const int t = r * 8 + (lane >> 2);
          if ((lane & 3) == 0 && c * kChunk + t < n_tok) {
            const int64_t th = static_cast<int64_t>(begin + c * kChunk + t) * p.heads + h;
            const float f0 = extra[t] + m, loc = extra[kChunk + t], mt = fmaxf(f0, loc);
            p.mt[th] = mt * kLn2;
            p.nq[th] = fmaf(p.q_scale * fast_exp2(f0 - mt), dot[r], fast_exp2(loc - mt) * extra[2 * kChunk + t]);
          }
        }
        m = m_end;
      }
      __syncthreads();
    }
    if (works && slot >= 0 && !*dead) {
      if (lane == 0) p.m[slot * p.heads + h] = m * kLn2;
#pragma unroll
      for (int ks = 0; ks < KS; ++ks)
#pragma unroll
        for (int i = 0; i < 4; ++i)
          if (lane < 4 && channel(ks, i) < p.dim) p.n[hbase + channel(ks, i)] = n[ks][i];
    }
    return;
  }
#pragma unroll
  for (int j = 0; j < 2 * KP; ++j)
#pragma unroll
    for (int i = 0; i < 4; ++i) S[j][i] = !fresh && in_state(j, i) ? *state_at(j, i) : 0.f;

  for (int c = 0; c < n_chunks; ++c) {
    arrived(c);
    const uint8_t* base = smem + c % C::STAGES * C::STAGE;
    const uint4* k_r = reinterpret_cast<const uint4*>(base + lay.k) + part * KP * 64;
    const float* extra = reinterpret_cast<const float*>(base + lay.extra);
    const uint4 vw = reinterpret_cast<const uint4*>(base + C::SHARED)[tile * 32 + lane];
    const uint32_t v[4] = {vw.x, vw.y, vw.z, vw.w};
    float row_f[2][2], row_b[2][2], alpha = 1.f, beta = 1.f, m_end = 0.f;
    if constexpr (EXP) {
      if (SPLIT == 1 || part == 0) {
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
          for (int i = 0; i < 2; ++i) {
            const int t = n * 8 + dq + i;
            const float from0 = extra[t] + m, local = extra[kChunk + t], mt = fmaxf(from0, local);
            row_f[n][i] = p.q_scale * fast_exp2(from0 - mt);
            row_b[n][i] = fast_exp2(local - mt);
          }
      }
      const float from0 = extra[kChunk - 1] + m, local = extra[2 * kChunk - 1];
      m_end = fmaxf(from0, local);
      alpha = fast_exp2(from0 - m_end); beta = fast_exp2(local - m_end);
    }
    float oa[2][4], ob[2][4], oc[2][4];
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int i = 0; i < 4; ++i) oa[n][i] = ob[n][i] = oc[n][i] = 0.f;
    if (SPLIT == 1 || part == 0) {                // V^T B^T
      const uint4* b_r = reinterpret_cast<const uint4*>(base + lay.b);
#pragma unroll
      for (int n = 0; n < 2; ++n) {
        const uint4 b = b_r[n * 32 + lane];
        mma_bf16_16816(oc[n], v, b.x, b.y);
        mma_bf16_16816(oc[n], v, b.z, b.w);
      }
    }
#pragma unroll
    for (int ks = 0; ks < KP; ++ks) {             // S0^T Q^T
      Split a;
      split_tile(S[2 * ks], S[2 * ks + 1], a);
      const int at = (part * KP + ks) * 64 + lane;
      if constexpr (EXP) {
        const uint2* q_r = reinterpret_cast<const uint2*>(base);
        const uint2 q0 = q_r[at], q1 = q_r[at + 32];
        mma_bf16_16816(oa[0], a.hi, q0.x, q0.y); mma_bf16_16816(oa[1], a.hi, q1.x, q1.y);
        mma_bf16_16816(ob[0], a.lo, q0.x, q0.y); mma_bf16_16816(ob[1], a.lo, q1.x, q1.y);
      } else {
        const uint4* q_r = reinterpret_cast<const uint4*>(base);
        const uint4 q0 = q_r[at], q1 = q_r[at + 32];
        mma_bf16_16816(oa[0], a.hi, q0.x, q0.y); mma_bf16_16816(oa[1], a.hi, q1.x, q1.y);
        mma_bf16_16816(ob[0], a.hi, q0.z, q0.w); mma_bf16_16816(ob[1], a.hi, q1.z, q1.w);
        mma_bf16_16816(ob[0], a.lo, q0.x, q0.y); mma_bf16_16816(ob[1], a.lo, q1.x, q1.y);
      }
    }
#pragma unroll
    for (int j = 0; j < 2 * KP; ++j) {            // S^T <- S^T decay + V^T K
      const uint4 k = k_r[j * 32 + lane];
      if constexpr (EXP) {
        float d[4] = {0.f, 0.f, 0.f, 0.f};
        mma_bf16_16816(d, v, k.x, k.y);
        mma_bf16_16816(d, v, k.z, k.w);
#pragma unroll
        for (int i = 0; i < 4; ++i) S[j][i] = fmaf(beta, d[i], alpha * S[j][i]);
      } else {
        const float2 g = *reinterpret_cast<const float2*>(extra + 8 * j + d0);
        S[j][0] *= g.x; S[j][1] *= g.y; S[j][2] *= g.x; S[j][3] *= g.y;
        mma_bf16_16816(S[j], v, k.x, k.y);
        mma_bf16_16816(S[j], v, k.z, k.w);
      }
    }
    m = m_end;
    float4* mine = reinterpret_cast<float4*>(sums) + (((c & 1) * WARPS + tile) * (SPLIT - 1)) * 64 + lane;
    if (SPLIT > 1 && part > 0) {
#pragma unroll
      for (int n = 0; n < 2; ++n)
        mine[((part - 1) * 2 + n) * 32] = make_float4(oa[n][0] + ob[n][0], oa[n][1] + ob[n][1], oa[n][2] + ob[n][2], oa[n][3] + ob[n][3]);
    }
    __syncthreads();                              // the stage has been read, the sums are there
    if (tid == 0 && c + C::STAGES < n_chunks) { fence_proxy_async(); fetch(c + C::STAGES); }
    if (SPLIT > 1 && part > 0) continue;
#pragma unroll
    for (int n = 0; n < 2; ++n) {
      float sum[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) sum[i] = oa[n][i] + ob[n][i];
#pragma unroll
      for (int k = 0; k < SPLIT - 1; ++k) {
        const float4 x = mine[(k * 2 + n) * 32];
        sum[0] += x.x; sum[1] += x.y; sum[2] += x.z; sum[3] += x.w;
      }
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int t = c * kChunk + n * 8 + dq + (i & 1), col = v0 + (i & 2) * 4;
        if (t >= n_tok) continue;
        const int64_t th = static_cast<int64_t>(begin + t) * p.heads + h;
        const float o = EXP ? fmaf(row_f[n][i & 1], sum[i], row_b[n][i & 1] * oc[n][i]) : sum[i] + oc[n][i];
        if (col < p.vdim) p.o[th * p.vdim + col] = o;
      }
    }
  }
  if (*dead) {                                    // let the copies in flight land, within bounds; keep the old state
    for (int k = max(0, n_chunks - C::STAGES); k < n_chunks; ++k) mbar_wait(&full[k % C::STAGES], (k / C::STAGES) & 1, 1u << 16);
    return;
  }
  if (slot < 0) return;
#pragma unroll
  for (int j = 0; j < 2 * KP; ++j)
#pragma unroll
    for (int i = 0; i < 4; ++i)
      if (in_state(j, i)) *state_at(j, i) = S[j][i];
}

template <bool EXP, int KS>
static int launch_linear_chunks(const LinearParams& p, cudaStream_t st) {
  constexpr int D32 = (16 * KS + 31) / 32 * 32;
  const size_t smem = (EXP ? kChunk * (16 * KS + 2) : 3 * kChunk * (D32 + 4)) * sizeof(float) + static_cast<size_t>(p.vtp) * 16 * kChunk * 2;
  if (smem > 200 * 1024) return kUnsupportedShape;
  const int slots = p.tokens / kChunk + p.num_seqs;
  struct PrepTag {};
  auto prep = EXP ? &exp_chunk_prep<KS> : &decay_chunk_prep<KS>;
  const int rc = opt_in_dynamic_smem<PrepTag>(reinterpret_cast<const void*>(prep), smem);
  if (rc != kOk) return rc;
  prep<<<dim3(slots, p.heads), 128, smem, st>>>(p);
  if (cudaGetLastError() != cudaSuccess) return kLaunchFailed;
  auto scan = [&](auto tiles, auto parts) -> int {
    constexpr int WARPS = decltype(tiles)::value, SPLIT = decltype(parts)::value;
    using C = LinearScanCfg<EXP, KS, WARPS, SPLIT>;
    struct ScanTag {};
    auto kernel = &linear_chunk_scan<EXP, KS, WARPS, SPLIT>;
    const int r = opt_in_dynamic_smem<ScanTag>(reinterpret_cast<const void*>(kernel), C::SMEM);
    if (r != kOk) return r;
    kernel<<<dim3(p.vtp / WARPS, p.heads, p.num_seqs), C::THREADS, C::SMEM, st>>>(p);
    return cudaGetLastError() == cudaSuccess ? kOk : kLaunchFailed;
  };
  using One = std::integral_constant<int, 1>; using Two = std::integral_constant<int, 2>;
  using Three = std::integral_constant<int, 3>; using Four = std::integral_constant<int, 4>;
  using Parts = std::conditional_t<KS % 2 == 0 && KS >= 4, Two, One>;
  switch (linear_warps(p)) {
    case 1: return scan(One{}, std::conditional_t<KS % 4 == 0, Four, Parts>{});
    case 2: return scan(Two{}, Parts{});
    case 3: return scan(Three{}, Parts{});
    default: return scan(Four{}, Parts{});
  }
}

}  // namespace mvb
