// State-space layer with one decay per head (the "state-space duality" form of Mamba-2) on a packed ragged batch, state carried per
// sequence.  Per head, with S [N, vdim] in fp32, keys B_t and queries C_t [N] shared by a group of heads, values x_t [vdim]:
//
//   dt_t = softplus(raw_t + bias)      S <- e^{a dt_t} S + dt_t B_t x_t^T      y_t = S^T C_t + D x_t
//
// Everything behind the projections and the short convolution (whose outputs x, B and C come in the activation type) is fp32: dt, the
// decays and their logarithms, the state.  State slots: [slots, heads, N, vp] fp32, vp = vdim rounded up to 4.
//
// Ragged step, bf16 (ssd_chunk_kernel): chunks of 64 tokens.  With F_t = sum_{s <= t} a dt_s inside a chunk and its initial S0:
//   y_t = e^{F_t} S0^T C_t + sum_{s <= t} M_ts x_s          M_ts = (C_t . B_s) e^{F_t - F_s} dt_s,  + D where t = s
//   S  <- e^{F_64} S0 + sum_s B_s (e^{F_64 - F_s} dt_s x_s)^T
// All exponents are <= 0, so no factor exceeds 1 whatever the steps are.  A CTA walks the chunks of one sequence for one head and 16
// value columns per warp; S^T stays in the accumulator registers of its warp, whose fragments are operand fragments of the next
// chunk's product as they stand.  C B^T is computed once per CTA, its rows shared out over the warps, and passes through shared
// memory; B, C and x of the next chunk arrive by cp.async meanwhile.  x, B and C are bf16 and enter exactly; M, S and the scaled
// values enter as bf16 high + low part (16 significant bits per factor, fp32 accumulation); the state itself is never rounded below
// fp32.
// Few (sequence, head) pairs with long prompts would leave most SMs idle, so there the sequences are cut into segments that are walked
// at the same time: a first pass of the same kernel leaves what each segment alone adds to the state (STATES), ssd_join_kernel turns that
// into the state in front of every segment, and the second pass starts from there.
// Ragged step, fp32 (ssd_tokens_kernel): token by token in plain fp32.
// One token per sequence (ssd_step_kernel): a CTA per sequence and up to 64 columns of a head, the state read once and
// written once.
//
// gated_group_norm_kernel finishes the mixer: y silu(z), over the root mean square of each of `groups` equal parts of the row, times w.
//
// Roofline: HBM for all of them (decode: 8 N vdim bytes per head and sequence); the chunk kernel is held by mma.sync issue.
#include "chunk_common.cuh"
#include "host_util.cuh"
#include "mini_vllm_b200.h"

namespace mvb {

struct SsdParams {
  const void *x, *b, *c; int64_t stride;       // row t: x [heads, vdim], b and c [groups, N]; one row stride
  const void* dt; int64_t dt_stride;           // raw step [heads]
  const float *dt_bias, *a_log2e, *d;          // [heads]; a log2(e) <= 0
  void* y; int64_t y_stride;                   // row t, [heads, vdim]
  float* state; const int32_t* slots; int64_t num_slots;
  const int32_t* cu; const int64_t* positions;
  int num_seqs, tokens, heads, per_group, n, vdim, vp;
  bool vec;                                    // rows of x, b and c may be read, and those of y written, as 16-byte vectors
  int seg;                                     // tokens of a segment (0: sequences are walked whole)
  float *seg_state, *seg_keep;                 // [segment slots, heads, N, vp], [segment slots, heads]
  int* dev_status;
};
// sequence s owns segment slots seg_base(first row, s) ..: never overlapping, no prefix sum needed
__device__ __forceinline__ int seg_base(const SsdParams& p, int s) { return p.cu[s] / p.seg + s; }

__device__ __forceinline__ int64_t ssd_slot(const SsdParams& p, int s) {
  if (p.state == nullptr) return -1;
  const int64_t slot = p.slots[s];
  if (slot >= p.num_slots) { report(p.dev_status, kDevBadSlot, s); return -1; }
  return slot;
}
template <class T> __device__ __forceinline__ float ssd_dt(const SsdParams& p, int64_t t, int h) {
  return softplus_of<T>(to_f(static_cast<const T*>(p.dt)[t * p.dt_stride + h]) + p.dt_bias[h]);
}
// S 2^x + in; in fp32 the decrement is computed instead of the factor, which may be close to 1 over thousands of tokens
template <class T> __device__ __forceinline__ float ssd_decay(float x) {
  if constexpr (sizeof(T) == 4) return expm1f(x * 0.6931471805599453f);
  else return fast_exp2(x);
}
template <class T> __device__ __forceinline__ float ssd_advance(float S, float decay, float in) {
  if constexpr (sizeof(T) == 4) return fmaf(S, decay, S) + in;
  else return fmaf(S, decay, in);
}

// ---- one token per sequence ------------------------------------------------------------------------------
// A CTA has tile_cols columns of a head, a thread kStepRows rows x 4 columns.
constexpr int kStepRows = 8;

template <class T>
__global__ void __launch_bounds__(512, 2) ssd_step_kernel(const SsdParams p, int tile_cols, int tiles) {
  extern __shared__ __align__(16) float sm[];
  const int s = blockIdx.y, h = blockIdx.x / tiles, col0 = blockIdx.x % tiles * tile_cols, tid = threadIdx.x, nt = blockDim.x;
  const int quads = tile_cols / 4, row_groups = (p.n + kStepRows - 1) / kStepRows;
  float* red = sm;                              // [row groups][tile_cols]
  float* b_s = red + row_groups * tile_cols;    // [n], times dt
  float* c_s = b_s + p.n;
  const int64_t slot = ssd_slot(p, s);
  const bool fresh = slot < 0 || p.positions[s] == 0;
  const int rg = tid / quads, cq = tid % quads, c = col0 + cq * 4;
  const int rows = rg < row_groups && c < p.vp ? (p.n - rg + row_groups - 1) / row_groups : 0;      // rows rg, rg + row_groups, ...
  const int64_t down = static_cast<int64_t>(row_groups) * p.vp;
  float* at = p.state + ((slot * p.heads + h) * static_cast<int64_t>(p.n) + rg) * p.vp + c;
  float4 S[kStepRows];
#pragma unroll
  for (int r = 0; r < kStepRows; ++r) {         // the state first: it is what the kernel waits for
    S[r] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (!fresh && r < rows) S[r] = __ldcs(reinterpret_cast<const float4*>(at + r * down));
  }
  const float dt = ssd_dt<T>(p, s, h), decay = ssd_decay<T>(p.a_log2e[h] * dt);
  const int64_t group = s * p.stride + static_cast<int64_t>(h / p.per_group) * p.n;
  for (int i = tid; i < p.n; i += nt) {
    b_s[i] = to_f(static_cast<const T*>(p.b)[group + i]) * dt;
    c_s[i] = to_f(static_cast<const T*>(p.c)[group + i]);
  }
  const T* xrow = static_cast<const T*>(p.x) + s * p.stride + static_cast<int64_t>(h) * p.vdim;
  float x[4];
#pragma unroll
  for (int j = 0; j < 4; ++j) x[j] = rows > 0 && c + j < p.vdim ? to_f(xrow[c + j]) : 0.f;
  __syncthreads();
  float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int r = 0; r < kStepRows; ++r) {
    if (r >= rows) break;
    const float k = b_s[rg + r * row_groups], q = c_s[rg + r * row_groups];
    S[r].x = ssd_advance<T>(S[r].x, decay, k * x[0]); S[r].y = ssd_advance<T>(S[r].y, decay, k * x[1]);
    S[r].z = ssd_advance<T>(S[r].z, decay, k * x[2]); S[r].w = ssd_advance<T>(S[r].w, decay, k * x[3]);
    acc.x = fmaf(S[r].x, q, acc.x); acc.y = fmaf(S[r].y, q, acc.y); acc.z = fmaf(S[r].z, q, acc.z); acc.w = fmaf(S[r].w, q, acc.w);
    if (slot >= 0) __stcs(reinterpret_cast<float4*>(at + r * down), S[r]);
  }
  if (rg < row_groups) *reinterpret_cast<float4*>(red + rg * tile_cols + cq * 4) = acc;
  __syncthreads();
  if (tid < tile_cols && col0 + tid < p.vdim) {
    float y = 0.f;
    for (int w = 0; w < row_groups; ++w) y += red[w * tile_cols + tid];
    y = fmaf(p.d[h], to_f(xrow[col0 + tid]), y);
    static_cast<T*>(p.y)[s * p.y_stride + static_cast<int64_t>(h) * p.vdim + col0 + tid] = from_f<T>(y);
  }
}

// ---- ragged step, fp32 ---------------------------------------------------------------------------------------
// NI: 32-row groups of S per column (n <= 32 NI); a CTA owns 16 columns of one (sequence, head), a warp four, a lane eight row groups
template <int NI>
__global__ void __launch_bounds__(128) ssd_tokens_kernel(const SsdParams p) {
  constexpr int DP = 32 * NI, TT = 16;
  __shared__ __align__(16) float b_s[TT][DP], c_s[TT][DP];
  __shared__ float x_s[TT][16], y_s[TT][16], dt_s[TT], decay_s[TT];
  const int s = blockIdx.z, h = blockIdx.y, col0 = blockIdx.x * 16;
  const int tid = threadIdx.x, lane = tid & 31, rg = lane >> 2, cl = (tid >> 5) * 4 + (lane & 3), col = col0 + cl;
  const int begin = p.cu[s], n_tok = p.cu[s + 1] - begin;
  if (n_tok <= 0) return;
  const int64_t slot = ssd_slot(p, s);
  const bool fresh = slot < 0 || p.positions[begin] == 0, holds = col < p.vdim;
  float* home = p.state + (slot * p.heads + h) * static_cast<int64_t>(p.n) * p.vp + col;
  float S[NI][4];
#pragma unroll
  for (int i = 0; i < NI; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int row = i * 32 + rg * 4 + j;
      S[i][j] = !fresh && holds && row < p.n ? home[static_cast<int64_t>(row) * p.vp] : 0.f;
    }
  const float *xp = static_cast<const float*>(p.x) + static_cast<int64_t>(h) * p.vdim, *bp = static_cast<const float*>(p.b),
              *cp = static_cast<const float*>(p.c);
  const int64_t group = static_cast<int64_t>(h / p.per_group) * p.n;
  for (int t0 = 0; t0 < n_tok; t0 += TT) {
    const int nt = min(TT, n_tok - t0);
    for (int e = tid; e < nt * DP; e += 128) {
      const int tl = e / DP, i = e % DP;
      const int64_t at = static_cast<int64_t>(begin + t0 + tl) * p.stride + group + i;
      b_s[tl][i] = i < p.n ? bp[at] : 0.f;
      c_s[tl][i] = i < p.n ? cp[at] : 0.f;
    }
    for (int e = tid; e < nt * 16; e += 128) {
      const int tl = e >> 4, c = col0 + (e & 15);
      x_s[tl][e & 15] = c < p.vdim ? xp[static_cast<int64_t>(begin + t0 + tl) * p.stride + c] : 0.f;
    }
    if (tid < nt) {
      dt_s[tid] = ssd_dt<float>(p, begin + t0 + tid, h);
      decay_s[tid] = ssd_decay<float>(p.a_log2e[h] * dt_s[tid]);
    }
    __syncthreads();
    for (int tl = 0; tl < nt; ++tl) {
      const float g = decay_s[tl], in = dt_s[tl] * x_s[tl][cl];
      float acc[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        const float4 b = *reinterpret_cast<const float4*>(&b_s[tl][i * 32 + rg * 4]), c = *reinterpret_cast<const float4*>(&c_s[tl][i * 32 + rg * 4]);
        S[i][0] = ssd_advance<float>(S[i][0], g, b.x * in); acc[0] = fmaf(S[i][0], c.x, acc[0]);
        S[i][1] = ssd_advance<float>(S[i][1], g, b.y * in); acc[1] = fmaf(S[i][1], c.y, acc[1]);
        S[i][2] = ssd_advance<float>(S[i][2], g, b.z * in); acc[2] = fmaf(S[i][2], c.z, acc[2]);
        S[i][3] = ssd_advance<float>(S[i][3], g, b.w * in); acc[3] = fmaf(S[i][3], c.w, acc[3]);
      }
      float y = (acc[0] + acc[1]) + (acc[2] + acc[3]);
#pragma unroll
      for (int off = 4; off < 32; off <<= 1) y += __shfl_xor_sync(0xffffffffu, y, off);
      if (rg == 0) y_s[tl][cl] = y;
    }
    __syncthreads();
    for (int e = tid; e < nt * 16; e += 128) {
      const int tl = e >> 4, c = col0 + (e & 15);
      if (c < p.vdim)
        static_cast<float*>(p.y)[static_cast<int64_t>(begin + t0 + tl) * p.y_stride + static_cast<int64_t>(h) * p.vdim + c] =
            fmaf(p.d[h], x_s[tl][e & 15], y_s[tl][e & 15]);
    }
    __syncthreads();                            // the operands are about to be overwritten
  }
  if (slot < 0 || !holds) return;
#pragma unroll
  for (int i = 0; i < NI; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int row = i * 32 + rg * 4 + j;
      if (row < p.n) home[static_cast<int64_t>(row) * p.vp] = S[i][j];
    }
}

// ---- ragged step, bf16: chunks of 64 tokens --------------------------------------------------------------------
constexpr int kSsdChunk = 64;

__device__ __forceinline__ void stmatrix_x4_trans(uint32_t addr, const uint32_t (&r)[4]) {
  asm volatile("stmatrix.sync.aligned.m8n8.x4.trans.shared.b16 [%0], {%1, %2, %3, %4};"
               ::"r"(addr), "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]) : "memory");
}

template <int KS, int WARPS, bool STATES>       // 16 KS state channels, 16 WARPS value columns
struct SsdCfg {
  static constexpr int NROW = 16 * KS + 8, XROW = 16 * WARPS + 8, MROW = kSsdChunk + 8;      // (odd numbers of 16-byte units: no bank conflicts)
  static constexpr int B = 0, X = kSsdChunk * NROW, C = X + kSsdChunk * XROW, STAGE = STATES ? C : C + kSsdChunk * NROW;      // in bf16 numbers
  static constexpr int SMEM = (2 * STAGE + (STATES ? 0 : 2 * kSsdChunk * MROW)) * 2;
  static constexpr int THREADS = WARPS * 32;
};

// STATES: only what the segment adds to the state (and what it leaves of the one before) is wanted
template <int KS, int WARPS, bool STATES>
__global__ void __launch_bounds__(SsdCfg<KS, WARPS, STATES>::THREADS) ssd_chunk_kernel(const SsdParams p) {
  using G = SsdCfg<KS, WARPS, STATES>;
  constexpr int Q = kSsdChunk;
  extern __shared__ __align__(128) uint8_t smem[];
  __nv_bfloat16* stages = reinterpret_cast<__nv_bfloat16*>(smem);
  __nv_bfloat16* m_hi = stages + 2 * G::STAGE;
  __nv_bfloat16* m_lo = m_hi + Q * G::MROW;
  __shared__ float f_s[2][Q], dt_s[2][Q];         // F_t (log2), dt_t; per chunk parity
  const int h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  int s = blockIdx.z, begin = 0, end = 0;
  if (p.seg == 0) {
    begin = p.cu[s]; end = p.cu[s + 1];
  } else {                                        // the sequence and the rows of a segment slot
    int lo = 0, hi = p.num_seqs;
    while (hi - lo > 1) {
      const int mid = (lo + hi) >> 1;
      if (seg_base(p, mid) <= s) lo = mid; else hi = mid;
    }
    begin = p.cu[lo] + (s - seg_base(p, lo)) * p.seg;
    end = min(begin + p.seg, p.cu[lo + 1]);
    s = lo;
  }
  const int n_tok = end - begin;
  const bool last = end == p.cu[s + 1];
  if (n_tok <= 0 || (STATES && last)) return;
  const int n_chunks = (n_tok + Q - 1) / Q, p0 = (blockIdx.x * WARPS + warp) * 16;           // the warp's first value column
  const int64_t slot = ssd_slot(p, s), states = static_cast<int64_t>(p.n) * p.vp;
  const float* from = nullptr;                    // the state in front, and where the one behind goes (nullptr: nowhere)
  float* to = last && slot >= 0 ? p.state + (slot * p.heads + h) * states : nullptr;
  if (p.seg != 0) {
    float* here = p.seg_state + (static_cast<int64_t>(blockIdx.z) * p.heads + h) * states;
    if (STATES) to = here; else from = here;
  } else if (slot >= 0 && p.positions[begin] != 0) {
    from = to;
  }
  const float a = p.a_log2e[h], skip = p.d[h];
  const int64_t group = static_cast<int64_t>(h / p.per_group) * p.n, col0 = static_cast<int64_t>(h) * p.vdim + blockIdx.x * (WARPS * 16);
  const int cols = min(WARPS * 16, p.vdim - blockIdx.x * (WARPS * 16));                      // value columns there are
  const __nv_bfloat16 *xg = static_cast<const __nv_bfloat16*>(p.x) + col0, *bg = static_cast<const __nv_bfloat16*>(p.b) + group,
                      *cg = static_cast<const __nv_bfloat16*>(p.c) + group;

  // rows behind the last token and columns behind the last channel are zeros
  auto fetch_rows = [&](__nv_bfloat16* dst, int row, const __nv_bfloat16* src, int width, int padded, int chunk) {
    const int nt = min(Q, n_tok - chunk * Q), units = padded / 8;
    src += static_cast<int64_t>(begin + chunk * Q) * p.stride;
    if (p.vec) {
      for (int e = tid; e < Q * units; e += G::THREADS) {
        const int t = e / units, i = e % units * 8;
        __nv_bfloat16* to = dst + t * row + i;
        if (t < nt && i < width) cp_async16(smem_u32(to), src + t * p.stride + i);
        else *reinterpret_cast<uint4*>(to) = make_uint4(0u, 0u, 0u, 0u);
      }
    } else {
      for (int e = tid; e < Q * padded; e += G::THREADS) {
        const int t = e / padded, i = e % padded;
        dst[t * row + i] = t < nt && i < width ? src[t * p.stride + i] : __float2bfloat16_rn(0.f);
      }
    }
  };
  auto fetch = [&](int chunk) {
    __nv_bfloat16* st = stages + (chunk & 1) * G::STAGE;
    fetch_rows(st + G::B, G::NROW, bg, p.n, 16 * KS, chunk);
    if constexpr (!STATES) fetch_rows(st + G::C, G::NROW, cg, p.n, 16 * KS, chunk);
    fetch_rows(st + G::X, G::XROW, xg, cols, 16 * WARPS, chunk);
    cp_async_commit();
  };
  // warp 0: steps and running sums of a chunk; a token past the end has step 0 and changes nothing
  auto raw_step = [&](int chunk, int t) {
    t += chunk * Q;
    return t < n_tok ? to_f(static_cast<const __nv_bfloat16*>(p.dt)[static_cast<int64_t>(begin + t) * p.dt_stride + h]) : 0.f;
  };
  float raw0 = 0.f, raw1 = 0.f;
  const float dt_bias = p.dt_bias[h];
  auto steps = [&](int chunk) {
    const int left = n_tok - chunk * Q;
    const float d0 = 2 * lane < left ? softplus_fast(raw0 + dt_bias) : 0.f, d1 = 2 * lane + 1 < left ? softplus_fast(raw1 + dt_bias) : 0.f;
    float sum = a * d0 + a * d1;
#pragma unroll
    for (int off = 1; off < 32; off <<= 1) {
      const float up = __shfl_up_sync(0xffffffffu, sum, off);
      if (lane >= off) sum += up;
    }
    dt_s[chunk & 1][2 * lane] = d0; dt_s[chunk & 1][2 * lane + 1] = d1;
    f_s[chunk & 1][2 * lane] = sum - a * d1; f_s[chunk & 1][2 * lane + 1] = sum;
  };

  fetch(0);
  if (warp == 0) { raw0 = raw_step(0, 2 * lane); raw1 = raw_step(0, 2 * lane + 1); steps(0); }
  // S^T: rows p0 + lane / 4 (+ 8), columns 8 j + 2 (lane mod 4) (+ 1)
  const int dq = (lane & 3) * 2, r0 = lane >> 2;
  auto in_state = [&](int j, int i) { return 8 * j + dq + (i & 1) < p.n && p0 + r0 + (i & 2) * 4 < p.vdim; };
  auto state_at = [&](int j, int i) { return static_cast<int64_t>(8 * j + dq + (i & 1)) * p.vp + p0 + r0 + (i & 2) * 4; };
  float S[2 * KS][4];
#pragma unroll
  for (int j = 0; j < 2 * KS; ++j)
#pragma unroll
    for (int i = 0; i < 4; ++i) S[j][i] = from != nullptr && in_state(j, i) ? from[state_at(j, i)] : 0.f;

  float kept = 0.f;                               // STATES: sum of the chunks' log decays
  for (int chunk = 0; chunk < n_chunks; ++chunk) {
    const int nt = min(Q, n_tok - chunk * Q), nb = (nt + 15) / 16;                           // tokens, blocks of 16 of them
    const __nv_bfloat16* st = stages + (chunk & 1) * G::STAGE;
    const float *F = f_s[chunk & 1], *D = dt_s[chunk & 1];
    cp_async_wait<0>();
    __syncthreads();                              // this chunk's rows are there; everyone is done with the last one's
    if (chunk + 1 < n_chunks) {
      fetch(chunk + 1);
      if (warp == 0) { raw0 = raw_step(chunk + 1, 2 * lane); raw1 = raw_step(chunk + 1, 2 * lane + 1); }
    }
    if constexpr (!STATES) {
      // M: a warp takes rows of 16 x 16 blocks on and below the diagonal (two warps: the first and the last row, and the two between)
#pragma unroll 1
      for (int turn = 0; turn < 4 / WARPS; ++turn) {
        const int tb = WARPS == 4 ? warp : WARPS == 2 ? (turn == 0 ? 3 - warp : warp) : turn;
        if (tb >= nb) continue;
        float g[8][4];
#pragma unroll
        for (int n = 0; n < 8; ++n)
#pragma unroll
          for (int i = 0; i < 4; ++i) g[n][i] = 0.f;
        const uint32_t ca = smem_u32(st + G::C + (tb * 16 + (lane & 15)) * G::NROW + (lane >> 4) * 8);
        const uint32_t ba = smem_u32(st + G::B + ((lane & 7) + (lane >> 4) * 8) * G::NROW + ((lane >> 3) & 1) * 8);
#pragma unroll
        for (int ks = 0; ks < KS; ++ks) {
          uint32_t cf[4];
          ldmatrix_x4(cf, ca + ks * 32);
#pragma unroll
          for (int sb = 0; sb < 4; ++sb) {
            if (sb > tb) break;
            uint32_t bf[4];
            ldmatrix_x4(bf, ba + (sb * 16 * G::NROW + ks * 16) * 2);
            mma_bf16_16816(g[2 * sb], cf, bf[0], bf[1]);
            mma_bf16_16816(g[2 * sb + 1], cf, bf[2], bf[3]);
          }
        }
#pragma unroll
        for (int n = 0; n < 8; ++n) {
          if (n > 2 * tb + 1) break;
          const int c = n * 8 + dq;
          const float f0 = F[c], f1 = F[c + 1], d0 = D[c], d1 = D[c + 1];
#pragma unroll
          for (int half = 0; half < 2; ++half) {
            const int t = tb * 16 + r0 + half * 8;
            const float ft = F[t];
            float v0 = c <= t ? g[n][half * 2] * fast_exp2(ft - f0) * d0 : 0.f, v1 = c + 1 <= t ? g[n][half * 2 + 1] * fast_exp2(ft - f1) * d1 : 0.f;
            if (c == t) v0 += skip;
            if (c + 1 == t) v1 += skip;
            uint32_t hi, lo;
            split_pair(v0, v1, hi, lo);
            *reinterpret_cast<uint32_t*>(m_hi + t * G::MROW + c) = hi;
            *reinterpret_cast<uint32_t*>(m_lo + t * G::MROW + c) = lo;
          }
        }
      }
    }
    if (warp == 0 && chunk + 1 < n_chunks) steps(chunk + 1);
    if constexpr (!STATES) __syncthreads();       // M is complete
    // y^T = e^{F_t} S0^T C^T + x^T M^T, 64 tokens wide
    float o[8][4];
#pragma unroll
    for (int n = 0; n < 8; ++n)
#pragma unroll
      for (int i = 0; i < 4; ++i) o[n][i] = 0.f;
    if constexpr (!STATES) {
      const uint32_t cb = smem_u32(st + G::C + ((lane & 7) + (lane >> 4) * 8) * G::NROW + ((lane >> 3) & 1) * 8);
#pragma unroll
      for (int ks = 0; ks < KS; ++ks) {
        Split f;
        split_tile(S[2 * ks], S[2 * ks + 1], f);
        uint32_t cf[4][4];                          // (products that add to one accumulator are kept far apart)
#pragma unroll
        for (int n = 0; n < 4; ++n)
          if (n < nb) ldmatrix_x4(cf[n], cb + (n * 16 * G::NROW + ks * 16) * 2);
#pragma unroll
        for (int n = 0; n < 4; ++n) {
          if (n >= nb) break;
          mma_bf16_16816(o[2 * n], f.hi, cf[n][0], cf[n][1]);
          mma_bf16_16816(o[2 * n + 1], f.hi, cf[n][2], cf[n][3]);
        }
#pragma unroll
        for (int n = 0; n < 4; ++n) {
          if (n >= nb) break;
          mma_bf16_16816(o[2 * n], f.lo, cf[n][0], cf[n][1]);
          mma_bf16_16816(o[2 * n + 1], f.lo, cf[n][2], cf[n][3]);
        }
      }
#pragma unroll
      for (int n = 0; n < 8; ++n) {
        const float e0 = fast_exp2(F[n * 8 + dq]), e1 = fast_exp2(F[n * 8 + dq + 1]);
        o[n][0] *= e0; o[n][1] *= e1; o[n][2] *= e0; o[n][3] *= e1;
      }
    }
    const float f_end = F[Q - 1], keep = fast_exp2(f_end);
    kept += f_end;
#pragma unroll
    for (int j = 0; j < 2 * KS; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i) S[j][i] *= keep;
    const uint32_t xa = smem_u32(st + G::X + ((lane & 7) + (lane >> 4) * 8) * G::XROW + warp * 16 + ((lane >> 3) & 1) * 8);
    const uint32_t ma = smem_u32(m_hi + ((lane & 7) + (lane >> 4) * 8) * G::MROW + ((lane >> 3) & 1) * 8);
    const uint32_t bb = smem_u32(st + G::B + ((lane & 7) + ((lane >> 3) & 1) * 8) * G::NROW + (lane >> 4) * 8);
    constexpr uint32_t LOW = Q * G::MROW * 2;     // bytes from the high to the low part
#pragma unroll
    for (int k = 0; k < 4; ++k) {                 // 16 tokens s at a time
      if (k >= nb) break;
      uint32_t xf[4];
      ldmatrix_x4_trans(xf, xa + k * 16 * G::XROW * 2);
#pragma unroll
      for (int low = 0; low < (STATES ? 0 : 2); ++low) {
#pragma unroll
        for (int n = k; n < 4; ++n) {
          if (n >= nb) break;
          uint32_t m[4];
          ldmatrix_x4(m, ma + low * LOW + (n * 16 * G::MROW + k * 16) * 2);
          mma_bf16_16816(o[2 * n], xf, m[0], m[1]);
          mma_bf16_16816(o[2 * n + 1], xf, m[2], m[3]);
        }
      }
      Split w;                                    // the same values times e^{F_64 - F_s} dt_s
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int t = k * 16 + dq + half * 8;
        const float w0 = fast_exp2(f_end - F[t]) * D[t], w1 = fast_exp2(f_end - F[t + 1]) * D[t + 1];
        split_pair(bf16_lo(xf[2 * half]) * w0, bf16_hi(xf[2 * half]) * w1, w.hi[2 * half], w.lo[2 * half]);
        split_pair(bf16_lo(xf[2 * half + 1]) * w0, bf16_hi(xf[2 * half + 1]) * w1, w.hi[2 * half + 1], w.lo[2 * half + 1]);
      }
      constexpr int JB = KS % 4 == 0 ? 4 : KS % 3 == 0 ? 3 : KS % 2 == 0 ? 2 : 1;
#pragma unroll
      for (int j0 = 0; j0 < KS; j0 += JB) {
        uint32_t bf[JB][4];
#pragma unroll
        for (int j = 0; j < JB; ++j) ldmatrix_x4_trans(bf[j], bb + (k * 16 * G::NROW + (j0 + j) * 16) * 2);
#pragma unroll
        for (int j = 0; j < JB; ++j) {
          mma_bf16_16816(S[2 * (j0 + j)], w.hi, bf[j][0], bf[j][1]);
          mma_bf16_16816(S[2 * (j0 + j) + 1], w.hi, bf[j][2], bf[j][3]);
        }
#pragma unroll
        for (int j = 0; j < JB; ++j) {
          mma_bf16_16816(S[2 * (j0 + j)], w.lo, bf[j][0], bf[j][1]);
          mma_bf16_16816(S[2 * (j0 + j) + 1], w.lo, bf[j][2], bf[j][3]);
        }
      }
    }
    if constexpr (STATES) continue;
    // y goes out through the warp's own columns of x, which nobody needs any more
    __syncwarp();
    __nv_bfloat16* out_s = stages + (chunk & 1) * G::STAGE + G::X + warp * 16;
#pragma unroll
    for (int n = 0; n < 4; ++n) {
      const uint32_t r[4] = {pack_bf16(o[2 * n][0], o[2 * n][1]), pack_bf16(o[2 * n][2], o[2 * n][3]),
                             pack_bf16(o[2 * n + 1][0], o[2 * n + 1][1]), pack_bf16(o[2 * n + 1][2], o[2 * n + 1][3])};
      // matrices in turn: columns 0..7 and 8..15 of tokens 16 n .. 16 n + 7, then of the next eight
      stmatrix_x4_trans(smem_u32(out_s + (n * 16 + (lane & 7) + (lane >> 4) * 8) * G::XROW + ((lane >> 3) & 1) * 8), r);
    }
    __syncwarp();
    __nv_bfloat16* yg = static_cast<__nv_bfloat16*>(p.y) + static_cast<int64_t>(begin + chunk * Q) * p.y_stride + col0 + warp * 16;
    const int mine = min(16, cols - warp * 16);   // (not positive: a warp behind the last column)
    if (p.vec) {
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int t = i * 16 + (lane >> 1), c = (lane & 1) * 8;
        if (t < nt && c < mine) *reinterpret_cast<uint4*>(yg + t * p.y_stride + c) = *reinterpret_cast<const uint4*>(out_s + t * G::XROW + c);
      }
    } else {
      for (int e = lane; e < nt * 16; e += 32)
        if ((e & 15) < mine) yg[(e >> 4) * p.y_stride + (e & 15)] = out_s[(e >> 4) * G::XROW + (e & 15)];
    }
  }
  if (to == nullptr) return;
  if (STATES && blockIdx.x == 0 && tid == 0) p.seg_keep[static_cast<int64_t>(blockIdx.z) * p.heads + h] = fast_exp2(kept);
#pragma unroll
  for (int j = 0; j < 2 * KS; ++j)
#pragma unroll
    for (int i = 0; i < 4; ++i)
      if (in_state(j, i)) to[state_at(j, i)] = S[j][i];
}

// What each segment adds, and leaves of what was there, becomes the state in front of it.  A thread owns four state entries.
__global__ void __launch_bounds__(256) ssd_join_kernel(const SsdParams p) {
  const int s = blockIdx.z, h = blockIdx.y, i = (blockIdx.x * 256 + threadIdx.x) * 4;
  const int64_t states = static_cast<int64_t>(p.n) * p.vp;
  const int begin = p.cu[s], n_tok = p.cu[s + 1] - begin, segments = (n_tok + p.seg - 1) / p.seg;
  if (i >= states || segments <= 0) return;
  const int64_t slot = ssd_slot(p, s), first = seg_base(p, s);
  float4 S = make_float4(0.f, 0.f, 0.f, 0.f);
  if (slot >= 0 && p.positions[begin] != 0) S = *reinterpret_cast<const float4*>(p.state + (slot * p.heads + h) * states + i);
  constexpr int U = 8;                            // segments whose parts are requested before the first is used
  for (int k0 = 0; k0 < segments; k0 += U) {
    float4 added[U];
    float keep[U];
#pragma unroll
    for (int j = 0; j < U; ++j)
      if (k0 + j + 1 < segments) {
        added[j] = *reinterpret_cast<const float4*>(p.seg_state + ((first + k0 + j) * p.heads + h) * states + i);
        keep[j] = p.seg_keep[(first + k0 + j) * p.heads + h];
      }
#pragma unroll
    for (int j = 0; j < U; ++j) {
      if (k0 + j >= segments) return;
      *reinterpret_cast<float4*>(p.seg_state + ((first + k0 + j) * p.heads + h) * states + i) = S;
      if (k0 + j + 1 == segments) return;
      S.x = fmaf(S.x, keep[j], added[j].x); S.y = fmaf(S.y, keep[j], added[j].y);
      S.z = fmaf(S.z, keep[j], added[j].z); S.w = fmaf(S.w, keep[j], added[j].w);
    }
  }
}

// ---- launches ------------------------------------------------------------------------------------------------
template <class T>
static int launch_ssd_step(const SsdParams& p, cudaStream_t st) {
  const int tile = p.vp < 64 ? p.vp : 64, tiles = (p.vp + tile - 1) / tile, quads = tile / 4;
  if (p.num_seqs > 65535) return kUnsupportedShape;
  const int row_groups = (p.n + kStepRows - 1) / kStepRows;
  int nt = (row_groups * quads + 31) / 32 * 32;                      // N <= 256 and 16 quads at most: never more than 512 threads
  if (nt < (tile + 31) / 32 * 32) nt = (tile + 31) / 32 * 32;        // a thread per column at the end
  const size_t smem = (2 * static_cast<size_t>(p.n) + static_cast<size_t>(row_groups) * tile) * sizeof(float);
  ssd_step_kernel<T><<<dim3(p.heads * tiles, p.num_seqs), nt, smem, st>>>(p, tile, tiles);
  return cudaGetLastError() == cudaSuccess ? kOk : kLaunchFailed;
}

// Segment length of a ragged step (0: whole sequences).  Worth its first pass, about half of the second's work, where the longest
// sequence would be walked for twice as long as an even share of all tokens takes: two CTAs of 64 columns fit an SM.
static int ssd_segment(int tokens, int longest, int heads, int vdim) {
  const int64_t work = static_cast<int64_t>(tokens) * heads * ((vdim + 63) / 64), room = 2 * sm_count();
  if (longest < 1024 || longest > tokens || longest * room <= 2 * work) return 0;
  int seg = 256;
  while (seg < 1024 && work / (2 * seg) >= 2 * room) seg *= 2;
  return seg;
}
static int64_t ssd_segment_slots(int tokens, int num_seqs, int seg) { return tokens / seg + num_seqs; }

template <int KS, int WARPS, bool STATES>
static int launch_ssd_pass(const SsdParams& p, cudaStream_t st) {
  using G = SsdCfg<KS, WARPS, STATES>;
  struct Tag {};
  auto kernel = &ssd_chunk_kernel<KS, WARPS, STATES>;
  const int rc = opt_in_dynamic_smem<Tag>(reinterpret_cast<const void*>(kernel), G::SMEM);
  if (rc != kOk) return rc;
  const unsigned z = p.seg == 0 ? p.num_seqs : static_cast<unsigned>(ssd_segment_slots(p.tokens, p.num_seqs, p.seg));
  kernel<<<dim3((p.vdim + 16 * WARPS - 1) / (16 * WARPS), p.heads, z), G::THREADS, G::SMEM, st>>>(p);
  return cudaGetLastError() == cudaSuccess ? kOk : kLaunchFailed;
}

template <int KS, int WARPS>
static int launch_ssd_chunks(const SsdParams& p, cudaStream_t st) {
  if (p.seg != 0) {
    const int rc = launch_ssd_pass<KS, WARPS, true>(p, st);
    if (rc != kOk) return rc;
    ssd_join_kernel<<<dim3((p.n * p.vp / 4 + 255) / 256, p.heads, p.num_seqs), 256, 0, st>>>(p);
    if (cudaGetLastError() != cudaSuccess) return kLaunchFailed;
  }
  return launch_ssd_pass<KS, WARPS, false>(p, st);
}

template <int KS>
static int launch_ssd_columns(const SsdParams& p, cudaStream_t st) {
  const int tiles = (p.vdim + 15) / 16;
  // few (sequence, head) pairs: narrower CTAs, so that they spread over the SMs
  const int64_t pairs = static_cast<int64_t>(p.heads) * (p.seg == 0 ? p.num_seqs : ssd_segment_slots(p.tokens, p.num_seqs, p.seg));
  if (tiles >= 3 && pairs * ((tiles + 3) / 4) >= sm_count()) return launch_ssd_chunks<KS, 4>(p, st);
  return tiles >= 2 ? launch_ssd_chunks<KS, 2>(p, st) : launch_ssd_chunks<KS, 1>(p, st);
}

template <int NI>
static int launch_ssd_tokens(const SsdParams& p, cudaStream_t st) {
  ssd_tokens_kernel<NI><<<dim3((p.vdim + 15) / 16, p.heads, p.num_seqs), 128, 0, st>>>(p);
  return cudaGetLastError() == cudaSuccess ? kOk : kLaunchFailed;
}

template <class T>
static int launch_ssd(const SsdParams& p, cudaStream_t st) {
  if (p.cu == nullptr) return launch_ssd_step<T>(p, st);
  if (p.heads > 65535 || p.num_seqs > 65535 || (p.seg != 0 && ssd_segment_slots(p.tokens, p.num_seqs, p.seg) > 65535)) return kUnsupportedShape;
  if constexpr (sizeof(T) == 2) {
    switch (chunk_ks(p.n)) {
      case 1: return launch_ssd_columns<1>(p, st);
      case 2: return launch_ssd_columns<2>(p, st);
      case 3: return launch_ssd_columns<3>(p, st);
      case 4: return launch_ssd_columns<4>(p, st);
      case 6: return launch_ssd_columns<6>(p, st);
      case 8: return launch_ssd_columns<8>(p, st);
      case 12: return launch_ssd_columns<12>(p, st);
      case 16: return launch_ssd_columns<16>(p, st);
      default: return kUnsupportedShape;
    }
  } else {
    switch ((p.n + 31) / 32) {
      case 1: return launch_ssd_tokens<1>(p, st);
      case 2: return launch_ssd_tokens<2>(p, st);
      case 3: case 4: return launch_ssd_tokens<4>(p, st);
      default: return launch_ssd_tokens<8>(p, st);
    }
  }
}

// ---- the norm behind the gate ----------------------------------------------------------------------------------
struct GroupNormParams {
  const void* y; int64_t y_stride; const void* z; int64_t z_stride;
  const float* w;
  void* out; int64_t out_stride;
  int part, groups, rows;                       // coordinates per part; rows = tokens x groups
  float eps;
};

// A warp per part, eight parts per block, or (WIDE) a block per part; a thread keeps ITEMS vectors, and what a part has beyond them is
// read a second time
template <class T, int V, int ITEMS, bool WIDE>
__global__ void __launch_bounds__(256) gated_group_norm_kernel(const GroupNormParams p) {
  __shared__ float wsum[8];
  constexpr int TPR = WIDE ? 256 : 32;
  const int lane = threadIdx.x & 31, me = WIDE ? threadIdx.x : lane;
  const int r = WIDE ? blockIdx.x : blockIdx.x * 8 + (threadIdx.x >> 5);
  if (r >= p.rows) return;                      // (WIDE: the whole block)
  const int64_t t = r / p.groups, base = static_cast<int64_t>(r % p.groups) * p.part;
  const T *y = static_cast<const T*>(p.y) + t * p.y_stride + base, *z = static_cast<const T*>(p.z) + t * p.z_stride + base;
  T* out = static_cast<T*>(p.out) + t * p.out_stride + base;
  const int nvec = p.part / V;
  auto gated = [&](int i, float (&v)[V]) {
    float g[V];
    load_vec<T, V>(y + i * V, v);
    load_vec<T, V>(z + i * V, g);
#pragma unroll
    for (int j = 0; j < V; ++j) {
      const float sg = sizeof(T) == 2 ? fast_rcp(1.f + fast_exp2(g[j] * -1.4426950408889634f)) : sigmoid_f(g[j]);
      v[j] *= g[j] * sg;
    }
  };
  float v[ITEMS][V], ss = 0.f;
#pragma unroll
  for (int k = 0; k < ITEMS; ++k) {
    const int i = me + k * TPR;
    if (i >= nvec) continue;
    gated(i, v[k]);
#pragma unroll
    for (int j = 0; j < V; ++j) ss += v[k][j] * v[k][j];
  }
  for (int i = me + ITEMS * TPR; i < nvec; i += TPR) {
    float x[V];
    gated(i, x);
#pragma unroll
    for (int j = 0; j < V; ++j) ss += x[j] * x[j];
  }
  ss = warp_sum(ss);
  if constexpr (WIDE) {
    if (lane == 0) wsum[threadIdx.x >> 5] = ss;
    __syncthreads();
    ss = 0.f;
#pragma unroll
    for (int w = 0; w < 8; ++w) ss += wsum[w];
  }
  const float rstd = 1.f / sqrtf(ss / static_cast<float>(p.part) + p.eps);
  auto finish = [&](int i, float (&x)[V]) {
    float w[V];
    load_f32<V>(p.w + base + i * V, w);
#pragma unroll
    for (int j = 0; j < V; ++j) x[j] *= rstd * w[j];
    store_vec<T, V>(out + i * V, x);
  };
#pragma unroll
  for (int k = 0; k < ITEMS; ++k) {
    const int i = me + k * TPR;
    if (i < nvec) finish(i, v[k]);
  }
  for (int i = me + ITEMS * TPR; i < nvec; i += TPR) {
    float x[V];
    gated(i, x);
    finish(i, x);
  }
}

template <class T, int V>
static int launch_group_norm(const GroupNormParams& p, cudaStream_t st) {
  const int nvec = p.part / V;
  if (nvec <= 128) {
    const unsigned grid = static_cast<unsigned>((p.rows + 7) / 8);
    if (nvec <= 32) gated_group_norm_kernel<T, V, 1, false><<<grid, 256, 0, st>>>(p);
    else if (nvec <= 64) gated_group_norm_kernel<T, V, 2, false><<<grid, 256, 0, st>>>(p);
    else gated_group_norm_kernel<T, V, 4, false><<<grid, 256, 0, st>>>(p);
  } else {
    const unsigned grid = static_cast<unsigned>(p.rows);
    if (nvec <= 256) gated_group_norm_kernel<T, V, 1, true><<<grid, 256, 0, st>>>(p);
    else if (nvec <= 512) gated_group_norm_kernel<T, V, 2, true><<<grid, 256, 0, st>>>(p);
    else gated_group_norm_kernel<T, V, 4, true><<<grid, 256, 0, st>>>(p);
  }
  return cudaGetLastError() == cudaSuccess ? kOk : kLaunchFailed;
}

}  // namespace mvb

extern "C" size_t mvb_state_space_scratch_bytes(int dtype, int num_tokens, int num_seqs, int longest, int heads, int num_states, int vdim,
                                                int ragged) {
  using namespace mvb;
  if (!ragged || dtype != kBf16 || num_seqs <= 0 || heads <= 0 || num_states <= 0 || vdim <= 0) return 0;
  const int seg = ssd_segment(num_tokens, longest, heads, vdim);
  if (seg == 0) return 0;
  return static_cast<size_t>(ssd_segment_slots(num_tokens, num_seqs, seg)) * heads * (static_cast<size_t>(num_states) * ((vdim + 3) / 4 * 4) + 1) * sizeof(float);
}

extern "C" int mvb_state_space(int dtype, const void* x, const void* b, const void* c, int64_t xbc_row_stride, const void* dt,
                               int64_t dt_row_stride, const float* dt_bias, const float* a_log2e, const float* d, void* y,
                               int64_t y_row_stride, float* state, const int32_t* state_slots, int64_t num_slots,
                               const int32_t* cu_seqlens_q, const int64_t* positions, int num_seqs, int num_tokens, int longest, int heads,
                               int groups, int num_states, int vdim, void* scratch, size_t scratch_bytes, int32_t* dev_status, void* stream) {
  using namespace mvb;
  if (!x || !b || !c || !dt || !dt_bias || !a_log2e || !d || !y || !positions) return kInvalidArgument;
  if (num_seqs < 0 || num_tokens < 0 || heads <= 0 || groups <= 0 || heads % groups != 0 || num_states <= 0 || vdim <= 0) return kInvalidArgument;
  if (state != nullptr && (state_slots == nullptr || num_slots <= 0)) return kInvalidArgument;
  if (cu_seqlens_q == nullptr && num_seqs != num_tokens) return kInvalidArgument;
  if (dtype != kBf16 && dtype != kF32) return kInvalidArgument;
  if (!is_aligned(state, 16)) return kMisaligned;
  if (num_states > 256) return kUnsupportedShape;
  if (num_tokens == 0 || num_seqs == 0) return kOk;
  const bool vec = vdim % 8 == 0 && num_states % 8 == 0 && xbc_row_stride % 8 == 0 && y_row_stride % 8 == 0 && is_aligned(x, 16) &&
                   is_aligned(b, 16) && is_aligned(c, 16) && is_aligned(y, 16);
  SsdParams p{x, b, c, xbc_row_stride, dt, dt_row_stride, dt_bias, a_log2e, d, y, y_row_stride, state, state_slots, num_slots,
                    cu_seqlens_q, positions, num_seqs, num_tokens, heads, heads / groups, num_states, vdim, (vdim + 3) / 4 * 4, vec, 0, nullptr,
              nullptr, dev_status};
  if (dtype == kBf16 && cu_seqlens_q != nullptr) p.seg = ssd_segment(num_tokens, longest, heads, vdim);
  if (p.seg != 0) {
    if (!scratch || scratch_bytes < mvb_state_space_scratch_bytes(dtype, num_tokens, num_seqs, longest, heads, num_states, vdim, 1)) return kInvalidArgument;
    if (!is_aligned(scratch, 16)) return kMisaligned;
    p.seg_state = static_cast<float*>(scratch);
    p.seg_keep = p.seg_state + ssd_segment_slots(num_tokens, num_seqs, p.seg) * heads * num_states * p.vp;
  }
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return dtype == kBf16 ? launch_ssd<__nv_bfloat16>(p, st) : launch_ssd<float>(p, st);
}

extern "C" int mvb_gated_group_norm(int dtype, const void* y, int64_t y_row_stride, const void* z, int64_t z_row_stride, const float* weight,
                                    void* out, int64_t out_row_stride, int rows, int width, int groups, float eps, void* stream) {
  using namespace mvb;
  if (!y || !z || !weight || !out || rows < 0 || width <= 0 || groups <= 0 || width % groups != 0) return kInvalidArgument;
  if (dtype != kBf16 && dtype != kF32) return kInvalidArgument;
  if (rows == 0) return kOk;
  if (static_cast<int64_t>(rows) * groups > 0x7fffffffLL) return kUnsupportedShape;
  const GroupNormParams p{y, y_row_stride, z, z_row_stride, weight, out, out_row_stride, width / groups, groups, rows * groups, eps};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const int v = dtype == kBf16 ? 8 : 4;
  const bool vec = p.part % v == 0 && y_row_stride % v == 0 && z_row_stride % v == 0 && out_row_stride % v == 0 && is_aligned(y, 16) &&
                   is_aligned(z, 16) && is_aligned(out, 16) && is_aligned(weight, 16);
  if (dtype == kBf16) return vec ? launch_group_norm<__nv_bfloat16, 8>(p, st) : launch_group_norm<__nv_bfloat16, 1>(p, st);
  return vec ? launch_group_norm<float, 4>(p, st) : launch_group_norm<float, 1>(p, st);
}
