// Linear attention with decay on a packed ragged batch, state carried per sequence.  Per head, with S [dim, vdim] in fp32:
//
//   channel decay (EXP = false)    S <- diag(a) S + k v^T;  o = S^T q
//       a = sigmoid(raw + bias)^(1 / tau), a factor per key channel; q times q_scale
//   exponential gates (EXP = true) m' = max(f + m, i);  S <- e^{f + m - m'} S + e^{i - m'} k v^T;  n likewise with k alone;
//       o = S^T q / (max(|n . q|, e^{-m'}) + 1e-6);  i = cap tanh((raw_i + bias_i) / cap), f = log sigmoid(cap tanh((raw_f + bias_f) / cap))
//
// and then o / rms(o) * w * gate function (head_norm.cuh).  Columns of S never mix; n is one more column, whose value is 1.
// State slots: S [slots, heads, dim, vp] fp32, vp = vdim rounded up to 4; n [slots, heads, dim]; m [slots, heads].
//
// One token per sequence (linear_step_kernel): a CTA per (sequence, head); a thread holds RPT rows x 4 columns of S in registers,
// so the state is read once and written once (the roofline: HBM, 8 * dim * vdim bytes per head and sequence); gates, normaliser and
// the gated output norm are in the same kernel.
// Ragged step, bf16 activations: chunks of 16 tokens on the tensor cores (linear_chunks.cuh).
// Ragged step, fp32 activations: plain fp32 throughout.  linear_prep_kernel writes q, k and the gates once per token;
// linear_tokens_kernel walks a sequence's tokens with S in registers (8 row groups x 4 columns per warp, three shuffles for the sum
// over rows), operands staged TT tokens ahead with cp.async.
#include "chunk_common.cuh"
#include "head_norm.cuh"
#include "host_util.cuh"
#include "mini_vllm_b200.h"

#include <type_traits>

namespace mvb {

struct LinearParams {
  const void *q, *k, *v; int64_t qkv_stride;   // row t; q/k [heads, dim], v [heads, vdim]
  const void* decay; int64_t decay_stride;     // raw decay [heads, dim], or raw forget gate [heads]
  const void* igate; int64_t igate_stride;     // raw input gate [heads]
  const float *decay_bias, *igate_bias;        // [heads, dim] or [heads]; [heads]
  const void* gate; int64_t gate_stride;       // raw output gate [heads, vdim]
  const float* norm_w; int head_stride;        // [vdim] (stride 0) or [heads, vdim]
  void* out; int64_t out_stride;               // row t, [heads, vdim]
  float *S, *n, *m; const int32_t* slots; int64_t num_slots;
  const int32_t* cu; const int64_t* positions;
  int num_seqs, tokens, heads, dim, vdim, vp;
  float q_scale, inv_tau, cap, eps;
  // scratch of a ragged step: chunk records, or q, k (and decay) rows of dp; gates; o; n . q and m per token; m at the start
  uint8_t* records;
  float *qn, *kn, *gn, *fn, *in, *o, *nq, *mt, *m0;
  int dp, vtp;
  int* dev_status;
};

constexpr float kLog2e = 1.4426950408889634f, kLn2 = 0.6931471805599453f;

__device__ __forceinline__ int64_t linear_slot(const LinearParams& p, int s) {
  if (p.S == nullptr) return -1;
  const int64_t slot = p.slots[s];
  if (slot >= p.num_slots) { report(p.dev_status, kDevBadSlot, s); return -1; }
  return slot;
}
template <class T> __device__ __forceinline__ float log_sigmoid_of(float z) { return -softplus_of<T>(-z); }
__device__ __forceinline__ float capped(float z, float cap) { return cap * tanhf(z / cap); }
// log forget and log input gate of (row t, head h)
template <class T> __device__ __forceinline__ float log_forget(const LinearParams& p, int64_t t, int h) {
  return -softplus_f(-capped(to_f(static_cast<const T*>(p.decay)[t * p.decay_stride + h]) + p.decay_bias[h], p.cap));
}
template <class T> __device__ __forceinline__ float log_input(const LinearParams& p, int64_t t, int h) {
  return capped(to_f(static_cast<const T*>(p.igate)[t * p.igate_stride + h]) + p.igate_bias[h], p.cap);
}

// ---- one token per sequence ------------------------------------------------------------------------------
template <class T, bool EXP, int RPT>
__global__ void __launch_bounds__(512) linear_step_kernel(const LinearParams p, int tile_cols) {
  extern __shared__ __align__(16) float sm[];
  const int s = blockIdx.y, h = blockIdx.x;
  const int tid = threadIdx.x, nt = blockDim.x, warp = tid >> 5, lane = tid & 31, nw = nt >> 5;
  const int quads = tile_cols / 4, row_groups = (p.dim + RPT - 1) / RPT;
  float* red = sm;                              // [row groups][tile_cols]
  float* o_s = red + row_groups * tile_cols;    // [vdim]
  float* q_s = o_s + p.vdim;                    // [dim]
  float* k_s = q_s + p.dim;
  float* g_s = k_s + p.dim;
  __shared__ float wsum[16];
  const int64_t slot = linear_slot(p, s);
  const bool fresh = slot < 0 || p.positions[s] == 0;
  const int rg = tid / quads, cq = tid % quads;
  const int64_t hbase = (slot * p.heads + h) * static_cast<int64_t>(p.dim);
  const T* vrow = static_cast<const T*>(p.v) + s * p.qkv_stride + static_cast<int64_t>(h) * p.vdim;
  float keep = 1.f, nq = 0.f, m_new = 0.f;
  for (int col0 = 0; col0 < p.vp; col0 += tile_cols) {
    const int c = col0 + cq * 4;
    const bool active = rg < row_groups && c < p.vp;
    float4 S[RPT];
#pragma unroll
    for (int r = 0; r < RPT; ++r) {             // the state first: it is what the kernel waits for
      const int row = rg + r * row_groups;
      S[r] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (active && !fresh && row < p.dim) S[r] = *reinterpret_cast<const float4*>(p.S + (hbase + row) * p.vp + c);
    }
    float v[4];
#pragma unroll
    for (int j = 0; j < 4; ++j) v[j] = active && c + j < p.vdim ? to_f(vrow[c + j]) : 0.f;
    if (col0 == 0) {
      const T* qrow = static_cast<const T*>(p.q) + s * p.qkv_stride + static_cast<int64_t>(h) * p.dim;
      const T* krow = static_cast<const T*>(p.k) + s * p.qkv_stride + static_cast<int64_t>(h) * p.dim;
      float take = 1.f;
      if constexpr (EXP) {
        const float m = fresh ? 0.f : p.m[slot * p.heads + h];
        const float f = log_forget<T>(p, s, h), i = log_input<T>(p, s, h);
        m_new = fmaxf(f + m, i);
        keep = expf(f + m - m_new); take = expf(i - m_new);
      }
      for (int i = tid; i < p.dim; i += nt) {
        const float q = to_f(qrow[i]) * p.q_scale, k = to_f(krow[i]) * take;
        q_s[i] = q; k_s[i] = k;
        if constexpr (EXP) {
          const float n = (fresh ? 0.f : keep * p.n[hbase + i]) + k;
          if (slot >= 0) p.n[hbase + i] = n;
          nq += n * q;
        } else {
          const float z = to_f(static_cast<const T*>(p.decay)[s * p.decay_stride + static_cast<int64_t>(h) * p.dim + i]) + p.decay_bias[h * p.dim + i];
          g_s[i] = expf(log_sigmoid_of<T>(z) * p.inv_tau);
        }
      }
      if constexpr (EXP) {
        nq = warp_sum(nq);
        if (lane == 0) wsum[warp] = nq;
      }
      __syncthreads();
      if constexpr (EXP) {
        nq = 0.f;
        for (int w = 0; w < nw; ++w) nq += wsum[w];
        if (tid == 0 && slot >= 0) p.m[slot * p.heads + h] = m_new;      // (every thread has read the old one)
      }
    }
    float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int r = 0; r < RPT; ++r) {
      const int row = rg + r * row_groups;
      if (!active || row >= p.dim) continue;
      const float g = EXP ? keep : g_s[row], k = k_s[row], q = q_s[row];
      S[r].x = fmaf(k, v[0], S[r].x * g); S[r].y = fmaf(k, v[1], S[r].y * g);
      S[r].z = fmaf(k, v[2], S[r].z * g); S[r].w = fmaf(k, v[3], S[r].w * g);
      acc.x = fmaf(S[r].x, q, acc.x); acc.y = fmaf(S[r].y, q, acc.y); acc.z = fmaf(S[r].z, q, acc.z); acc.w = fmaf(S[r].w, q, acc.w);
      if (slot >= 0) *reinterpret_cast<float4*>(p.S + (hbase + row) * p.vp + c) = S[r];
    }
    if (active) *reinterpret_cast<float4*>(red + rg * tile_cols + cq * 4) = acc;
    __syncthreads();
    if (tid < tile_cols && col0 + tid < p.vdim) {
      float o = 0.f;
      for (int w = 0; w < row_groups; ++w) o += red[w * tile_cols + tid];
      o_s[col0 + tid] = o;
    }
    __syncthreads();                            // red is about to be reused; o_s is complete behind the last tile
  }
  const float d = EXP ? normaliser_scale(nq, m_new) : 1.f;
  float ss = 0.f;
  for (int i = tid; i < p.vdim; i += nt) { const float o = o_s[i] * d; ss += o * o; }
  ss = warp_sum(ss);
  if (lane == 0) wsum[warp] = ss;
  __syncthreads();
  ss = 0.f;
  for (int w = 0; w < nw; ++w) ss += wsum[w];
  const float r = d / sqrtf(ss / static_cast<float>(p.vdim) + p.eps);
  for (int i = tid; i < p.vdim; i += nt) {
    const float z = to_f(static_cast<const T*>(p.gate)[s * p.gate_stride + static_cast<int64_t>(h) * p.vdim + i]);
    const float gt = EXP ? sigmoid_f(z) : z * sigmoid_f(z);
    static_cast<T*>(p.out)[s * p.out_stride + static_cast<int64_t>(h) * p.vdim + i] = from_f<T>(o_s[i] * r * p.norm_w[h * p.head_stride + i] * gt);
  }
}

// the running maximum at the start of a ragged step, for kernels whose CTAs may start after another has stored the new one
__device__ __forceinline__ void stash_maximum(const LinearParams& p, int s, int h) {
  const int64_t slot = linear_slot(p, s);
  p.m0[s * p.heads + h] = slot < 0 || p.positions[p.cu[s]] == 0 ? 0.f : p.m[slot * p.heads + h];
}

// ---- ragged step, fp32: per-token operands ------------------------------------------------------------------------
template <bool EXP>
__global__ void __launch_bounds__(256) linear_prep_kernel(const LinearParams p) {
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int s = EXP ? seq_of_row(p.cu, p.num_seqs, t) : 0;
  for (int h = warp; h < p.heads; h += 8) {
    const float* qrow = static_cast<const float*>(p.q) + t * p.qkv_stride + static_cast<int64_t>(h) * p.dim;
    const float* krow = static_cast<const float*>(p.k) + t * p.qkv_stride + static_cast<int64_t>(h) * p.dim;
    const int64_t row = (static_cast<int64_t>(t) * p.heads + h) * p.dp;
    for (int i = lane; i < p.dp; i += 32) {
      p.qn[row + i] = i < p.dim ? qrow[i] * p.q_scale : 0.f;
      p.kn[row + i] = i < p.dim ? krow[i] : 0.f;
      if constexpr (!EXP)
        p.gn[row + i] = i < p.dim ? expf(log_sigmoid_of<float>(static_cast<const float*>(p.decay)[t * p.decay_stride + static_cast<int64_t>(h) * p.dim + i] +
                                                               p.decay_bias[h * p.dim + i]) * p.inv_tau) : 0.f;
    }
    if constexpr (EXP) {
      if (lane == 0) {
        p.fn[static_cast<int64_t>(t) * p.heads + h] = log_forget<float>(p, t, h);
        p.in[static_cast<int64_t>(t) * p.heads + h] = log_input<float>(p, t, h);
        if (p.cu[s] == t) stash_maximum(p, s, h);
      }
    }
  }
}

// ---- ragged step, fp32: the recurrence -------------------------------------------------------------------------
// NI: 32-row groups of S per column (dim <= 32 NI); a CTA owns 16 columns of one (sequence, head)
template <bool EXP, int NI>
__global__ void __launch_bounds__(128) linear_tokens_kernel(const LinearParams p) {
  constexpr int DP = 32 * NI, TT = NI <= 4 ? 16 : (NI <= 8 ? 8 : 4), NV = EXP ? 2 : 3;
  extern __shared__ __align__(16) float sm[];
  float* ops = sm;                                             // [2][TT][NV][DP]: q, k (, decay)
  float* v_s = sm + 2 * TT * NV * DP;                          // [TT][16]
  float* o_s = v_s + TT * 16;                                  // [TT][16]
  float* f_s = o_s + TT * 16;                                  // [TT] log forget, [TT] log input
  const int s = blockIdx.z, h = blockIdx.y, col0 = blockIdx.x * 16;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, rg = lane >> 2;
  const int cl = warp * 4 + (lane & 3), col = col0 + cl;
  const int begin = p.cu[s], n_tok = p.cu[s + 1] - begin;
  if (n_tok <= 0) return;
  const int64_t slot = linear_slot(p, s);
  const bool fresh = slot < 0 || p.positions[begin] == 0;
  const int64_t hbase = (slot * p.heads + h) * static_cast<int64_t>(p.dim);
  const bool holds = col < p.vdim + (EXP ? 1 : 0);             // column vdim is the normaliser
  auto state_at = [&](int row) -> float* { return EXP && col == p.vdim ? p.n + hbase + row : p.S + (hbase + row) * p.vp + col; };
  float S[NI][4];
#pragma unroll
  for (int i = 0; i < NI; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int row = i * 32 + rg * 4 + j;
      S[i][j] = (!fresh && holds && row < p.dim) ? *state_at(row) : 0.f;
    }
  float m = EXP ? p.m0[s * p.heads + h] : 0.f;
  auto stage = [&](int t0, int buf) {
    const int nt = min(TT, n_tok - t0);
    for (int e = tid; e < nt * NV * (DP / 4); e += 128) {
      const int tl = e / (NV * (DP / 4)), r = e % (NV * (DP / 4)), which = r / (DP / 4), q4 = r % (DP / 4);
      const float* src = (which == 0 ? p.qn : which == 1 ? p.kn : p.gn) + (static_cast<int64_t>(begin + t0 + tl) * p.heads + h) * DP;
      cp_async16(smem_u32(ops + ((buf * TT + tl) * NV + which) * DP + q4 * 4), src + q4 * 4);
    }
    cp_async_commit();
  };
  stage(0, 0);
  int buf = 0;
  for (int t0 = 0; t0 < n_tok; t0 += TT, buf ^= 1) {
    const int nt = min(TT, n_tok - t0);
    for (int e = tid; e < nt * 16; e += 128) {
      const int tl = e >> 4, c = col0 + (e & 15);
      const int64_t t = begin + t0 + tl;
      v_s[e] = c < p.vdim ? static_cast<const float*>(p.v)[t * p.qkv_stride + static_cast<int64_t>(h) * p.vdim + c] : (EXP && c == p.vdim ? 1.f : 0.f);
      if (EXP && (e & 15) == 0) { f_s[tl] = p.fn[t * p.heads + h]; f_s[TT + tl] = p.in[t * p.heads + h]; }
    }
    if (t0 + TT < n_tok) { stage(t0 + TT, buf ^ 1); cp_async_wait<1>(); } else { cp_async_wait<0>(); }
    __syncthreads();
    for (int tl = 0; tl < nt; ++tl) {
      const float* base = ops + (buf * TT + tl) * NV * DP + rg * 4;
      float keep = 1.f, val = v_s[tl * 16 + cl];
      if constexpr (EXP) {
        const float m_new = fmaxf(f_s[tl] + m, f_s[TT + tl]);
        keep = expf(f_s[tl] + m - m_new);
        val *= expf(f_s[TT + tl] - m_new);
        m = m_new;
        if (blockIdx.x == 0 && tid == 0) p.mt[static_cast<int64_t>(begin + t0 + tl) * p.heads + h] = m;
      }
      float oa[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        const float4 qv = *reinterpret_cast<const float4*>(base + i * 32), kv = *reinterpret_cast<const float4*>(base + DP + i * 32);
        float4 gv = make_float4(keep, keep, keep, keep);
        if constexpr (!EXP) gv = *reinterpret_cast<const float4*>(base + 2 * DP + i * 32);
        S[i][0] = fmaf(kv.x, val, S[i][0] * gv.x); S[i][1] = fmaf(kv.y, val, S[i][1] * gv.y);
        S[i][2] = fmaf(kv.z, val, S[i][2] * gv.z); S[i][3] = fmaf(kv.w, val, S[i][3] * gv.w);
        oa[0] = fmaf(S[i][0], qv.x, oa[0]); oa[1] = fmaf(S[i][1], qv.y, oa[1]);
        oa[2] = fmaf(S[i][2], qv.z, oa[2]); oa[3] = fmaf(S[i][3], qv.w, oa[3]);
      }
      float o = (oa[0] + oa[1]) + (oa[2] + oa[3]);
#pragma unroll
      for (int off = 4; off < 32; off <<= 1) o += __shfl_xor_sync(0xffffffffu, o, off);
      if (rg == 0) o_s[tl * 16 + cl] = o;
    }
    __syncthreads();
    for (int e = tid; e < nt * 16; e += 128) {
      const int64_t th = static_cast<int64_t>(begin + t0 + (e >> 4)) * p.heads + h;
      const int c = col0 + (e & 15);
      if (c < p.vdim) p.o[th * p.vdim + c] = o_s[e];
      else if (EXP && c == p.vdim) p.nq[th] = o_s[e];
    }
  }
  if (slot < 0) return;
  if (EXP && blockIdx.x == 0 && tid == 0) p.m[slot * p.heads + h] = m;
  if (holds) {
#pragma unroll
    for (int i = 0; i < NI; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int row = i * 32 + rg * 4 + j;
        if (row < p.dim) *state_at(row) = S[i][j];
      }
  }
}

}  // namespace mvb

#include "linear_chunks.cuh"

namespace mvb {

static int linear_row_pad(int dim) { return (dim + 31) / 32 * 32; }

template <class T, bool EXP>
static int launch_linear_norm(const LinearParams& p, cudaStream_t st) {
  HeadNormParams n{};
  n.o = p.o; n.gate = p.gate; n.gate_stride = p.gate_stride; n.norm_w = p.norm_w; n.head_stride = p.head_stride;
  n.out = p.out; n.out_stride = p.out_stride; n.nq = p.nq; n.m = p.mt;
  n.tokens = p.tokens; n.heads = p.heads; n.vdim = p.vdim; n.eps = p.eps; n.out_scale = 1.f;
  return launch_head_norm<T, EXP ? kGateSigmoid : kGateSilu, EXP>(n, st);
}

template <class T, bool EXP>
static int launch_linear_step(const LinearParams& p, cudaStream_t st) {
  const int tile = p.vp < 128 ? p.vp : 128, quads = tile / 4;
  if (p.num_seqs > 65535) return kUnsupportedShape;
  auto go = [&](auto tag) -> int {
    constexpr int RPT = decltype(tag)::value;
    const int row_groups = (p.dim + RPT - 1) / RPT;
    int nt = (row_groups * quads + 31) / 32 * 32;
    if (nt < (tile + 31) / 32 * 32) nt = (tile + 31) / 32 * 32;  // a thread per column at the end
    const size_t smem = (3 * static_cast<size_t>(p.dim) + p.vdim + static_cast<size_t>(row_groups) * tile) * sizeof(float);
    if (nt > 512 || smem > 47 * 1024) return kUnsupportedShape;
    linear_step_kernel<T, EXP, RPT><<<dim3(p.heads, p.num_seqs), nt, smem, st>>>(p, tile);
    return cudaGetLastError() == cudaSuccess ? kOk : kLaunchFailed;
  };
  // dim <= 256 and 32 quads at most: 16 rows per thread never take more than 512 threads
  return (p.dim + 7) / 8 * quads <= 256 ? go(std::integral_constant<int, 8>{}) : go(std::integral_constant<int, 16>{});
}

template <bool EXP, int NI>
static int launch_linear_tokens(const LinearParams& p, cudaStream_t st) {
  constexpr int DP = 32 * NI, TT = NI <= 4 ? 16 : (NI <= 8 ? 8 : 4), NV = EXP ? 2 : 3;
  constexpr size_t smem = (2 * TT * NV * DP + TT * 34) * sizeof(float);
  struct Tag {};
  const int rc = opt_in_dynamic_smem<Tag>(reinterpret_cast<const void*>(&linear_tokens_kernel<EXP, NI>), smem);
  if (rc != kOk) return rc;
  linear_tokens_kernel<EXP, NI><<<dim3((p.vdim + (EXP ? 1 : 0) + 15) / 16, p.heads, p.num_seqs), 128, smem, st>>>(p);
  return cudaGetLastError() == cudaSuccess ? kOk : kLaunchFailed;
}

template <class T, bool EXP>
static int launch_linear(const LinearParams& p, cudaStream_t st) {
  if (p.cu == nullptr) return launch_linear_step<T, EXP>(p, st);
  if (p.heads > 65535 || p.num_seqs > 65535) return kUnsupportedShape;
  int rc = kUnsupportedShape;
  if constexpr (sizeof(T) == 2) {
    switch (chunk_ks(p.dim)) {
      case 1: rc = launch_linear_chunks<EXP, 1>(p, st); break;
      case 2: rc = launch_linear_chunks<EXP, 2>(p, st); break;
      case 3: rc = launch_linear_chunks<EXP, 3>(p, st); break;
      case 4: rc = launch_linear_chunks<EXP, 4>(p, st); break;
      case 6: rc = launch_linear_chunks<EXP, 6>(p, st); break;
      case 8: rc = launch_linear_chunks<EXP, 8>(p, st); break;
      case 12: rc = launch_linear_chunks<EXP, 12>(p, st); break;
      case 16: rc = launch_linear_chunks<EXP, 16>(p, st); break;
      default: break;
    }
  } else {
    linear_prep_kernel<EXP><<<p.tokens, 256, 0, st>>>(p);
    if (cudaGetLastError() != cudaSuccess) return kLaunchFailed;
    switch (p.dp / 32) {
      case 1: rc = launch_linear_tokens<EXP, 1>(p, st); break;
      case 2: rc = launch_linear_tokens<EXP, 2>(p, st); break;
      case 3: rc = launch_linear_tokens<EXP, 3>(p, st); break;
      case 4: rc = launch_linear_tokens<EXP, 4>(p, st); break;
      case 5: rc = launch_linear_tokens<EXP, 5>(p, st); break;
      case 6: rc = launch_linear_tokens<EXP, 6>(p, st); break;
      case 7: rc = launch_linear_tokens<EXP, 7>(p, st); break;
      case 8: rc = launch_linear_tokens<EXP, 8>(p, st); break;
      default: break;
    }
  }
  return rc == kOk ? launch_linear_norm<T, EXP>(p, st) : rc;
}

static size_t pad64(size_t n) { return (n + 63) / 64 * 64; }

// floats of a ragged step's scratch, carved off `base` into p (base may be null: sizes only)
static size_t carve_linear_scratch(LinearParams& p, int dtype, bool exp_gates, float* base) {
  const size_t t = p.tokens, h = p.heads, rows = pad64(t * h * p.dp), th = pad64(t * h);
  size_t used = 0;
  auto take = [&](size_t n) { float* q = base == nullptr ? nullptr : base + used; used += n; return q; };
  if (dtype == kBf16) {
    p.records = reinterpret_cast<uint8_t*>(take(pad64((t / kChunk + p.num_seqs) * h * (linear_layout(chunk_ks(p.dim), p.vtp, exp_gates).total / 4))));
  } else {
    p.qn = take(rows); p.kn = take(rows);
    if (exp_gates) { p.fn = take(th); p.in = take(th); } else { p.gn = take(rows); }
  }
  p.o = take(pad64(t * h * p.vdim));
  if (exp_gates) { p.nq = take(th); p.mt = take(th); p.m0 = take(pad64(static_cast<size_t>(p.num_seqs) * h)); }
  return used;
}

static int run_linear(LinearParams& p, int dtype, bool exp_gates, void* scratch, size_t scratch_bytes, cudaStream_t st) {
  if (!p.q || !p.k || !p.v || !p.decay || !p.decay_bias || !p.gate || !p.norm_w || !p.out || !p.positions) return kInvalidArgument;
  if (p.num_seqs < 0 || p.tokens < 0 || p.heads <= 0 || p.dim <= 0 || p.vdim <= 0) return kInvalidArgument;
  if (p.S != nullptr && (p.slots == nullptr || p.num_slots <= 0 || (exp_gates && (!p.n || !p.m)))) return kInvalidArgument;
  if (p.cu == nullptr && p.num_seqs != p.tokens) return kInvalidArgument;
  if (dtype != kBf16 && dtype != kF32) return kInvalidArgument;
  if (!is_aligned(p.S, 16) || !is_aligned(scratch, 16)) return kMisaligned;
  if (p.dim > 256) return kUnsupportedShape;
  if (p.tokens == 0 || p.num_seqs == 0) return kOk;
  p.vp = (p.vdim + 3) / 4 * 4;
  p.dp = linear_row_pad(p.dim);
  p.vtp = linear_tiles(p);
  if (p.cu != nullptr) {
    if (!scratch || scratch_bytes < carve_linear_scratch(p, dtype, exp_gates, nullptr) * sizeof(float)) return kInvalidArgument;
    carve_linear_scratch(p, dtype, exp_gates, static_cast<float*>(scratch));
  }
  if (exp_gates) return dtype == kBf16 ? launch_linear<__nv_bfloat16, true>(p, st) : launch_linear<float, true>(p, st);
  return dtype == kBf16 ? launch_linear<__nv_bfloat16, false>(p, st) : launch_linear<float, false>(p, st);
}

}  // namespace mvb

extern "C" size_t mvb_linear_attn_scratch_bytes(int dtype, int num_tokens, int num_seqs, int heads, int dim, int vdim, int exp_gates,
                                                int ragged) {
  using namespace mvb;
  if (num_tokens <= 0 || num_seqs <= 0 || heads <= 0 || dim <= 0 || dim > 256 || vdim <= 0) return 0;
  if (!ragged) return 64;
  LinearParams p{};
  p.tokens = num_tokens; p.num_seqs = num_seqs; p.heads = heads; p.dim = dim; p.vdim = vdim;
  p.dp = linear_row_pad(dim);
  p.vtp = linear_tiles(p);
  return carve_linear_scratch(p, dtype, exp_gates != 0, nullptr) * sizeof(float);
}

extern "C" int mvb_gated_linear(int dtype, const void* q, const void* k, const void* v, int64_t qkv_row_stride, const void* decay,
                                int64_t decay_row_stride, const float* decay_bias, float inv_tau, const void* gate,
                                int64_t gate_row_stride, const float* norm_weight, void* out, int64_t out_row_stride, float* state,
                                const int32_t* state_slots, int64_t num_slots, const int32_t* cu_seqlens_q, const int64_t* positions,
                                int num_seqs, int num_tokens, int heads, int dim, int vdim, float q_scale, float eps, void* scratch,
                                size_t scratch_bytes, int32_t* dev_status, void* stream) {
  using namespace mvb;
  if (!(inv_tau > 0.f)) return kInvalidArgument;
  LinearParams p{};
  p.q = q; p.k = k; p.v = v; p.qkv_stride = qkv_row_stride;
  p.decay = decay; p.decay_stride = decay_row_stride; p.decay_bias = decay_bias; p.inv_tau = inv_tau;
  p.gate = gate; p.gate_stride = gate_row_stride; p.norm_w = norm_weight; p.head_stride = 0;
  p.out = out; p.out_stride = out_row_stride;
  p.S = state; p.slots = state_slots; p.num_slots = num_slots;
  p.cu = cu_seqlens_q; p.positions = positions;
  p.num_seqs = num_seqs; p.tokens = num_tokens; p.heads = heads; p.dim = dim; p.vdim = vdim;
  p.q_scale = q_scale; p.eps = eps; p.cap = 1.f; p.dev_status = dev_status;
  return run_linear(p, dtype, false, scratch, scratch_bytes, static_cast<cudaStream_t>(stream));
}

extern "C" int mvb_mlstm(int dtype, const void* q, const void* k, const void* v, int64_t qkv_row_stride, const void* forget,
                         int64_t forget_row_stride, const float* forget_bias, const void* input, int64_t input_row_stride,
                         const float* input_bias, float cap, const void* gate, int64_t gate_row_stride, const float* norm_weight,
                         void* out, int64_t out_row_stride, float* state, float* normaliser, float* maximum, const int32_t* state_slots,
                         int64_t num_slots, const int32_t* cu_seqlens_q, const int64_t* positions, int num_seqs, int num_tokens,
                         int heads, int dim, int vdim, float q_scale, float eps, void* scratch, size_t scratch_bytes,
                         int32_t* dev_status, void* stream) {
  using namespace mvb;
  if (!(cap > 0.f) || !input || !input_bias) return kInvalidArgument;
  LinearParams p{};
  p.q = q; p.k = k; p.v = v; p.qkv_stride = qkv_row_stride;
  p.decay = forget; p.decay_stride = forget_row_stride; p.decay_bias = forget_bias;
  p.igate = input; p.igate_stride = input_row_stride; p.igate_bias = input_bias; p.cap = cap;
  p.gate = gate; p.gate_stride = gate_row_stride; p.norm_w = norm_weight; p.head_stride = vdim;
  p.out = out; p.out_stride = out_row_stride;
  p.S = state; p.n = normaliser; p.m = maximum; p.slots = state_slots; p.num_slots = num_slots;
  p.cu = cu_seqlens_q; p.positions = positions;
  p.num_seqs = num_seqs; p.tokens = num_tokens; p.heads = heads; p.dim = dim; p.vdim = vdim;
  p.q_scale = q_scale; p.eps = eps; p.inv_tau = 1.f; p.dev_status = dev_status;
  return run_linear(p, dtype, true, scratch, scratch_bytes, static_cast<cudaStream_t>(stream));
}
