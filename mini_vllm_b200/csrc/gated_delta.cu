// Gated delta rule with a decay per head and key channel, on a packed ragged batch, state carried per sequence.
//
// Per head, with S [dim, vdim] in fp32:
//   S <- g * S (row i by g_i);  e = beta (v - S^T k);  S <- S + k e^T;  o = S^T q
//   q, k: unit vectors of the convolved projections (q also times dim^-1/2), g = exp(-exp(A_log) softplus(raw + bias)),
//   beta = sigmoid(raw_b); then o / rms(o) * w * sigmoid(gate), times the mixer's output factor.
//
// Columns of S never mix, so any cut of vdim is free.  State slots: [slots, heads, dim, vp] fp32, vp = vdim rounded up to 4.
//
// One token per sequence (delta_step_kernel): a CTA per (sequence, head, tile of at most 128 columns); a thread holds RPT
// rows x 4 columns of S in registers, so the state is read once and written once (the roofline: HBM, 8 * dim * vdim bytes per
// head and sequence); gates, norms and, when one tile covers the head, the gated output norm are in the same kernel.
// Ragged step, bf16 activations: chunks of 16 tokens on the tensor cores (delta_chunks.cuh).
// Ragged step, fp32 activations: plain fp32 throughout.  delta_prep_kernel writes q, k, g as [tokens, heads, dp] once per token;
// delta_tokens_kernel walks a sequence's tokens with S in registers (8 row groups x 4 columns per warp, the sum over rows is
// three shuffles), operands staged TT tokens ahead with cp.async.
// head_norm_kernel (head_norm.cuh) finishes the rows of either.
#include "chunk_common.cuh"
#include "head_norm.cuh"
#include "host_util.cuh"
#include "mini_vllm_b200.h"

#include <type_traits>

namespace mvb {

struct DeltaParams {
  const void *q, *k, *v; int64_t qkv_stride;   // convolved, row t; q/k [kv_heads, dim], v [heads, vdim]
  const void* a; int64_t a_stride;             // raw decay [heads, dim]
  const void* b; int64_t b_stride;             // raw beta [heads]
  const void* gate; int64_t gate_stride;       // raw output gate [heads, vdim]
  const float *exp_a, *dt_bias, *norm_w;       // exp(A_log) [heads], [heads, dim], [vdim]
  void* out; int64_t out_stride;               // row t, [heads, vdim]
  float* state; const int32_t* slots; int64_t num_slots;
  const int32_t* cu; const int64_t* positions;
  int num_seqs, tokens, heads, kv_heads, dim, vdim, vp;
  float q_scale, eps, out_scale;
  // scratch of a ragged step: q, k per kv head, g per head (rows of dp, zero in the padding), beta, o
  float *qn, *kn, *gn, *beta, *o;
  int dp;
  int* dev_status;
};

constexpr float kUnitEps = 1e-6f;              // inside the root of the unit norm

__device__ __forceinline__ int64_t delta_slot(const DeltaParams& p, int s) {
  if (p.state == nullptr) return -1;
  const int64_t slot = p.slots[s];
  if (slot >= p.num_slots) { report(p.dev_status, kDevBadSlot, s); return -1; }
  return slot;
}
__device__ __forceinline__ float decay_of(float raw, float bias, float exp_a) { return expf(-exp_a * softplus_f(raw + bias)); }

// ---- one token per sequence ------------------------------------------------------------------------------
template <class T, int RPT>
__global__ void __launch_bounds__(512) delta_step_kernel(const DeltaParams p, int tile_cols) {
  extern __shared__ float sm[];
  const int s = blockIdx.z, h = blockIdx.x, kvh = h / (p.heads / p.kv_heads);
  const int tid = threadIdx.x, nt = blockDim.x, warp = tid >> 5, lane = tid & 31, nw = nt >> 5;
  const int col0 = blockIdx.y * tile_cols, cols = min(tile_cols, p.vp - col0), quads = tile_cols / 4;
  float* q_s = sm;                              // [dim]
  float* k_s = q_s + p.dim;
  float* g_s = k_s + p.dim;
  float* red = g_s + p.dim;                     // [row groups][tile_cols]
  __shared__ float wsum[2][16];
  const int64_t slot = delta_slot(p, s);
  const bool fresh = slot < 0 || p.positions[s] == 0;
  // the state first: it is what the kernel waits for
  const int rg = tid / quads, cq = tid % quads, row_groups = (p.dim + RPT - 1) / RPT;
  const bool active = rg < row_groups && cq * 4 < cols;
  const int64_t sbase = ((slot * p.heads + h) * p.dim) * static_cast<int64_t>(p.vp) + col0 + cq * 4;
  float4 S[RPT];
#pragma unroll
  for (int r = 0; r < RPT; ++r) {
    const int row = rg + r * row_groups;
    S[r] = make_float4(0.f, 0.f, 0.f, 0.f);
    if (active && !fresh && row < p.dim) S[r] = *reinterpret_cast<const float4*>(p.state + sbase + static_cast<int64_t>(row) * p.vp);
  }
  float qq = 0.f, kk = 0.f;
  const T* qrow = static_cast<const T*>(p.q) + s * p.qkv_stride + static_cast<int64_t>(kvh) * p.dim;
  const T* krow = static_cast<const T*>(p.k) + s * p.qkv_stride + static_cast<int64_t>(kvh) * p.dim;
  const T* arow = static_cast<const T*>(p.a) + s * p.a_stride + static_cast<int64_t>(h) * p.dim;
  const float ea = p.exp_a[h];
  for (int i = tid; i < p.dim; i += nt) {
    const float qv = to_f(qrow[i]), kv = to_f(krow[i]);
    q_s[i] = qv; k_s[i] = kv;
    g_s[i] = decay_of(to_f(arow[i]), p.dt_bias[h * p.dim + i], ea);
    qq += qv * qv; kk += kv * kv;
  }
  qq = warp_sum(qq); kk = warp_sum(kk);
  if (lane == 0) { wsum[0][warp] = qq; wsum[1][warp] = kk; }
  __syncthreads();
  qq = kk = 0.f;
  for (int w = 0; w < nw; ++w) { qq += wsum[0][w]; kk += wsum[1][w]; }
  const float rq = p.q_scale / sqrtf(qq + kUnitEps), rk = 1.f / sqrtf(kk + kUnitEps);
  const float beta = sigmoid_f(to_f(static_cast<const T*>(p.b)[s * p.b_stride + h]));

  float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int r = 0; r < RPT; ++r) {
    const int row = rg + r * row_groups;
    if (!active || row >= p.dim) continue;
    const float g = g_s[row], k = k_s[row] * rk;
    S[r].x *= g; S[r].y *= g; S[r].z *= g; S[r].w *= g;
    acc.x = fmaf(S[r].x, k, acc.x); acc.y = fmaf(S[r].y, k, acc.y); acc.z = fmaf(S[r].z, k, acc.z); acc.w = fmaf(S[r].w, k, acc.w);
  }
  if (active) *reinterpret_cast<float4*>(red + rg * tile_cols + cq * 4) = acc;
  __syncthreads();
  float4 e = make_float4(0.f, 0.f, 0.f, 0.f);
  if (active) {
    float4 pr = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int w = 0; w < row_groups; ++w) {
      const float4 x = *reinterpret_cast<const float4*>(red + w * tile_cols + cq * 4);
      pr.x += x.x; pr.y += x.y; pr.z += x.z; pr.w += x.w;
    }
    const T* vrow = static_cast<const T*>(p.v) + s * p.qkv_stride + static_cast<int64_t>(h) * p.vdim;
    const int c = col0 + cq * 4;
    e.x = c + 0 < p.vdim ? beta * (to_f(vrow[c + 0]) - pr.x) : 0.f;
    e.y = c + 1 < p.vdim ? beta * (to_f(vrow[c + 1]) - pr.y) : 0.f;
    e.z = c + 2 < p.vdim ? beta * (to_f(vrow[c + 2]) - pr.z) : 0.f;
    e.w = c + 3 < p.vdim ? beta * (to_f(vrow[c + 3]) - pr.w) : 0.f;
  }
  __syncthreads();                              // red is about to be reused
  acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int r = 0; r < RPT; ++r) {
    const int row = rg + r * row_groups;
    if (!active || row >= p.dim) continue;
    const float k = k_s[row] * rk, q = q_s[row] * rq;
    S[r].x = fmaf(k, e.x, S[r].x); S[r].y = fmaf(k, e.y, S[r].y); S[r].z = fmaf(k, e.z, S[r].z); S[r].w = fmaf(k, e.w, S[r].w);
    acc.x = fmaf(S[r].x, q, acc.x); acc.y = fmaf(S[r].y, q, acc.y); acc.z = fmaf(S[r].z, q, acc.z); acc.w = fmaf(S[r].w, q, acc.w);
    if (slot >= 0) *reinterpret_cast<float4*>(p.state + sbase + static_cast<int64_t>(row) * p.vp) = S[r];
  }
  if (active) *reinterpret_cast<float4*>(red + rg * tile_cols + cq * 4) = acc;
  __syncthreads();
  // columns of the tile: sum the row groups, then norm and gate (one tile) or leave o for the finishing kernel
  const bool whole = gridDim.y == 1;
  float o_mine = 0.f, ss = 0.f;
  if (tid < cols && col0 + tid < p.vdim) {
    for (int w = 0; w < row_groups; ++w) o_mine += red[w * tile_cols + tid];
    if (!whole) p.o[(static_cast<int64_t>(s) * p.heads + h) * p.vdim + col0 + tid] = o_mine;
    ss = o_mine * o_mine;
  }
  if (!whole) return;
  ss = warp_sum(ss);
  __syncthreads();
  if (lane == 0) wsum[0][warp] = ss;
  __syncthreads();
  ss = 0.f;
  for (int w = 0; w < nw; ++w) ss += wsum[0][w];
  if (tid < p.vdim) {
    const float r = 1.f / sqrtf(ss / static_cast<float>(p.vdim) + p.eps);
    const float gt = sigmoid_f(to_f(static_cast<const T*>(p.gate)[s * p.gate_stride + static_cast<int64_t>(h) * p.vdim + tid]));
    static_cast<T*>(p.out)[s * p.out_stride + static_cast<int64_t>(h) * p.vdim + tid] = from_f<T>(o_mine * r * p.norm_w[tid] * gt * p.out_scale);
  }
}

// ---- ragged step: per-token operands ------------------------------------------------------------------------
template <class T>
__global__ void __launch_bounds__(256) delta_prep_kernel(const DeltaParams p) {
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  for (int it = warp; it < p.kv_heads + p.heads; it += 8) {
    if (it < p.kv_heads) {
      const T* qrow = static_cast<const T*>(p.q) + t * p.qkv_stride + static_cast<int64_t>(it) * p.dim;
      const T* krow = static_cast<const T*>(p.k) + t * p.qkv_stride + static_cast<int64_t>(it) * p.dim;
      float qq = 0.f, kk = 0.f;
      for (int i = lane; i < p.dim; i += 32) { const float a = to_f(qrow[i]), b = to_f(krow[i]); qq += a * a; kk += b * b; }
      qq = warp_sum(qq); kk = warp_sum(kk);
      const float rq = p.q_scale / sqrtf(qq + kUnitEps), rk = 1.f / sqrtf(kk + kUnitEps);
      float* qo = p.qn + (static_cast<int64_t>(t) * p.kv_heads + it) * p.dp;
      float* ko = p.kn + (static_cast<int64_t>(t) * p.kv_heads + it) * p.dp;
      for (int i = lane; i < p.dp; i += 32) {
        qo[i] = i < p.dim ? to_f(qrow[i]) * rq : 0.f;
        ko[i] = i < p.dim ? to_f(krow[i]) * rk : 0.f;
      }
    } else {
      const int h = it - p.kv_heads;
      const T* arow = static_cast<const T*>(p.a) + t * p.a_stride + static_cast<int64_t>(h) * p.dim;
      const float ea = p.exp_a[h];
      float* go = p.gn + (static_cast<int64_t>(t) * p.heads + h) * p.dp;
      for (int i = lane; i < p.dp; i += 32) go[i] = i < p.dim ? decay_of(to_f(arow[i]), p.dt_bias[h * p.dim + i], ea) : 0.f;
      if (lane == 0) p.beta[static_cast<int64_t>(t) * p.heads + h] = sigmoid_f(to_f(static_cast<const T*>(p.b)[t * p.b_stride + h]));
    }
  }
}

// ---- ragged step: the recurrence -------------------------------------------------------------------------
// NI: 32-row groups of S per column (dim <= 32 NI); a CTA owns 16 columns of one (sequence, head)
template <class T, int NI>
__global__ void __launch_bounds__(128) delta_tokens_kernel(const DeltaParams p) {
  constexpr int DP = 32 * NI, TT = NI <= 4 ? 16 : (NI <= 8 ? 8 : 4);
  extern __shared__ __align__(16) float sm[];
  float* ops = sm;                                             // [2][TT][3][DP]: q, k, g
  float* v_s = sm + 2 * TT * 3 * DP;                           // [TT][16]
  float* b_s = v_s + TT * 16;                                  // [TT]
  float* o_s = b_s + TT;                                       // [TT][16]
  const int s = blockIdx.z, h = blockIdx.y, kvh = h / (p.heads / p.kv_heads), col0 = blockIdx.x * 16;
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, rg = lane >> 2;
  const int cl = warp * 4 + (lane & 3), col = col0 + cl;
  const int begin = p.cu[s], n_tok = p.cu[s + 1] - begin;
  if (n_tok <= 0) return;
  const int64_t slot = delta_slot(p, s);
  const bool fresh = slot < 0 || p.positions[begin] == 0;
  const int64_t sbase = ((slot * p.heads + h) * p.dim) * static_cast<int64_t>(p.vp) + col;
  float S[NI][4];
#pragma unroll
  for (int i = 0; i < NI; ++i)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int row = i * 32 + rg * 4 + j;
      S[i][j] = (!fresh && col < p.vdim && row < p.dim) ? p.state[sbase + static_cast<int64_t>(row) * p.vp] : 0.f;
    }
  auto stage = [&](int t0, int buf) {
    const int nt = min(TT, n_tok - t0);
    for (int e = tid; e < nt * 3 * (DP / 4); e += 128) {
      const int tl = e / (3 * (DP / 4)), r = e % (3 * (DP / 4)), which = r / (DP / 4), q4 = r % (DP / 4);
      const int64_t t = begin + t0 + tl;
      const float* src = which == 0 ? p.qn + (t * p.kv_heads + kvh) * DP : which == 1 ? p.kn + (t * p.kv_heads + kvh) * DP
                                                                                  : p.gn + (t * p.heads + h) * DP;
      cp_async16(smem_u32(ops + ((buf * TT + tl) * 3 + which) * DP + q4 * 4), src + q4 * 4);
    }
    cp_async_commit();
  };
  stage(0, 0);
  int buf = 0;
  for (int t0 = 0; t0 < n_tok; t0 += TT, buf ^= 1) {
    const int nt = min(TT, n_tok - t0);
    for (int e = tid; e < nt * 16; e += 128) {
      const int tl = e >> 4, c = e & 15;
      const int64_t t = begin + t0 + tl;
      v_s[e] = col0 + c < p.vdim ? to_f(static_cast<const T*>(p.v)[t * p.qkv_stride + static_cast<int64_t>(h) * p.vdim + col0 + c]) : 0.f;
      if (c == 0) b_s[tl] = p.beta[t * p.heads + h];
    }
    if (t0 + TT < n_tok) { stage(t0 + TT, buf ^ 1); cp_async_wait<1>(); } else { cp_async_wait<0>(); }
    __syncthreads();
    for (int tl = 0; tl < nt; ++tl) {
      const float* base = ops + (buf * TT + tl) * 3 * DP + rg * 4;
      float kk[NI][4], pr[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        const float4 kv = *reinterpret_cast<const float4*>(base + DP + i * 32);
        const float4 gv = *reinterpret_cast<const float4*>(base + 2 * DP + i * 32);
        kk[i][0] = kv.x; kk[i][1] = kv.y; kk[i][2] = kv.z; kk[i][3] = kv.w;
        S[i][0] *= gv.x; S[i][1] *= gv.y; S[i][2] *= gv.z; S[i][3] *= gv.w;
#pragma unroll
        for (int j = 0; j < 4; ++j) pr[j] = fmaf(S[i][j], kk[i][j], pr[j]);
      }
      float pred = (pr[0] + pr[1]) + (pr[2] + pr[3]);
#pragma unroll
      for (int off = 4; off < 32; off <<= 1) pred += __shfl_xor_sync(0xffffffffu, pred, off);
      const float e = b_s[tl] * (v_s[tl * 16 + cl] - pred);
      float oa[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        const float4 qv = *reinterpret_cast<const float4*>(base + i * 32);
        const float qq[4] = {qv.x, qv.y, qv.z, qv.w};
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          S[i][j] = fmaf(kk[i][j], e, S[i][j]);
          oa[j] = fmaf(S[i][j], qq[j], oa[j]);
        }
      }
      float o = (oa[0] + oa[1]) + (oa[2] + oa[3]);
#pragma unroll
      for (int off = 4; off < 32; off <<= 1) o += __shfl_xor_sync(0xffffffffu, o, off);
      if (rg == 0) o_s[tl * 16 + cl] = o;
    }
    __syncthreads();
    for (int e = tid; e < nt * 16; e += 128) {
      const int tl = e >> 4, c = e & 15;
      if (col0 + c < p.vdim) p.o[(static_cast<int64_t>(begin + t0 + tl) * p.heads + h) * p.vdim + col0 + c] = o_s[e];
    }
  }
  if (slot >= 0 && col < p.vdim) {
#pragma unroll
    for (int i = 0; i < NI; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const int row = i * 32 + rg * 4 + j;
        if (row < p.dim) p.state[sbase + static_cast<int64_t>(row) * p.vp] = S[i][j];
      }
  }
}

}  // namespace mvb

#include "delta_chunks.cuh"

namespace mvb {

template <class T>
static int launch_gated_norm(const DeltaParams& p, cudaStream_t st) {
  HeadNormParams n{};
  n.o = p.o; n.gate = p.gate; n.gate_stride = p.gate_stride; n.norm_w = p.norm_w; n.out = p.out; n.out_stride = p.out_stride;
  n.tokens = p.tokens; n.heads = p.heads; n.vdim = p.vdim; n.eps = p.eps; n.out_scale = p.out_scale;
  return launch_head_norm<T, kGateSigmoid>(n, st);
}

static int delta_row_pad(int dim) { return (dim + 31) / 32 * 32; }

static int step_tile_cols(int vp) {                            // columns per CTA: the whole head up to 128, else 128
  return vp <= 128 ? vp : 128;
}

template <class T>
static int launch_step(const DeltaParams& p, cudaStream_t st) {
  const int tile = step_tile_cols(p.vp), tiles = (p.vp + tile - 1) / tile, quads = tile / 4;
  if (p.num_seqs > 65535) return kUnsupportedShape;
  auto go = [&](auto tag) -> int {
    constexpr int RPT = decltype(tag)::value;
    const int row_groups = (p.dim + RPT - 1) / RPT;
    int nt = (row_groups * quads + 31) / 32 * 32;
    if (nt < (tile + 31) / 32 * 32) nt = (tile + 31) / 32 * 32;  // a thread per column at the end
    const size_t smem = (3 * static_cast<size_t>(p.dim) + static_cast<size_t>(row_groups) * tile) * sizeof(float);
    if (nt > 512 || smem > 47 * 1024) return kUnsupportedShape;
    delta_step_kernel<T, RPT><<<dim3(p.heads, tiles, p.num_seqs), nt, smem, st>>>(p, tile);
    return cudaGetLastError() == cudaSuccess ? kOk : kLaunchFailed;
  };
  int rc = kUnsupportedShape;
  const int groups8 = (p.dim + 7) / 8, groups16 = (p.dim + 15) / 16;
  if (groups8 * quads <= 256) rc = go(std::integral_constant<int, 8>{});
  else if (groups16 * quads <= 512) rc = go(std::integral_constant<int, 16>{});
  else rc = go(std::integral_constant<int, 32>{});
  if (rc == kOk && tiles > 1) rc = launch_gated_norm<T>(p, st);
  return rc;
}

template <class T, int NI>
static int launch_tokens_ni(const DeltaParams& p, cudaStream_t st) {
  constexpr int DP = 32 * NI, TT = NI <= 4 ? 16 : (NI <= 8 ? 8 : 4);
  constexpr size_t smem = (2 * TT * 3 * DP + TT * 33) * sizeof(float);
  struct Tag {};
  const int rc = opt_in_dynamic_smem<Tag>(reinterpret_cast<const void*>(&delta_tokens_kernel<T, NI>), smem);
  if (rc != kOk) return rc;
  delta_tokens_kernel<T, NI><<<dim3((p.vdim + 15) / 16, p.heads, p.num_seqs), 128, smem, st>>>(p);
  return cudaGetLastError() == cudaSuccess ? kOk : kLaunchFailed;
}

template <class T>
static int launch_delta(const DeltaParams& p, cudaStream_t st) {
  if (p.cu == nullptr) return launch_step<T>(p, st);
  if (p.heads > 65535 || p.num_seqs > 65535) return kUnsupportedShape;
  if constexpr (sizeof(T) == 2) {
    uint8_t* records = reinterpret_cast<uint8_t*>(p.qn);
    int rc = kUnsupportedShape;
    switch (chunk_ks(p.dim)) {
      case 1: rc = launch_delta_chunks<T, 1>(p, records, st); break;
      case 2: rc = launch_delta_chunks<T, 2>(p, records, st); break;
      case 3: rc = launch_delta_chunks<T, 3>(p, records, st); break;
      case 4: rc = launch_delta_chunks<T, 4>(p, records, st); break;
      case 6: rc = launch_delta_chunks<T, 6>(p, records, st); break;
      case 8: rc = launch_delta_chunks<T, 8>(p, records, st); break;
      case 12: rc = launch_delta_chunks<T, 12>(p, records, st); break;
      case 16: rc = launch_delta_chunks<T, 16>(p, records, st); break;
      default: break;
    }
    return rc == kOk ? launch_gated_norm<T>(p, st) : rc;
  } else {
  delta_prep_kernel<T><<<p.tokens, 256, 0, st>>>(p);
  if (cudaGetLastError() != cudaSuccess) return kLaunchFailed;
  int rc = kUnsupportedShape;
  switch (p.dp / 32) {
    case 1: rc = launch_tokens_ni<T, 1>(p, st); break;
    case 2: rc = launch_tokens_ni<T, 2>(p, st); break;
    case 3: rc = launch_tokens_ni<T, 3>(p, st); break;
    case 4: rc = launch_tokens_ni<T, 4>(p, st); break;
    case 5: rc = launch_tokens_ni<T, 5>(p, st); break;
    case 6: rc = launch_tokens_ni<T, 6>(p, st); break;
    case 7: rc = launch_tokens_ni<T, 7>(p, st); break;
    case 8: rc = launch_tokens_ni<T, 8>(p, st); break;
    default: break;
  }
  if (rc != kOk) return rc;
  return launch_gated_norm<T>(p, st);
  }
}

static size_t up64(size_t n) { return (n + 63) / 64 * 64; }

}  // namespace mvb

// floats in front of o in the scratch of a ragged step: the chunk records, or q, k, g and beta
static size_t delta_operand_floats(int dtype, size_t t, size_t num_seqs, int heads, int kv_heads, int dim, int vdim) {
  using namespace mvb;
  if (dtype == kBf16) return up64((t / kChunk + num_seqs) * heads * (chunk_layout(chunk_ks(dim), vdim).total / 4));
  const size_t dp = delta_row_pad(dim);
  return 2 * up64(t * kv_heads * dp) + up64(t * heads * dp) + up64(t * heads);
}

extern "C" size_t mvb_gated_delta_scratch_bytes(int dtype, int num_tokens, int num_seqs, int heads, int kv_heads, int dim, int vdim,
                                                int ragged) {
  using namespace mvb;
  if (num_tokens <= 0 || num_seqs <= 0 || heads <= 0 || kv_heads <= 0 || dim <= 0 || dim > 256 || vdim <= 0) return 0;
  const size_t t = num_tokens, o = up64(t * heads * vdim);
  if (!ragged) return (vdim + 3) / 4 * 4 > 128 ? o * sizeof(float) : 64;
  return (delta_operand_floats(dtype, t, num_seqs, heads, kv_heads, dim, vdim) + o) * sizeof(float);
}

extern "C" int mvb_gated_delta(int dtype, const void* q, const void* k, const void* v, int64_t qkv_row_stride, const void* a,
                               int64_t a_row_stride, const void* b, int64_t b_row_stride, const void* gate,
                               int64_t gate_row_stride, const float* exp_a, const float* dt_bias, const float* norm_weight,
                               void* out, int64_t out_row_stride, float* state, const int32_t* state_slots, int64_t num_slots,
                               const int32_t* cu_seqlens_q, const int64_t* positions, int num_seqs, int num_tokens, int heads,
                               int kv_heads, int dim, int vdim, float q_scale, float eps, float out_scale, void* scratch,
                               size_t scratch_bytes, int32_t* dev_status, void* stream) {
  using namespace mvb;
  if (!q || !k || !v || !a || !b || !gate || !exp_a || !dt_bias || !norm_weight || !out || !positions) return kInvalidArgument;
  if (num_seqs < 0 || num_tokens < 0 || heads <= 0 || kv_heads <= 0 || heads % kv_heads != 0 || dim <= 0 || vdim <= 0) return kInvalidArgument;
  if (state != nullptr && (state_slots == nullptr || num_slots <= 0)) return kInvalidArgument;
  if (cu_seqlens_q == nullptr && num_seqs != num_tokens) return kInvalidArgument;
  if (dtype != kBf16 && dtype != kF32) return kInvalidArgument;
  if (!is_aligned(state, 16) || !is_aligned(scratch, 16)) return kMisaligned;
  if (dim > 256) return kUnsupportedShape;
  if (num_tokens == 0 || num_seqs == 0) return kOk;
  if (!scratch || scratch_bytes < mvb_gated_delta_scratch_bytes(dtype, num_tokens, num_seqs, heads, kv_heads, dim, vdim, cu_seqlens_q != nullptr))
    return kInvalidArgument;
  DeltaParams p;
  p.q = q; p.k = k; p.v = v; p.qkv_stride = qkv_row_stride;
  p.a = a; p.a_stride = a_row_stride; p.b = b; p.b_stride = b_row_stride; p.gate = gate; p.gate_stride = gate_row_stride;
  p.exp_a = exp_a; p.dt_bias = dt_bias; p.norm_w = norm_weight;
  p.out = out; p.out_stride = out_row_stride;
  p.state = state; p.slots = state_slots; p.num_slots = num_slots;
  p.cu = cu_seqlens_q; p.positions = positions;
  p.num_seqs = num_seqs; p.tokens = num_tokens; p.heads = heads; p.kv_heads = kv_heads; p.dim = dim; p.vdim = vdim;
  p.vp = (vdim + 3) / 4 * 4;
  p.q_scale = q_scale; p.eps = eps; p.out_scale = out_scale;
  p.dp = delta_row_pad(dim);
  p.dev_status = dev_status;
  float* f = static_cast<float*>(scratch);
  const size_t t = num_tokens;
  p.qn = p.kn = p.gn = p.beta = nullptr;
  if (cu_seqlens_q != nullptr && dtype == kBf16) {
    p.qn = f;                                                  // (the records)
    f += delta_operand_floats(dtype, t, num_seqs, heads, kv_heads, dim, vdim);
  } else if (cu_seqlens_q != nullptr) {
    p.qn = f; f += up64(t * kv_heads * p.dp);
    p.kn = f; f += up64(t * kv_heads * p.dp);
    p.gn = f; f += up64(t * heads * p.dp);
    p.beta = f; f += up64(t * heads);
  }
  p.o = f;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return dtype == kBf16 ? launch_delta<__nv_bfloat16>(p, st) : launch_delta<float>(p, st);
}
