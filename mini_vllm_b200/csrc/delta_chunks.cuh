// Gated delta rule over chunks of 16 tokens on the tensor cores (ragged steps with bf16 activations).
//
// With log-decays summed inside a chunk, G_t = sum_{s <= t} log g_s (per key channel), and the chunk's initial state S0:
//   e_t = beta_t (v_t - (k_t e^{G_t}) S0 - sum_{s < t} A_ts e_s)      A_ts = sum_d k_t k_s e^{G_t - G_s}
//   o_t = (q_t e^{G_t}) S0 + sum_{s <= t} B_ts e_s                    B_ts = sum_d q_t k_s e^{G_t - G_s}
//   S  <- e^{G_16} S0 + sum_s (k_s e^{G_16 - G_s}) e_s^T
// All exponents are <= 0, whatever the decays are.  e solves a unit lower-triangular system, so with T = (I + beta A)^-1 beta,
// U = T V and W = T (k e^G):  E = U - W S0.
//
// delta_chunk_prep (parallel over chunks and heads, fp32): unit norms, decays, A, B, T, W, U, and one contiguous record per
// (chunk, head) with everything the recurrence needs, already in the register order of mma.sync operands.
// delta_chunk_scan (sequential over the chunks of a sequence, parallel over heads and 16-column tiles): S^T stays in the fp32
// accumulator registers of one warp per 16 columns; records arrive by bulk copies, three chunks ahead.
// Accumulator fragments of S^T (and E^T) are operand fragments of the next product as they stand, so nothing is shuffled.
// Every fp32 operand enters as bf16 high + low part and every product as high*high + high*low + low*high: 16 significant bits
// per factor with fp32 accumulation; the state itself is never rounded below fp32.
#pragma once
#include "chunk_common.cuh"

namespace mvb {

struct ChunkLayout {              // bytes inside a record
  int ks, vtp, q, k, b, decay, u, total;
};
__host__ __device__ inline ChunkLayout chunk_layout(int ks, int vdim) {
  ChunkLayout l;
  l.ks = ks;
  l.vtp = ((vdim + 15) / 16 + 3) / 4 * 4;                    // 16-column tiles, a multiple of the four warps of a CTA
  l.q = ks * 1024; l.k = 2 * ks * 1024; l.b = 3 * ks * 1024; l.decay = l.b + 1024;
  l.u = l.decay + ks * 64;
  l.total = l.u + l.vtp * 1024;
  return l;
}

template <class T, int KS>
__global__ void __launch_bounds__(128, KS <= 8 ? 4 : 2) delta_chunk_prep(const DeltaParams p, uint8_t* records) {
  constexpr int DP = 16 * KS, D32 = (DP + 31) / 32 * 32, ROW = D32 + 4, NI = D32 / 32;
  extern __shared__ __align__(16) float sm[];
  float* q_s = sm;                               // [16][ROW]
  float* k_s = q_s + kChunk * ROW;
  float* g_s = k_s + kChunk * ROW;               // log2 of the decay, then its running sum
  float* u_s = g_s + kChunk * ROW;               // [columns of U][17]
  __shared__ float am[kChunk][kChunk + 1], bm[kChunk][kChunk + 1], beta_s[kChunk];
  __shared__ __align__(16) float tm[kChunk][kChunk];
  const int slot = blockIdx.x, h = blockIdx.y, kvh = h / (p.heads / p.kv_heads);
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  int lo = 0, hi = p.num_seqs;
  while (hi - lo > 1) {
    const int mid = (lo + hi) >> 1;
    if (chunk_base(p.cu[mid], mid) <= slot) lo = mid; else hi = mid;
  }
  const int begin = p.cu[lo], n_tok = p.cu[lo + 1] - begin, t0 = (slot - chunk_base(begin, lo)) * kChunk;
  if (t0 >= n_tok) return;
  const int nt = min(kChunk, n_tok - t0);
  const ChunkLayout lay = chunk_layout(KS, p.vdim);
  uint8_t* rec = records + (static_cast<int64_t>(slot) * p.heads + h) * lay.total;

  // a warp takes every fourth token; the raw operands of U tokens are requested before any is worked on
  constexpr int U = NI <= 4 ? 4 : 2;
  const float ea = -p.exp_a[h] * 1.4426950408889634f;
  float bias[NI];
#pragma unroll
  for (int i = 0; i < NI; ++i) bias[i] = i * 32 + lane < p.dim ? p.dt_bias[h * p.dim + i * 32 + lane] : 0.f;
  const float raw_b = tid < nt ? to_f(static_cast<const T*>(p.b)[(begin + t0 + tid) * p.b_stride + h]) : 0.f;
  for (int v = tid; v < lay.vtp * 16; v += 128) {              // v waits in the columns that U will take
    T vv[kChunk];
#pragma unroll
    for (int s = 0; s < kChunk; ++s)
      vv[s] = v < p.vdim && s < nt ? static_cast<const T*>(p.v)[(begin + t0 + s) * p.qkv_stride + h * p.vdim + v] : from_f<T>(0.f);
#pragma unroll
    for (int s = 0; s < kChunk; ++s) u_s[v * 17 + s] = to_f(vv[s]);
  }
#pragma unroll 1
  for (int tb = warp; tb < kChunk; tb += 4 * U) {
    T rq[U][NI], rk[U][NI], ra[U][NI];
#pragma unroll
    for (int m = 0; m < U; ++m) {
      const int t = tb + 4 * m;
      const int64_t row = begin + t0 + t;
      const T* qr = static_cast<const T*>(p.q) + row * p.qkv_stride + kvh * p.dim;
      const T* kr = static_cast<const T*>(p.k) + row * p.qkv_stride + kvh * p.dim;
      const T* ar = static_cast<const T*>(p.a) + row * p.a_stride + h * p.dim;
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        const int d = i * 32 + lane;
        const bool in = t < nt && d < p.dim;
        rq[m][i] = in ? qr[d] : from_f<T>(0.f);
        rk[m][i] = in ? kr[d] : from_f<T>(0.f);
        ra[m][i] = in ? ar[d] : from_f<T>(0.f);
      }
    }
#pragma unroll
    for (int m = 0; m < U; ++m) {
      const int t = tb + 4 * m;
      float qq = 0.f, kk = 0.f;
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        const int d = i * 32 + lane;
        const bool in = t < nt && d < p.dim;
        g_s[t * ROW + d] = in ? ea * softplus_of<T>(to_f(ra[m][i]) + bias[i]) : 0.f;
        const float q = to_f(rq[m][i]), k = to_f(rk[m][i]);
        qq += q * q; kk += k * k;
      }
      qq = warp_sum(qq); kk = warp_sum(kk);
      const float nq = p.q_scale / sqrtf(qq + kUnitEps), nk = 1.f / sqrtf(kk + kUnitEps);
#pragma unroll
      for (int i = 0; i < NI; ++i) {
        q_s[t * ROW + i * 32 + lane] = to_f(rq[m][i]) * nq;
        k_s[t * ROW + i * 32 + lane] = to_f(rk[m][i]) * nk;
      }
    }
  }
  if (tid < kChunk) beta_s[tid] = tid < nt ? sigmoid_f(raw_b) : 0.f;
  __syncthreads();
  for (int d = tid; d < D32; d += 128) {
    float run = 0.f;
#pragma unroll
    for (int t = 0; t < kChunk; ++t) { run += g_s[t * ROW + d]; g_s[t * ROW + d] = run; }
  }
  __syncthreads();
  // A and B below and on the diagonal: a warp takes every fourth row
  for (int t = warp; t < kChunk; t += 4) {
    float q[NI], k[NI], g[NI];
#pragma unroll
    for (int i = 0; i < NI; ++i) { const int x = t * ROW + i * 32 + lane; q[i] = q_s[x]; k[i] = k_s[x]; g[i] = g_s[x]; }
    // four columns at a time (those past the diagonal are not stored): eight sums over the warp.  Halving exchanges leave
    // lane groups of four with one sum each - 4 + 2 + 1 exchanges instead of five per sum - and two more finish it.
#pragma unroll 1
    for (int s0 = 0; s0 <= t; s0 += 4) {
      float v[8];
#pragma unroll
      for (int m = 0; m < 4; ++m) {
        float a = 0.f, b = 0.f;
#pragma unroll
        for (int i = 0; i < NI; ++i) {
          const int x = (s0 + m) * ROW + i * 32 + lane;
          const float w = k_s[x] * fast_exp2(fminf(g[i] - g_s[x], 0.f));
          a = fmaf(k[i], w, a); b = fmaf(q[i], w, b);
        }
        v[m] = a; v[4 + m] = b;
      }
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
      const int sc = s0 + (up8 ? 2 : 0) + (up4 ? 1 : 0);
      if ((lane & 3) == 0 && sc <= t) (up16 ? bm : am)[t][sc] = v[0];
    }
  }
  __syncthreads();
  if (warp == 0) {                               // column `lane` of T by forward substitution
    float x[kChunk];
#pragma unroll
    for (int t = 0; t < kChunk; ++t) {
      float acc = t == lane ? 1.f : 0.f;
#pragma unroll
      for (int s = 0; s < t; ++s) acc = fmaf(-am[t][s], x[s], acc);
      x[t] = beta_s[t] * acc;
      if (lane < kChunk) tm[t][lane] = x[t];
    }
  } else if (warp == 1) {                        // B as the second operand of O^T += E^T B^T
    uint4* dst = reinterpret_cast<uint4*>(rec + lay.b);
#pragma unroll
    for (int n = 0; n < 2; ++n) {
      const int t = n * 8 + (lane >> 2), s = (lane & 3) * 2;
      auto at = [&](int c) { return c <= t ? bm[t][c] : 0.f; };
      uint4 w;
      split_pair(at(s), at(s + 1), w.x, w.z);
      split_pair(at(s + 8), at(s + 9), w.y, w.w);
      dst[n * 32 + lane] = w;
    }
  }
  __syncthreads();
  // a thread owns a key channel: its columns of q, k, g turn into those of Q = q e^G, K = k e^{G_16 - G} and W in place
  for (int d = tid; d < D32; d += 128) {
    float kh[kChunk];
    const float g_end = g_s[(kChunk - 1) * ROW + d];
#pragma unroll
    for (int t = 0; t < kChunk; ++t) {
      const float g = g_s[t * ROW + d], eg = fast_exp2(g), k = k_s[t * ROW + d];
      kh[t] = k * eg;
      q_s[t * ROW + d] *= eg;
      k_s[t * ROW + d] = k * fast_exp2(g_end - g);
    }
#pragma unroll
    for (int t = 0; t < kChunk; ++t) {
      float acc = 0.f;
#pragma unroll
      for (int s = 0; s <= t; ++s) acc = fmaf(tm[t][s], kh[s], acc);
      g_s[t * ROW + d] = acc;
    }
    if (d < DP) reinterpret_cast<float*>(rec + lay.decay)[d] = fast_exp2(g_end);
  }
  for (int v = tid; v < lay.vtp * 16; v += 128) {
    float vv[kChunk];
#pragma unroll
    for (int s = 0; s < kChunk; ++s) vv[s] = u_s[v * 17 + s];
#pragma unroll
    for (int t = 0; t < kChunk; ++t) {
      float u = 0.f;
#pragma unroll
      for (int s = 0; s <= t; ++s) u = fmaf(tm[t][s], vv[s], u);
      u_s[v * 17 + t] = u;
    }
  }
  __syncthreads();
  // the record, 16 bytes at a time in the order in which lanes will read it
  for (int i = tid; i < 2 * KS * 64; i += 128) {
    const int w = i < KS * 64 ? i : i - KS * 64, ln = w & 31, n = (w >> 5) & 1, ks = w >> 6;
    const float* src = (i < KS * 64 ? g_s : q_s) + (n * 8 + (ln >> 2)) * ROW + ks * 16 + (ln & 3) * 2;
    const float2 x = *reinterpret_cast<const float2*>(src), y = *reinterpret_cast<const float2*>(src + 8);
    uint4 o;
    split_pair(x.x, x.y, o.x, o.z);
    split_pair(y.x, y.y, o.y, o.w);
    reinterpret_cast<uint4*>(rec)[i] = o;
  }
  for (int i = tid; i < KS * 64; i += 128) {
    const int ln = i & 31, d = (i >> 5) * 8 + (ln >> 2), t = (ln & 3) * 2;
    uint4 o;
    split_pair(k_s[t * ROW + d], k_s[(t + 1) * ROW + d], o.x, o.z);
    split_pair(k_s[(t + 8) * ROW + d], k_s[(t + 9) * ROW + d], o.y, o.w);
    reinterpret_cast<uint4*>(rec + lay.k)[i] = o;
  }
  for (int i = tid; i < lay.vtp * 64; i += 128) {
    const int ln = i & 31, t = ((i >> 5) & 1) * 8 + (ln & 3) * 2, v = (i >> 6) * 16 + (ln >> 2);
    reinterpret_cast<float4*>(rec + lay.u)[i] =
        make_float4(u_s[v * 17 + t], u_s[v * 17 + t + 1], u_s[(v + 8) * 17 + t], u_s[(v + 8) * 17 + t + 1]);
  }
}

template <int KS, int WARPS>
struct ChunkScanCfg {
  static constexpr int STAGES = 3;
  static constexpr int SHARED = KS * 3136 + 1024, STAGE = SHARED + WARPS * 1024;     // common part + a U tile per warp
  static constexpr int SMEM = STAGES * STAGE + 64;
};

template <int KS, int WARPS>
__global__ void __launch_bounds__(WARPS * 32) delta_chunk_scan(const DeltaParams p, const uint8_t* __restrict__ records) {
  using C = ChunkScanCfg<KS, WARPS>;
  extern __shared__ __align__(128) uint8_t smem[];
  uint64_t* full = reinterpret_cast<uint64_t*>(smem + C::STAGES * C::STAGE);
  const int s = blockIdx.z, h = blockIdx.y, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
  const int begin = p.cu[s], n_tok = p.cu[s + 1] - begin;
  if (n_tok <= 0) return;
  const int n_chunks = (n_tok + kChunk - 1) / kChunk, vt = blockIdx.x * WARPS + warp;
  const ChunkLayout lay = chunk_layout(KS, p.vdim);
  const uint8_t* rec = records + (static_cast<int64_t>(chunk_base(begin, s)) * p.heads + h) * lay.total;
  const int64_t rec_step = static_cast<int64_t>(p.heads) * lay.total;
  if (tid == 0) {
    for (int i = 0; i < C::STAGES; ++i) mbar_init(&full[i], 1);
    fence_mbar_init();
  }
  __syncthreads();
  auto fetch = [&](int c) {                       // one thread
    const int st = c % C::STAGES;
    const uint8_t* src = rec + c * rec_step;
    const uint32_t dst = smem_u32(smem + st * C::STAGE), bar = smem_u32(&full[st]);
    mbar_arrive_expect_tx(&full[st], C::STAGE);
    bulk_copy(dst, src, C::SHARED, bar);
    bulk_copy(dst + C::SHARED, src + lay.u + blockIdx.x * (WARPS * 1024), WARPS * 1024, bar);
  };
  if (tid == 0)
    for (int c = 0; c < min(C::STAGES, n_chunks); ++c) fetch(c);

  const int64_t slot = delta_slot(p, s);
  const bool fresh = slot < 0 || p.positions[begin] == 0;
  const int v0 = vt * 16 + (lane >> 2), dq = (lane & 3) * 2;
  float S[2 * KS][4];                             // S^T: rows v0, v0 + 8; columns 8 j + dq, + 1
  auto state_at = [&](int j, int i) { return p.state + ((slot * p.heads + h) * p.dim + 8 * j + dq + (i & 1)) * static_cast<int64_t>(p.vp) + v0 + (i & 2) * 4; };
  auto in_state = [&](int j, int i) { return 8 * j + dq + (i & 1) < p.dim && v0 + (i & 2) * 4 < p.vdim; };
#pragma unroll
  for (int j = 0; j < 2 * KS; ++j)
#pragma unroll
    for (int i = 0; i < 4; ++i) S[j][i] = !fresh && in_state(j, i) ? *state_at(j, i) : 0.f;

  bool ok = true;
  int c = 0;
  for (; c < n_chunks; ++c) {
    const int st = c % C::STAGES;
    ok = mbar_wait(&full[st], (c / C::STAGES) & 1);
    if (!__syncthreads_and(ok)) break;            // (uniform: every thread leaves together)
    const uint8_t* base = smem + st * C::STAGE;
    const uint4* w_r = reinterpret_cast<const uint4*>(base);
    const uint4* q_r = reinterpret_cast<const uint4*>(base + KS * 1024);
    const uint4* k_r = reinterpret_cast<const uint4*>(base + 2 * KS * 1024);
    const uint4* b_r = reinterpret_cast<const uint4*>(base + 3 * KS * 1024);
    const float* decay = reinterpret_cast<const float*>(base + 3 * KS * 1024 + 1024);
    const float4* u_r = reinterpret_cast<const float4*>(base + C::SHARED) + warp * 64;
    float wa[2][4], wb[2][4], oa[2][4], ob[2][4];
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int i = 0; i < 4; ++i) wa[n][i] = wb[n][i] = oa[n][i] = ob[n][i] = 0.f;
#pragma unroll
    for (int ks = 0; ks < KS; ++ks) {             // W S0 and Q S0
      Split a;
      split_tile(S[2 * ks], S[2 * ks + 1], a);
      const uint4 w0 = w_r[(ks * 2) * 32 + lane], w1 = w_r[(ks * 2 + 1) * 32 + lane];
      const uint4 q0 = q_r[(ks * 2) * 32 + lane], q1 = q_r[(ks * 2 + 1) * 32 + lane];
      mma_bf16_16816(wa[0], a.hi, w0.x, w0.y); mma_bf16_16816(wa[1], a.hi, w1.x, w1.y);
      mma_bf16_16816(oa[0], a.hi, q0.x, q0.y); mma_bf16_16816(oa[1], a.hi, q1.x, q1.y);
      mma_bf16_16816(wb[0], a.hi, w0.z, w0.w); mma_bf16_16816(wb[1], a.hi, w1.z, w1.w);
      mma_bf16_16816(ob[0], a.hi, q0.z, q0.w); mma_bf16_16816(ob[1], a.hi, q1.z, q1.w);
      mma_bf16_16816(wb[0], a.lo, w0.x, w0.y); mma_bf16_16816(wb[1], a.lo, w1.x, w1.y);
      mma_bf16_16816(ob[0], a.lo, q0.x, q0.y); mma_bf16_16816(ob[1], a.lo, q1.x, q1.y);
    }
    float e[2][4];
#pragma unroll
    for (int n = 0; n < 2; ++n) {
      const float4 u = u_r[n * 32 + lane];
      e[n][0] = u.x - (wa[n][0] + wb[n][0]); e[n][1] = u.y - (wa[n][1] + wb[n][1]);
      e[n][2] = u.z - (wa[n][2] + wb[n][2]); e[n][3] = u.w - (wa[n][3] + wb[n][3]);
    }
    Split x;
    split_tile(e[0], e[1], x);
#pragma unroll
    for (int j = 0; j < 2 * KS; ++j) {            // S^T <- S^T decay + E^T K
      const float2 g = *reinterpret_cast<const float2*>(decay + 8 * j + dq);
      const uint4 k = k_r[j * 32 + lane];
      S[j][0] *= g.x; S[j][1] *= g.y; S[j][2] *= g.x; S[j][3] *= g.y;
      mma_bf16_16816(S[j], x.hi, k.x, k.y);
      mma_bf16_16816(S[j], x.hi, k.z, k.w);
      mma_bf16_16816(S[j], x.lo, k.x, k.y);
    }
#pragma unroll
    for (int n = 0; n < 2; ++n) {                 // O += E^T B^T
      const uint4 b = b_r[n * 32 + lane];
      mma_bf16_16816(oa[n], x.hi, b.x, b.y);
      mma_bf16_16816(ob[n], x.hi, b.z, b.w);
      mma_bf16_16816(ob[n], x.lo, b.x, b.y);
    }
    __syncthreads();                              // the stage has been read
    if (tid == 0 && c + C::STAGES < n_chunks) { fence_proxy_async(); fetch(c + C::STAGES); }
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const int t = c * kChunk + n * 8 + dq + (i & 1), v = v0 + (i & 2) * 4;
        if (t < n_tok && v < p.vdim) p.o[(static_cast<int64_t>(begin + t) * p.heads + h) * p.vdim + v] = oa[n][i] + ob[n][i];
      }
  }
  if (c < n_chunks) {                             // a copy did not arrive in time: report it, let those in flight land, keep the old state
    if (!ok) report(p.dev_status, kDevWaitTimeout, c);
    for (int k = c; k < min(c + C::STAGES, n_chunks); ++k) mbar_wait(&full[k % C::STAGES], (k / C::STAGES) & 1, 1u << 16);
    return;
  }
  if (slot >= 0) {
#pragma unroll
    for (int j = 0; j < 2 * KS; ++j)
#pragma unroll
      for (int i = 0; i < 4; ++i)
        if (in_state(j, i)) *state_at(j, i) = S[j][i];
  }
}

template <class T, int KS>
static int launch_delta_chunks(const DeltaParams& p, uint8_t* records, cudaStream_t st) {
  constexpr int D32 = (16 * KS + 31) / 32 * 32;
  const ChunkLayout lay = chunk_layout(KS, p.vdim);
  const size_t prep_smem = (3 * kChunk * (D32 + 4) + lay.vtp * 16 * 17) * sizeof(float);
  if (prep_smem > 200 * 1024) return kUnsupportedShape;
  struct PrepTag {};
  int rc = opt_in_dynamic_smem<PrepTag>(reinterpret_cast<const void*>(&delta_chunk_prep<T, KS>), prep_smem);
  if (rc != kOk) return rc;
  const int slots = p.tokens / kChunk + p.num_seqs;
  delta_chunk_prep<T, KS><<<dim3(slots, p.heads), 128, prep_smem, st>>>(p, records);
  if (cudaGetLastError() != cudaSuccess) return kLaunchFailed;
  auto scan = [&](auto tag) -> int {
    constexpr int WARPS = decltype(tag)::value;
    struct ScanTag {};
    const int r = opt_in_dynamic_smem<ScanTag>(reinterpret_cast<const void*>(&delta_chunk_scan<KS, WARPS>), ChunkScanCfg<KS, WARPS>::SMEM);
    if (r != kOk) return r;
    const int tiles = (p.vdim + 15) / 16;
    delta_chunk_scan<KS, WARPS><<<dim3((tiles + WARPS - 1) / WARPS, p.heads, p.num_seqs), WARPS * 32, ChunkScanCfg<KS, WARPS>::SMEM, st>>>(p, records);
    return cudaGetLastError() == cudaSuccess ? kOk : kLaunchFailed;
  };
  // few (sequence, head) pairs: one warp per CTA, so that they spread over the SMs
  const bool few = static_cast<int64_t>(lay.vtp) * p.heads * p.num_seqs <= sm_count() * 2;
  return few ? scan(std::integral_constant<int, 1>{}) : scan(std::integral_constant<int, 4>{});
}

}  // namespace mvb
