// Selective state-space scan (input-dependent diagonal recurrence) on a packed ragged batch, state carried per sequence.
//
//   S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c u_c B_n        dt_c = softplus(raw_c + bias_c)
//   out_c   = (sum_n S[c, n] C_n + D_c u_c) * silu(z_c)
//
// Everything between the projections and the output is fp32; the state lives in fp32 slots [slots, channels, N'] (N' =
// N rounded up to 4).  A lane owns 4 R consecutive states of one channel, L lanes a channel; the sum over n is a shuffle
// reduction.  exp(dt A) is one ex2 with A pre-multiplied by log2(e).
//
// Ragged step (scan_tokens_kernel): a CTA of 4 warps walks the tokens of one sequence for 128 / L channels, TT tokens at a
// time: raw operands of the next tile are requested into registers before the current tile is worked on, dt and dt*u
// are computed once per (token, channel) into shared memory.
// One token per sequence (scan_step_kernel): bound by reading and writing the state; no shared memory.
//
// Roofline: a ragged step is bound by the special-function unit (channels * N exponentials per token, 16 per clock and SM)
// or, for few states, by HBM (4 activations of channels elements per token); a decode step by HBM (2 * 4 * channels * N bytes
// per sequence).
#include "dtype.cuh"
#include "host_util.cuh"
#include "mini_vllm_b200.h"

namespace mvb {

struct ScanParams {
  const void* u; int64_t u_stride;
  const void* dt; int64_t dt_stride;       // raw, before bias and softplus
  const void* z; int64_t z_stride;
  const void* b; const void* c; int64_t bc_stride;
  const float* dt_bias;                    // [channels]
  const float* a_log2e;                    // [channels, np] = A log2(e), zero in the padding
  const float* d;                          // [channels]
  void* out; int64_t out_stride;
  float* state;                            // [slots, channels, np] or nullptr
  const int32_t* slots; int64_t num_slots;
  const int32_t* cu; const int64_t* positions;
  int num_seqs, tokens, channels, n, np;
  bool bc_vec;                             // four consecutive elements of b or c may be read as one vector
  int* dev_status;
};

__device__ __forceinline__ int64_t scan_slot(const ScanParams& p, int s) {
  if (p.state == nullptr) return -1;
  const int64_t slot = p.slots[s];
  if (slot >= p.num_slots) { report(p.dev_status, kDevBadSlot, s); return -1; }
  return slot;
}
__device__ __forceinline__ float silu_f(float z) { return z * fast_rcp(1.f + fast_exp2(z * -1.4426950408889634f)); }

// S 2^x + in.  A decay close to 1 acts over thousands of tokens, where the couple of ulps of the hardware exponential would
// add up to more than an fp32 model's own rounding: there the decrement is computed instead of the factor.
template <class T>
__device__ __forceinline__ float advance(float S, float x, float in) {
  if constexpr (sizeof(T) == 4) return fmaf(S, expm1f(x * 0.6931471805599453f), S) + in;
  else return fmaf(fast_exp2(x), S, in);
}

// four values at p[0..n), zeros past n; vec: p is aligned for one vector access
template <class T>
__device__ __forceinline__ void load4(const T* p, int n, bool vec, float (&v)[4]) {
  if (vec && n >= 4) {
    if constexpr (sizeof(T) == 2) {
      const uint2 w = *reinterpret_cast<const uint2*>(p);
      v[0] = bf16_lo(w.x); v[1] = bf16_hi(w.x); v[2] = bf16_lo(w.y); v[3] = bf16_hi(w.y);
    } else {
      const float4 w = *reinterpret_cast<const float4*>(p);
      v[0] = w.x; v[1] = w.y; v[2] = w.z; v[3] = w.w;
    }
  } else {
#pragma unroll
    for (int j = 0; j < 4; ++j) v[j] = j < n ? to_f(p[j]) : 0.f;
  }
}

// E neighbouring elements as they lie in memory
template <class T, int E> struct Raw { T v[E]; };
template <class T, int E> __device__ __forceinline__ Raw<T, E> load_raw(const T* p, bool ok) {
  Raw<T, E> r;
  if constexpr (E == 1) {
    r.v[0] = ok ? *p : from_f<T>(0.f);
  } else if constexpr (sizeof(T) == 2) {
    const uint32_t w = ok ? *reinterpret_cast<const uint32_t*>(p) : 0u;
    *reinterpret_cast<uint32_t*>(r.v) = w;
  } else {
    const float2 w = ok ? *reinterpret_cast<const float2*>(p) : make_float2(0.f, 0.f);
    r.v[0] = w.x; r.v[1] = w.y;
  }
  return r;
}

// E: channels per thread in the elementwise part (2 where the operands are aligned for it)
template <class T, int L, int R, int E>
__global__ void __launch_bounds__(128) scan_tokens_kernel(const ScanParams p) {
  constexpr int CHW = 32 / L, CH = 4 * CHW, NP = 4 * L * R, TT = L <= 8 ? 32 : 16;
  constexpr int ECH = CH / E, EPT = TT * ECH >= 128 ? TT * ECH / 128 : 1, BPT = TT * 2 * NP / 128;
  __shared__ __align__(8) float dt_s[TT][CH];
  __shared__ __align__(8) float du_s[TT][CH];
  __shared__ __align__(8) float y_s[TT][CH];
  __shared__ __align__(16) float b_s[TT][NP];
  __shared__ __align__(16) float c_s[TT][NP];
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, sub = lane % L;
  const int chl = warp * CHW + lane / L, c0 = blockIdx.y * CH, c = c0 + chl, s = blockIdx.x;
  const int begin = p.cu[s], n_tok = p.cu[s + 1] - begin;
  if (n_tok <= 0) return;
  const int64_t slot = scan_slot(p, s);
  const bool fresh = p.positions[begin] == 0 || slot < 0;

  float a[R][4], S[R][4];
#pragma unroll
  for (int r = 0; r < R; ++r) {
    const int n0 = (sub + L * r) * 4;
    float4 av = make_float4(0.f, 0.f, 0.f, 0.f), sv = av;
    if (c < p.channels && n0 < p.np) {
      av = *reinterpret_cast<const float4*>(p.a_log2e + static_cast<int64_t>(c) * p.np + n0);
      if (!fresh) sv = *reinterpret_cast<const float4*>(p.state + (slot * p.channels + c) * p.np + n0);
    }
    a[r][0] = av.x; a[r][1] = av.y; a[r][2] = av.z; a[r][3] = av.w;
    S[r][0] = sv.x; S[r][1] = sv.y; S[r][2] = sv.z; S[r][3] = sv.w;
  }

  // a thread keeps its E channels throughout and takes every ESTEP-th token of a tile
  constexpr int ESTEP = 128 / ECH;
  const int ech = tid % ECH * E, etok = tid / ECH;
  const bool ech_ok = c0 + ech < p.channels;
  float bias[E], dskip[E];
#pragma unroll
  for (int j = 0; j < E; ++j) {
    bias[j] = ech_ok ? p.dt_bias[c0 + ech + j] : 0.f;
    dskip[j] = ech_ok ? p.d[c0 + ech + j] : 0.f;
  }
  const int64_t first = begin + etok;
  const T* pu = static_cast<const T*>(p.u) + first * p.u_stride + c0 + ech;
  const T* pd = static_cast<const T*>(p.dt) + first * p.dt_stride + c0 + ech;
  const T* pz = static_cast<const T*>(p.z) + first * p.z_stride + c0 + ech;
  T* po = static_cast<T*>(p.out) + first * p.out_stride + c0 + ech;
  Raw<T, E> ru[EPT], rdt[EPT], rz[EPT];
  T rbc[BPT];
  auto request = [&](int t0) {
#pragma unroll
    for (int k = 0; k < EPT; ++k) {
      const int tl = etok + k * ESTEP;
      const bool ok = ech_ok && tl < TT && t0 + tl < n_tok;
      ru[k] = load_raw<T, E>(pu + k * ESTEP * p.u_stride, ok);
      rdt[k] = load_raw<T, E>(pd + k * ESTEP * p.dt_stride, ok);
      rz[k] = load_raw<T, E>(pz + k * ESTEP * p.z_stride, ok);
    }
    pu += TT * p.u_stride; pd += TT * p.dt_stride; pz += TT * p.z_stride;
#pragma unroll
    for (int k = 0; k < BPT; ++k) {
      const int e = tid + k * 128, t = t0 + e / (2 * NP), j = e % (2 * NP), nn = j % NP;
      const T* src = static_cast<const T*>(j < NP ? p.b : p.c);
      rbc[k] = t < n_tok && nn < p.n ? src[(begin + t) * p.bc_stride + nn] : from_f<T>(0.f);
    }
  };
  request(0);
  for (int t0 = 0; t0 < n_tok; t0 += TT) {
    Raw<T, E> cu_[EPT], cz[EPT];
#pragma unroll
    for (int k = 0; k < EPT; ++k) {
      const int tl = etok + k * ESTEP;
      cu_[k] = ru[k]; cz[k] = rz[k];
      if (TT * ECH < 128 && tl >= TT) continue;
      const bool in = t0 + tl < n_tok;                       // (a token past the end changes nothing)
      float dt[E], du[E];
#pragma unroll
      for (int j = 0; j < E; ++j) {
        dt[j] = in ? softplus_of<T>(to_f(rdt[k].v[j]) + bias[j]) : 0.f;
        du[j] = dt[j] * to_f(ru[k].v[j]);
      }
      if constexpr (E == 2) {
        *reinterpret_cast<float2*>(&dt_s[tl][ech]) = make_float2(dt[0], dt[1]);
        *reinterpret_cast<float2*>(&du_s[tl][ech]) = make_float2(du[0], du[1]);
      } else {
        dt_s[tl][ech] = dt[0];
        du_s[tl][ech] = du[0];
      }
    }
#pragma unroll
    for (int k = 0; k < BPT; ++k) {
      const int e = tid + k * 128, tl = e / (2 * NP), j = e % (2 * NP);
      if (j < NP) b_s[tl][j] = to_f(rbc[k]); else c_s[tl][j - NP] = to_f(rbc[k]);
    }
    __syncthreads();
    if (t0 + TT < n_tok) request(t0 + TT);
    const int nt = min(TT, n_tok - t0);
    // four tokens at a time: all operands and exponentials first, so that only the multiply-adds of S are a chain
    for (int tb = 0; tb < nt; tb += 4) {
      float dt[4], du[4], acc[4];
#pragma unroll
      for (int m = 0; m < 4; ++m) { dt[m] = dt_s[tb + m][chl]; du[m] = du_s[tb + m][chl]; acc[m] = 0.f; }
#pragma unroll
      for (int r = 0; r < R; ++r) {
        const int n0 = (sub + L * r) * 4;
        float4 bv[4], cv[4];
#pragma unroll
        for (int m = 0; m < 4; ++m) {
          bv[m] = *reinterpret_cast<const float4*>(&b_s[tb + m][n0]);
          cv[m] = *reinterpret_cast<const float4*>(&c_s[tb + m][n0]);
        }
#pragma unroll
        for (int m = 0; m < 4; ++m) {
          S[r][0] = advance<T>(S[r][0], dt[m] * a[r][0], du[m] * bv[m].x); acc[m] = fmaf(S[r][0], cv[m].x, acc[m]);
          S[r][1] = advance<T>(S[r][1], dt[m] * a[r][1], du[m] * bv[m].y); acc[m] = fmaf(S[r][1], cv[m].y, acc[m]);
          S[r][2] = advance<T>(S[r][2], dt[m] * a[r][2], du[m] * bv[m].z); acc[m] = fmaf(S[r][2], cv[m].z, acc[m]);
          S[r][3] = advance<T>(S[r][3], dt[m] * a[r][3], du[m] * bv[m].w); acc[m] = fmaf(S[r][3], cv[m].w, acc[m]);
        }
      }
#pragma unroll
      for (int off = 1; off < L; off <<= 1)
#pragma unroll
        for (int m = 0; m < 4; ++m) acc[m] += __shfl_xor_sync(0xffffffffu, acc[m], off);
      if (sub == 0) {
#pragma unroll
        for (int m = 0; m < 4; ++m) y_s[tb + m][chl] = acc[m];
      }
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < EPT; ++k) {
      const int tl = etok + k * ESTEP;
      if (!ech_ok || tl >= nt) continue;
      float y[E];
#pragma unroll
      for (int j = 0; j < E; ++j) y[j] = fmaf(dskip[j], to_f(cu_[k].v[j]), y_s[tl][ech + j]) * silu_f(to_f(cz[k].v[j]));
      T* dst = po + k * ESTEP * p.out_stride;
      if constexpr (E == 1) *dst = from_f<T>(y[0]);
      else if constexpr (sizeof(T) == 2) *reinterpret_cast<uint32_t*>(dst) = pack_bf16(y[0], y[1]);
      else *reinterpret_cast<float2*>(dst) = make_float2(y[0], y[1]);
    }
    po += TT * p.out_stride;
  }
  if (slot >= 0 && c < p.channels) {
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const int n0 = (sub + L * r) * 4;
      if (n0 < p.np)
        *reinterpret_cast<float4*>(p.state + (slot * p.channels + c) * p.np + n0) = make_float4(S[r][0], S[r][1], S[r][2], S[r][3]);
    }
  }
}

template <class T, int L, int R>
__global__ void __launch_bounds__(256) scan_step_kernel(const ScanParams p) {
  const int s = blockIdx.y, i = blockIdx.x * 256 + threadIdx.x, c = i / L, sub = i % L;
  const int64_t slot = scan_slot(p, s);
  const bool fresh = slot < 0 || p.positions[s] == 0, ok = c < p.channels;
  float acc = 0.f, u = 0.f;
  if (ok) {
    float4 sv[R];
#pragma unroll
    for (int r = 0; r < R; ++r) {                            // what the kernel waits for goes out first
      const int n0 = (sub + L * r) * 4;
      sv[r] = make_float4(0.f, 0.f, 0.f, 0.f);
      if (!fresh && n0 < p.np) sv[r] = *reinterpret_cast<const float4*>(p.state + (slot * p.channels + c) * p.np + n0);
    }
    u = to_f(static_cast<const T*>(p.u)[s * p.u_stride + c]);
    const float dt = softplus_of<T>(to_f(static_cast<const T*>(p.dt)[s * p.dt_stride + c]) + p.dt_bias[c]), du = dt * u;
#pragma unroll
    for (int r = 0; r < R; ++r) {
      const int n0 = (sub + L * r) * 4;
      if (n0 >= p.np) continue;
      const float4 av = *reinterpret_cast<const float4*>(p.a_log2e + static_cast<int64_t>(c) * p.np + n0);
      const float a[4] = {av.x, av.y, av.z, av.w};
      float S[4] = {sv[r].x, sv[r].y, sv[r].z, sv[r].w}, bn[4], cn[4];
      load4(static_cast<const T*>(p.b) + s * p.bc_stride + n0, p.n - n0, p.bc_vec, bn);
      load4(static_cast<const T*>(p.c) + s * p.bc_stride + n0, p.n - n0, p.bc_vec, cn);
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        S[j] = advance<T>(S[j], dt * a[j], du * bn[j]);
        acc = fmaf(S[j], cn[j], acc);
      }
      if (slot >= 0) *reinterpret_cast<float4*>(p.state + (slot * p.channels + c) * p.np + n0) = make_float4(S[0], S[1], S[2], S[3]);
    }
  }
#pragma unroll
  for (int off = 1; off < L; off <<= 1) acc += __shfl_xor_sync(0xffffffffu, acc, off);
  if (ok && sub == 0) {
    const float z = to_f(static_cast<const T*>(p.z)[s * p.z_stride + c]);
    static_cast<T*>(p.out)[s * p.out_stride + c] = from_f<T>(fmaf(p.d[c], u, acc) * silu_f(z));
  }
}

template <class T, int L, int R>
static int launch_scan_lr(const ScanParams& p, cudaStream_t st) {
  if (p.cu == nullptr) {
    const int64_t threads = static_cast<int64_t>(p.channels) * L;
    if (p.num_seqs > 65535) return kUnsupportedShape;
    scan_step_kernel<T, L, R><<<dim3(static_cast<unsigned>((threads + 255) / 256), p.num_seqs), 256, 0, st>>>(p);
  } else {
    constexpr int CH = 4 * (32 / L);
    const int gy = (p.channels + CH - 1) / CH;
    if (gy > 65535) return kUnsupportedShape;
    constexpr uintptr_t A = 2 * sizeof(T);
    const bool pairs = p.channels % 2 == 0 && p.u_stride % 2 == 0 && p.dt_stride % 2 == 0 && p.z_stride % 2 == 0 && p.out_stride % 2 == 0 &&
                       is_aligned(p.u, A) && is_aligned(p.dt, A) && is_aligned(p.z, A) && is_aligned(p.out, A);
    if (pairs) scan_tokens_kernel<T, L, R, 2><<<dim3(p.num_seqs, gy), 128, 0, st>>>(p);
    else scan_tokens_kernel<T, L, R, 1><<<dim3(p.num_seqs, gy), 128, 0, st>>>(p);
  }
  return cudaGetLastError() == cudaSuccess ? kOk : kLaunchFailed;
}

template <class T>
static int launch_scan(const ScanParams& p, cudaStream_t st) {
  if (p.np <= 16) return launch_scan_lr<T, 4, 1>(p, st);
  if (p.np <= 32) return launch_scan_lr<T, 8, 1>(p, st);
  if (p.np <= 64) return launch_scan_lr<T, 16, 1>(p, st);
  if (p.np <= 128) return launch_scan_lr<T, 32, 1>(p, st);
  if (p.np <= 256) return launch_scan_lr<T, 32, 2>(p, st);
  return kUnsupportedShape;
}

}  // namespace mvb

extern "C" int mvb_selective_scan(int dtype, const void* u, int64_t u_row_stride, const void* dt, int64_t dt_row_stride,
                                  const void* z, int64_t z_row_stride, const void* b, const void* c, int64_t bc_row_stride,
                                  const float* dt_bias, const float* a_log2e, const float* d, void* out,
                                  int64_t out_row_stride, float* state, const int32_t* state_slots, int64_t num_slots,
                                  const int32_t* cu_seqlens_q, const int64_t* positions, int num_seqs, int num_tokens,
                                  int channels, int num_states, int state_stride, int32_t* dev_status, void* stream) {
  using namespace mvb;
  if (!u || !dt || !z || !b || !c || !dt_bias || !a_log2e || !d || !out || !positions) return kInvalidArgument;
  if (num_seqs < 0 || num_tokens < 0 || channels <= 0 || num_states <= 0 || state_stride < num_states) return kInvalidArgument;
  if (state != nullptr && (state_slots == nullptr || num_slots <= 0)) return kInvalidArgument;
  if (cu_seqlens_q == nullptr && num_seqs != num_tokens) return kInvalidArgument;
  if (dtype != kBf16 && dtype != kF32) return kInvalidArgument;
  if (state_stride % 4 != 0 || !is_aligned(state, 16) || !is_aligned(a_log2e, 16)) return kMisaligned;
  if (num_tokens == 0 || num_seqs == 0) return kOk;
  const ScanParams p{u, u_row_stride, dt, dt_row_stride, z, z_row_stride, b, c, bc_row_stride, dt_bias, a_log2e, d, out,
                     out_row_stride, state, state_slots, num_slots, cu_seqlens_q, positions, num_seqs, num_tokens, channels,
                     num_states, state_stride,
                     bc_row_stride % 4 == 0 && is_aligned(b, 16 / (dtype == kBf16 ? 2 : 1)) && is_aligned(c, 16 / (dtype == kBf16 ? 2 : 1)),
                     dev_status};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return dtype == kBf16 ? launch_scan<__nv_bfloat16>(p, st) : launch_scan<float>(p, st);
}
