// Kernels that run in bf16 or in fp32: 16-byte vectors of the activation type, with fp32 values in registers.
#pragma once
#include <cuda_bf16.h>
#include <stdint.h>

#include "common.cuh"

namespace mvb {

enum DType : int { kBf16 = 0, kF32 = 1 };

template <class T> constexpr int kVec = 16 / static_cast<int>(sizeof(T));    // elements of a 16-byte vector

__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ float to_f(float v) { return v; }
template <class T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ __nv_bfloat16 from_f<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }

// V consecutive elements (V = kVec<T>: one 16-byte access at an aligned address; V = 1: one element)
template <class T, int V>
__device__ __forceinline__ void load_vec(const T* p, float (&out)[V]) {
  if constexpr (V == 1) {
    out[0] = to_f(*p);
  } else if constexpr (sizeof(T) == 2) {
    static_assert(V == 8, "");
    const uint4 w = *reinterpret_cast<const uint4*>(p);
    const uint32_t a[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) { out[2 * i] = bf16_lo(a[i]); out[2 * i + 1] = bf16_hi(a[i]); }
  } else {
    static_assert(V == 4, "");
    const float4 w = *reinterpret_cast<const float4*>(p);
    out[0] = w.x; out[1] = w.y; out[2] = w.z; out[3] = w.w;
  }
}
template <class T, int V>
__device__ __forceinline__ void store_vec(T* p, const float (&v)[V]) {
  if constexpr (V == 1) {
    *p = from_f<T>(v[0]);
  } else if constexpr (sizeof(T) == 2) {
    *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]), pack_bf16(v[4], v[5]), pack_bf16(v[6], v[7]));
  } else {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
  }
}
// V consecutive floats of the fp32 residual stream
template <int V>
__device__ __forceinline__ void load_f32(const float* p, float (&out)[V]) {
  if constexpr (V == 1) out[0] = *p;
  else {
#pragma unroll
    for (int i = 0; i < V; i += 4) {
      const float4 w = *reinterpret_cast<const float4*>(p + i);
      out[i] = w.x; out[i + 1] = w.y; out[i + 2] = w.z; out[i + 3] = w.w;
    }
  }
}
template <int V>
__device__ __forceinline__ void store_f32(float* p, const float (&v)[V]) {
  if constexpr (V == 1) *p = v[0];
  else {
#pragma unroll
    for (int i = 0; i < V; i += 4) *reinterpret_cast<float4*>(p + i) = make_float4(v[i], v[i + 1], v[i + 2], v[i + 3]);
  }
}

// z >= -inf: log(1 + e^z) without overflow; 1 / (1 + e^-z)
__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
// The same for bf16 activations, where a few fp32 ulps do not matter but instructions do: with y = e^-|z| in (0, 1] and
// w = y / (2 + y), log(1 + y) = 2 artanh(w) = 2 w (1 + w^2/3 + w^4/5 + ...), w <= 1/3, so eight terms reach fp32.
__device__ __forceinline__ float softplus_fast(float z) {
  const float y = fast_exp2(-1.4426950408889634f * fabsf(z)), w = y * fast_rcp(2.f + y), q = w * w;
  float t = 1.f / 15.f;
  t = fmaf(t, q, 1.f / 13.f); t = fmaf(t, q, 1.f / 11.f); t = fmaf(t, q, 1.f / 9.f); t = fmaf(t, q, 1.f / 7.f);
  t = fmaf(t, q, 1.f / 5.f); t = fmaf(t, q, 1.f / 3.f); t = fmaf(t, q, 1.f);
  return fmaf(2.f * w, t, fmaxf(z, 0.f));
}
template <class T> __device__ __forceinline__ float softplus_of(float z) {
  if constexpr (sizeof(T) == 2) return softplus_fast(z);
  else return softplus_f(z);
}
__device__ __forceinline__ float sigmoid_f(float z) { return 1.f / (1.f + expf(-z)); }

// the sequence of packed row t: the largest s with cu[s] <= t (cu ascending, cu[0] = 0, t < cu[n]); rows of a step
// without cu (every sequence brings one token) are their own sequence
__device__ __forceinline__ int seq_of_row(const int32_t* __restrict__ cu, int n, int t) {
  if (cu == nullptr) return t;
  int lo = 0, hi = n;                       // cu[lo] <= t < cu[hi]
  while (hi - lo > 1) {
    const int mid = (lo + hi) >> 1;
    if (cu[mid] <= t) lo = mid; else hi = mid;
  }
  return lo;
}

}  // namespace mvb
