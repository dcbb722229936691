// Finishing a recurrent mixer's heads: out[t, h, :] = o / rms(o) * w * gate function * factor, from fp32 o [tokens, heads, vdim].
// One warp per (token, head).
//   norm_w     [vdim] shared by the heads (head_stride 0), or [heads, vdim] (head_stride vdim)
//   gate       raw, through a sigmoid or SiLU
//   NORMALISED o is first divided by max(|nq|, e^-m) + 1e-6 (nq, m: [tokens, heads])
#pragma once
#include "chunk_common.cuh"
#include "host_util.cuh"

namespace mvb {

enum GateKind : int { kGateSigmoid = 0, kGateSilu = 1 };

struct HeadNormParams {
  const float* o;
  const void* gate; int64_t gate_stride;
  const float* norm_w; int head_stride;
  void* out; int64_t out_stride;
  const float *nq, *m;                           // NORMALISED only
  int tokens, heads, vdim;
  float eps, out_scale;
};

constexpr float kNormaliserEps = 1e-6f;
__device__ __forceinline__ float normaliser_scale(float nq, float m) { return 1.f / (fmaxf(fabsf(nq), expf(-m)) + kNormaliserEps); }

template <class T, int GATE>
__device__ __forceinline__ float gate_of(float z) {
  const float s = sizeof(T) == 2 ? fast_rcp(1.f + fast_exp2(z * -1.4426950408889634f)) : sigmoid_f(z);
  return GATE == kGateSilu ? z * s : s;          // z -> -inf: the sigmoid is 0 and so is the product with the finite z
}

template <class T, int GATE, bool NORMALISED>
__global__ void __launch_bounds__(256) head_norm_kernel(const HeadNormParams p, bool vec) {
  const int64_t w = (static_cast<int64_t>(blockIdx.x) * 256 + threadIdx.x) >> 5;
  const int lane = threadIdx.x & 31, t = static_cast<int>(w / p.heads), h = static_cast<int>(w % p.heads);
  if (t >= p.tokens) return;
  const float* o = p.o + w * p.vdim;
  const float* nw = p.norm_w + h * p.head_stride;
  const T* gate = static_cast<const T*>(p.gate) + t * p.gate_stride + static_cast<int64_t>(h) * p.vdim;
  T* out = static_cast<T*>(p.out) + t * p.out_stride + static_cast<int64_t>(h) * p.vdim;
  float d = 1.f;
  if constexpr (NORMALISED) d = normaliser_scale(p.nq[w], p.m[w]);
  if (sizeof(T) == 2 && vec && p.vdim <= 128) {               // a lane keeps its four columns
    float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
    uint2 gw = make_uint2(0u, 0u);
    const int i = lane * 4;
    if (i < p.vdim) { x = *reinterpret_cast<const float4*>(o + i); gw = *reinterpret_cast<const uint2*>(gate + i); }
    x.x *= d; x.y *= d; x.z *= d; x.w *= d;
    const float r = p.out_scale * rsqrtf(warp_sum(x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w) / static_cast<float>(p.vdim) + p.eps);
    if (i < p.vdim) {
      const float4 n = *reinterpret_cast<const float4*>(nw + i);
      uint2 y;
      y.x = pack_bf16(x.x * r * n.x * gate_of<T, GATE>(bf16_lo(gw.x)), x.y * r * n.y * gate_of<T, GATE>(bf16_hi(gw.x)));
      y.y = pack_bf16(x.z * r * n.z * gate_of<T, GATE>(bf16_lo(gw.y)), x.w * r * n.w * gate_of<T, GATE>(bf16_hi(gw.y)));
      *reinterpret_cast<uint2*>(out + i) = y;
    }
    return;
  }
  float ss = 0.f;
  for (int i = lane; i < p.vdim; i += 32) { const float x = o[i] * d; ss += x * x; }
  const float r = p.out_scale / sqrtf(warp_sum(ss) / static_cast<float>(p.vdim) + p.eps);
  for (int i = lane; i < p.vdim; i += 32) out[i] = from_f<T>(o[i] * d * r * nw[i] * gate_of<T, GATE>(to_f(gate[i])));
}

template <class T, int GATE, bool NORMALISED = false>
static int launch_head_norm(const HeadNormParams& p, cudaStream_t st) {
  const int64_t blocks = (static_cast<int64_t>(p.tokens) * p.heads * 32 + 255) / 256;
  if (blocks > 0x7fffffffLL) return kUnsupportedShape;
  const bool vec = p.vdim % 4 == 0 && p.gate_stride % 4 == 0 && p.out_stride % 4 == 0 && is_aligned(p.gate, 8) &&
                   is_aligned(p.out, 8) && is_aligned(p.norm_w, 16) && is_aligned(p.o, 16);
  head_norm_kernel<T, GATE, NORMALISED><<<static_cast<unsigned>(blocks), 256, 0, st>>>(p, vec);
  return cudaGetLastError() == cudaSuccess ? kOk : kLaunchFailed;
}

}  // namespace mvb
