// Decoder glue around an fp32 residual stream (activations in bf16 or fp32): embedding lookup + first norm, branch
// norm + residual add + next norm, the clamped gated activation, xIELU, and the tanh cap of the logits.
//
// One CTA per row for the norms; a row stays in registers between the reductions, so the residual stream is read and
// written once per sublayer.  Roofline: HBM at prefill (rows * hidden * (8 + 2 * sizeof(T)) bytes for the add + norm),
// launch latency at decode.
#include "dtype.cuh"
#include "host_util.cuh"
#include "mini_vllm_b200.h"

namespace mvb {

struct NormParams {
  float* x;                     // residual stream [rows, width], fp32
  const void* y;                // branch output (add form) or the embedding table (lookup form)
  int64_t y_stride;
  const int64_t* ids;           // lookup form: row r of x becomes table[ids[r]]
  int64_t vocab;
  const void* y_weight;         // nullptr: the branch output is added as it is
  const void* weight;
  void* out;
  const int32_t* row_ends;      // nullptr, or: output row r comes from source row row_ends[r + 1] - 1 and x is left alone
  int width;
  float eps;
  // the form with two norms of the same stream (PAIR): a factor of the looked-up row, further rows to add (row `row` of the stream
  // gets extra[extra_index[row, j]], j < num_extra, none for an index of -1, and own_weights[row] times its row of `own`), and a second
  // weight and output (nullptr: none)
  float table_scale;
  const void* extra; const int32_t* extra_index; int num_extra; int64_t extra_stride, extra_rows;
  const void* own; int64_t own_stride; const float* own_weights;
  const void* weight2;
  void* out2;
  int* dev_status;
};

__device__ __forceinline__ float row_sum(float v, float* scratch) {
#pragma unroll
  for (int off = 16; off > 0; off >>= 1) v += __shfl_xor_sync(0xffffffffu, v, off);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
  if (nw == 1) return v;
  __syncthreads();                                          // scratch may still be read from a previous call
  if (lane == 0) scratch[warp] = v;
  __syncthreads();
  float s = lane < nw ? scratch[lane] : 0.f;
#pragma unroll
  for (int off = 16; off > 0; off >>= 1) s += __shfl_xor_sync(0xffffffffu, s, off);
  return s;
}

template <class T, int V, int ITEMS, bool PAIR>
__global__ void __launch_bounds__(1024) residual_norm_kernel(const NormParams p) {
  __shared__ float scratch[32];
  const int out_row = blockIdx.x;
  const int row = p.row_ends != nullptr ? p.row_ends[out_row + 1] - 1 : out_row;
  if (row < 0) return;
  const int nvec = p.width / V, nt = blockDim.x;
  float* xrow = p.x + static_cast<int64_t>(row) * p.width;
  const T* yrow = static_cast<const T*>(p.y) + static_cast<int64_t>(row) * p.y_stride;
  if (p.ids != nullptr) {
    int64_t id = p.ids[row];
    if (id < 0 || id >= p.vocab) {
      if (threadIdx.x == 0) report(p.dev_status, kDevBadPosition, row);
      id = 0;
    }
    yrow = static_cast<const T*>(p.y) + id * p.y_stride;
  }
  float v[ITEMS][V], res[ITEMS][V];
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < ITEMS; ++k) {
    const int i = threadIdx.x + k * nt;
    if (i >= nvec) continue;
    load_vec<T, V>(yrow + i * V, v[k]);
    if (p.ids == nullptr) load_f32<V>(xrow + i * V, res[k]);
    if constexpr (PAIR) {
      if (p.ids != nullptr) {
#pragma unroll
        for (int j = 0; j < V; ++j) v[k][j] *= p.table_scale;
      }
    }
  }
  if constexpr (PAIR) {
    for (int e = 0; e < p.num_extra; ++e) {
      const int32_t r = p.extra_index[static_cast<int64_t>(row) * p.num_extra + e];
      if (r == -1) continue;
      if (r < 0 || r >= p.extra_rows) {
        if (threadIdx.x == 0) report(p.dev_status, kDevBadPosition, row);
        continue;
      }
      const T* erow = static_cast<const T*>(p.extra) + r * p.extra_stride;
#pragma unroll
      for (int k = 0; k < ITEMS; ++k) {
        const int i = threadIdx.x + k * nt;
        if (i >= nvec) continue;
        float a[V];
        load_vec<T, V>(erow + i * V, a);
#pragma unroll
        for (int j = 0; j < V; ++j) v[k][j] += a[j];
      }
    }
    const float own = p.own_weights != nullptr ? p.own_weights[row] : 0.f;
    if (own != 0.f) {
      const T* orow = static_cast<const T*>(p.own) + row * p.own_stride;
#pragma unroll
      for (int k = 0; k < ITEMS; ++k) {
        const int i = threadIdx.x + k * nt;
        if (i >= nvec) continue;
        float a[V];
        load_vec<T, V>(orow + i * V, a);
#pragma unroll
        for (int j = 0; j < V; ++j) v[k][j] = fmaf(own, a[j], v[k][j]);
      }
    }
  }
  if (p.y_weight != nullptr) {
#pragma unroll
    for (int k = 0; k < ITEMS; ++k)
      if (threadIdx.x + k * nt < nvec) {
#pragma unroll
        for (int j = 0; j < V; ++j) ss += v[k][j] * v[k][j];
      }
    const float r = rsqrtf(row_sum(ss, scratch) / static_cast<float>(p.width) + p.eps);
#pragma unroll
    for (int k = 0; k < ITEMS; ++k) {
      const int i = threadIdx.x + k * nt;
      if (i >= nvec) continue;
      float w[V];
      load_vec<T, V>(static_cast<const T*>(p.y_weight) + i * V, w);
#pragma unroll
      for (int j = 0; j < V; ++j) v[k][j] = v[k][j] * r * w[j];
    }
  }
  ss = 0.f;
#pragma unroll
  for (int k = 0; k < ITEMS; ++k) {
    const int i = threadIdx.x + k * nt;
    if (i >= nvec) continue;
    if (p.ids == nullptr) {
#pragma unroll
      for (int j = 0; j < V; ++j) v[k][j] += res[k][j];
    }
    if (p.row_ends == nullptr) store_f32<V>(xrow + i * V, v[k]);
#pragma unroll
    for (int j = 0; j < V; ++j) ss += v[k][j] * v[k][j];
  }
  const float r = rsqrtf(row_sum(ss, scratch) / static_cast<float>(p.width) + p.eps);
  T* orow = static_cast<T*>(p.out) + static_cast<int64_t>(out_row) * p.width;
#pragma unroll
  for (int k = 0; k < ITEMS; ++k) {
    const int i = threadIdx.x + k * nt;
    if (i >= nvec) continue;
    float w[V];
    load_vec<T, V>(static_cast<const T*>(p.weight) + i * V, w);
#pragma unroll
    for (int j = 0; j < V; ++j) w[j] = v[k][j] * r * w[j];
    store_vec<T, V>(orow + i * V, w);
    if constexpr (PAIR) {
      if (p.weight2 != nullptr) {
        load_vec<T, V>(static_cast<const T*>(p.weight2) + i * V, w);
#pragma unroll
        for (int j = 0; j < V; ++j) w[j] = v[k][j] * r * w[j];
        store_vec<T, V>(static_cast<T*>(p.out2) + static_cast<int64_t>(out_row) * p.width + i * V, w);
      }
    }
  }
}

template <class T, int V, bool PAIR>
static int launch_norm_v(const NormParams& p, int rows, cudaStream_t st) {
  const int nvec = p.width / V;
  // about four vectors in flight per thread for wide rows, a whole warp at least for narrow ones
  int items = nvec <= 128 ? 1 : (nvec <= 512 ? 2 : 4);
  while (items < 8 && (nvec + items - 1) / items > 1024) items *= 2;
  const int nt = ((nvec + items - 1) / items + 31) / 32 * 32;
  if (nt > 1024) return kUnsupportedShape;
  if (items == 1) residual_norm_kernel<T, V, 1, PAIR><<<rows, nt, 0, st>>>(p);
  else if (items == 2) residual_norm_kernel<T, V, 2, PAIR><<<rows, nt, 0, st>>>(p);
  else if (items == 4) residual_norm_kernel<T, V, 4, PAIR><<<rows, nt, 0, st>>>(p);
  else residual_norm_kernel<T, V, 8, PAIR><<<rows, nt, 0, st>>>(p);
  return cudaGetLastError() == cudaSuccess ? kOk : kLaunchFailed;
}

template <class T, bool PAIR = false>
static int launch_norm(const NormParams& p, int rows, cudaStream_t st) {
  constexpr int V = kVec<T>;
  const bool vec = p.width % V == 0 && p.width % 4 == 0 && p.y_stride % V == 0 && is_aligned(p.x, 16) && is_aligned(p.y, 16) &&
                   is_aligned(p.y_weight, 16) && is_aligned(p.weight, 16) && is_aligned(p.out, 16) &&
                   p.extra_stride % V == 0 && is_aligned(p.extra, 16) && p.own_stride % V == 0 && is_aligned(p.own, 16) && is_aligned(p.weight2, 16) && is_aligned(p.out2, 16);
  return vec ? launch_norm_v<T, V, PAIR>(p, rows, st) : launch_norm_v<T, 1, PAIR>(p, rows, st);
}

// out = g sigmoid(alpha g) (u + offset) with g = min(gate, limit), u = clamp(up, -limit, limit), times sigmoid(row_gate) of the row
// (alpha 1, offset 0, limit infinite: the SiLU-gated unit)
template <class T, int V>
__global__ void __launch_bounds__(128) clamped_glu_kernel(const T* __restrict__ gate_up, int64_t in_stride, T* __restrict__ out,
                                                          int64_t out_stride, int rows, int inter, float limit, float alpha,
                                                          float offset, const T* __restrict__ row_gate, int64_t gate_stride) {
  const int c = (blockIdx.x * 128 + threadIdx.x) * V;
  if (c >= inter) return;
  const float k = -alpha * 1.4426950408889634f;
  for (int t = blockIdx.y; t < rows; t += gridDim.y) {
    const T* r = gate_up + t * in_stride + c;
    float g[V], u[V];
    load_vec<T, V>(r, g);
    load_vec<T, V>(r + inter, u);
    const float f = row_gate != nullptr ? sigmoid_f(to_f(row_gate[t * gate_stride])) : 1.f;
#pragma unroll
    for (int i = 0; i < V; ++i) {
      const float gi = fminf(g[i], limit), ui = fminf(fmaxf(u[i], -limit), limit);
      // gi -> -inf: exp2 -> inf, the reciprocal -> 0 and the product with the finite gi -> 0
      g[i] = gi * fast_rcp(1.f + fast_exp2(k * gi)) * (ui + offset) * f;
    }
    store_vec<T, V>(out + t * out_stride + c, g);
  }
}

template <class T>
static int launch_glu(const void* gu, int64_t is, void* out, int64_t os, int rows, int inter, float limit, float alpha, float offset,
                      const void* row_gate, int64_t gate_stride, cudaStream_t st) {
  constexpr int V = kVec<T>;
  const bool vec = inter % V == 0 && is % V == 0 && os % V == 0 && is_aligned(gu, 16) && is_aligned(out, 16);
  const int v = vec ? V : 1, bx = (inter + 128 * v - 1) / (128 * v);
  int by = rows, cap = (sm_count() * 16 + bx - 1) / bx;
  if (by > cap) by = cap;
  if (by > 65535) by = 65535;
  auto tg = static_cast<const T*>(gu), tr = static_cast<const T*>(row_gate);
  auto to = static_cast<T*>(out);
  if (vec) clamped_glu_kernel<T, V><<<dim3(bx, by), 128, 0, st>>>(tg, is, to, os, rows, inter, limit, alpha, offset, tr, gate_stride);
  else clamped_glu_kernel<T, 1><<<dim3(bx, by), 128, 0, st>>>(tg, is, to, os, rows, inter, limit, alpha, offset, tr, gate_stride);
  return cudaGetLastError() == cudaSuccess ? kOk : kLaunchFailed;
}

// xIELU: act[0] z^2 + z / 2 for z > 0, act[1] (e^z - 1 - z) + z / 2 for z <= 0
template <class T, int V>
__global__ void __launch_bounds__(128) xielu_kernel(const T* __restrict__ in, int64_t in_stride, T* __restrict__ out, int64_t out_stride,
                                                    int rows, int cols, const float* __restrict__ act) {
  const int c = (blockIdx.x * 128 + threadIdx.x) * V;
  if (c >= cols) return;
  const float above = act[0], below = act[1];
  for (int t = blockIdx.y; t < rows; t += gridDim.y) {
    float z[V];
    load_vec<T, V>(in + t * in_stride + c, z);
#pragma unroll
    for (int i = 0; i < V; ++i) {
      const float n = fminf(z[i], 0.f);
      float e;                                    // e^n - 1 - n, where a small n would leave the difference nothing but rounding
      if (sizeof(T) == 2) e = n > -0.25f ? n * n * fmaf(n, fmaf(n, fmaf(n, 1.f / 120.f, 1.f / 24.f), 1.f / 6.f), 0.5f)
                                         : fast_exp2(n * 1.4426950408889634f) - 1.f - n;
      else e = expm1f(n) - n;
      z[i] = (z[i] > 0.f ? above * z[i] * z[i] : below * e) + 0.5f * z[i];
    }
    store_vec<T, V>(out + t * out_stride + c, z);
  }
}

template <class T>
static int launch_xielu(const void* in, int64_t is, void* out, int64_t os, int rows, int cols, const float* act, cudaStream_t st) {
  constexpr int V = kVec<T>;
  const bool vec = cols % V == 0 && is % V == 0 && os % V == 0 && is_aligned(in, 16) && is_aligned(out, 16);
  const int v = vec ? V : 1, bx = (cols + 128 * v - 1) / (128 * v);
  int by = rows, cap = (sm_count() * 16 + bx - 1) / bx;
  if (by > cap) by = cap;
  if (by > 65535) by = 65535;
  auto ti = static_cast<const T*>(in);
  auto to = static_cast<T*>(out);
  if (vec) xielu_kernel<T, V><<<dim3(bx, by), 128, 0, st>>>(ti, is, to, os, rows, cols, act);
  else xielu_kernel<T, 1><<<dim3(bx, by), 128, 0, st>>>(ti, is, to, os, rows, cols, act);
  return cudaGetLastError() == cudaSuccess ? kOk : kLaunchFailed;
}

template <class TI, class TO>
__global__ void __launch_bounds__(256) cap_logits_kernel(const TI* __restrict__ in, int64_t in_stride, TO* __restrict__ out,
                                                         int64_t out_stride, int cols, float cap, float inv_cap) {
  const int64_t row = blockIdx.y;
  for (int c = blockIdx.x * 256 + threadIdx.x; c < cols; c += gridDim.x * 256) {
    const float v = to_f(in[row * in_stride + c]);
    out[row * out_stride + c] = from_f<TO>(cap > 0.f ? cap * tanhf(v * inv_cap) : v);
  }
}

// greedy token of fp32 logits: one CTA per row, the lowest column winning ties
__global__ void __launch_bounds__(1024) argmax_f32_kernel(const float* __restrict__ logits, int64_t stride, int cols,
                                                          int64_t* __restrict__ out, int64_t* __restrict__ scatter_table,
                                                          const int32_t* __restrict__ scatter_index) {
  __shared__ float bv[32];
  __shared__ int bi[32];
  const float* row = logits + blockIdx.x * stride;
  float v = -INFINITY;
  int idx = cols;
  auto take = [&](float x, int i) { if (x > v || (x == v && i < idx)) { v = x; idx = i; } };
  for (int c = threadIdx.x; c < cols; c += 1024) take(row[c], c);
#pragma unroll
  for (int off = 16; off > 0; off >>= 1) {
    const float x = __shfl_xor_sync(0xffffffffu, v, off);
    const int i = __shfl_xor_sync(0xffffffffu, idx, off);
    take(x, i);
  }
  if ((threadIdx.x & 31) == 0) { bv[threadIdx.x >> 5] = v; bi[threadIdx.x >> 5] = idx; }
  __syncthreads();
  if (threadIdx.x == 0) {
    for (int w = 1; w < 32; ++w) take(bv[w], bi[w]);
    const int64_t tok = idx < cols ? idx : 0;
    out[blockIdx.x] = tok;
    if (scatter_table != nullptr) scatter_table[scatter_index[blockIdx.x]] = tok;
  }
}

}  // namespace mvb

extern "C" int mvb_argmax_f32(const float* logits, int64_t row_stride, int rows, int cols, int64_t* out, int64_t* scatter_table,
                              const int32_t* scatter_index, void* stream) {
  using namespace mvb;
  if (!logits || !out || rows < 0 || cols <= 0 || (scatter_table == nullptr) != (scatter_index == nullptr)) return kInvalidArgument;
  if (rows == 0) return kOk;
  argmax_f32_kernel<<<rows, 1024, 0, static_cast<cudaStream_t>(stream)>>>(logits, row_stride, cols, out, scatter_table, scatter_index);
  return cudaGetLastError() == cudaSuccess ? kOk : kLaunchFailed;
}

extern "C" int mvb_residual_norm(int dtype, float* x, const void* y, int64_t y_row_stride, const void* y_weight,
                                 const void* weight, void* out, const int32_t* row_ends, int rows, int width, float eps,
                                 void* stream) {
  using namespace mvb;
  if (!x || !y || !weight || !out || rows < 0 || width <= 0 || (dtype != kBf16 && dtype != kF32)) return kInvalidArgument;
  if (rows == 0) return kOk;
  const NormParams p{x, y, y_row_stride, nullptr, 0, y_weight, weight, out, row_ends, width, eps, 1.f, nullptr, nullptr, 0, 0, 0, nullptr, 0, nullptr, nullptr,
                     nullptr, nullptr};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return dtype == kBf16 ? launch_norm<__nv_bfloat16>(p, rows, st) : launch_norm<float>(p, rows, st);
}

extern "C" int mvb_embed_norm(int dtype, const int64_t* ids, const void* table, int64_t vocab, float* x, const void* weight,
                              void* out, int rows, int width, float eps, int32_t* dev_status, void* stream) {
  using namespace mvb;
  if (!ids || !table || !x || !weight || !out || rows < 0 || width <= 0 || vocab <= 0 || (dtype != kBf16 && dtype != kF32))
    return kInvalidArgument;
  if (rows == 0) return kOk;
  const NormParams p{x, table, width, ids, vocab, nullptr, weight, out, nullptr, width, eps, 1.f, nullptr, nullptr, 0, 0, 0, nullptr,
                     0, nullptr, nullptr, nullptr, dev_status};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return dtype == kBf16 ? launch_norm<__nv_bfloat16>(p, rows, st) : launch_norm<float>(p, rows, st);
}

extern "C" int mvb_glu(int dtype, const void* gate_up, int64_t in_row_stride, void* out, int64_t out_row_stride, int rows,
                       int intermediate, float limit, float alpha, float offset, const void* row_gate, int64_t gate_row_stride,
                       void* stream) {
  using namespace mvb;
  if (!gate_up || !out || rows < 0 || intermediate <= 0 || (dtype != kBf16 && dtype != kF32)) return kInvalidArgument;
  if (rows == 0) return kOk;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return dtype == kBf16 ? launch_glu<__nv_bfloat16>(gate_up, in_row_stride, out, out_row_stride, rows, intermediate, limit, alpha, offset,
                                                    row_gate, gate_row_stride, st)
                        : launch_glu<float>(gate_up, in_row_stride, out, out_row_stride, rows, intermediate, limit, alpha, offset,
                                            row_gate, gate_row_stride, st);
}

extern "C" int mvb_clamped_glu(int dtype, const void* gate_up, int64_t in_row_stride, void* out, int64_t out_row_stride,
                               int rows, int intermediate, float limit, float alpha, void* stream) {
  return mvb_glu(dtype, gate_up, in_row_stride, out, out_row_stride, rows, intermediate, limit, alpha, 1.f, nullptr, 0, stream);
}

extern "C" int mvb_embed_norm_pair(int dtype, const int64_t* ids, const void* table, int64_t vocab, float scale, float* x,
                                   const void* weight, void* out, const void* weight2, void* out2, int rows, int width, float eps,
                                   int32_t* dev_status, void* stream) {
  using namespace mvb;
  if (!ids || !table || !x || !weight || !out || rows < 0 || width <= 0 || vocab <= 0 || (dtype != kBf16 && dtype != kF32))
    return kInvalidArgument;
  if ((weight2 == nullptr) != (out2 == nullptr)) return kInvalidArgument;
  if (rows == 0) return kOk;
  const NormParams p{x, table, width, ids, vocab, nullptr, weight, out, nullptr, width, eps, scale, nullptr, nullptr, 0, 0, 0, nullptr, 0, nullptr, weight2, out2,
                     dev_status};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return dtype == kBf16 ? launch_norm<__nv_bfloat16, true>(p, rows, st) : launch_norm<float, true>(p, rows, st);
}

extern "C" int mvb_residual_norm_pair_ext(int dtype, float* x, const void* y, int64_t y_row_stride, const void* extra,
                                          int64_t extra_row_stride, int64_t extra_rows, const int32_t* extra_index, int num_extra,
                                          const void* own, int64_t own_row_stride, const float* own_weights, const void* weight, void* out,
                                          const void* weight2, void* out2, const int32_t* row_ends, int rows, int width, float eps,
                                          int32_t* dev_status, void* stream) {
  using namespace mvb;
  if (!x || !y || !weight || !out || rows < 0 || width <= 0 || (dtype != kBf16 && dtype != kF32)) return kInvalidArgument;
  if ((weight2 == nullptr) != (out2 == nullptr) || num_extra < 0 || (num_extra > 0 && (!extra || !extra_index))) return kInvalidArgument;
  if (own_weights != nullptr && own == nullptr) return kInvalidArgument;
  if (rows == 0) return kOk;
  const NormParams p{x, y, y_row_stride, nullptr, 0, nullptr, weight, out, row_ends, width, eps, 1.f, extra, extra_index, num_extra,
                     extra_row_stride, extra_rows, own, own_row_stride, own_weights, weight2, out2, dev_status};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return dtype == kBf16 ? launch_norm<__nv_bfloat16, true>(p, rows, st) : launch_norm<float, true>(p, rows, st);
}

extern "C" int mvb_residual_norm_pair(int dtype, float* x, const void* y, int64_t y_row_stride, const void* extra,
                                      int64_t extra_row_stride, int64_t extra_rows, const int32_t* extra_index, int num_extra,
                                      const void* weight, void* out, const void* weight2, void* out2, const int32_t* row_ends, int rows,
                                      int width, float eps, int32_t* dev_status, void* stream) {
  return mvb_residual_norm_pair_ext(dtype, x, y, y_row_stride, extra, extra_row_stride, extra_rows, extra_index, num_extra, nullptr, 0,
                                    nullptr, weight, out, weight2, out2, row_ends, rows, width, eps, dev_status, stream);
}

extern "C" int mvb_xielu(int dtype, const void* in, int64_t in_row_stride, void* out, int64_t out_row_stride, int rows, int cols,
                         const float* act, void* stream) {
  using namespace mvb;
  if (!in || !out || !act || rows < 0 || cols <= 0 || (dtype != kBf16 && dtype != kF32)) return kInvalidArgument;
  if (rows == 0) return kOk;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return dtype == kBf16 ? launch_xielu<__nv_bfloat16>(in, in_row_stride, out, out_row_stride, rows, cols, act, st)
                        : launch_xielu<float>(in, in_row_stride, out, out_row_stride, rows, cols, act, st);
}

extern "C" int mvb_cap_logits(int in_dtype, int out_dtype, const void* in, int64_t in_row_stride, void* out,
                              int64_t out_row_stride, int rows, int cols, float cap, void* stream) {
  using namespace mvb;
  if (!in || !out || rows < 0 || cols <= 0 || !(cap >= 0.f)) return kInvalidArgument;
  if (rows == 0) return kOk;
  if (rows > 65535) return kUnsupportedShape;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  int bx = (cols + 1023) / 1024;
  if (bx > 64) bx = 64;
  const dim3 grid(bx, rows);
  const float inv = cap > 0.f ? 1.f / cap : 0.f;
  auto bi = static_cast<const __nv_bfloat16*>(in); auto fi = static_cast<const float*>(in);
  auto bo = static_cast<__nv_bfloat16*>(out); auto fo = static_cast<float*>(out);
  if (in_dtype == kBf16 && out_dtype == kBf16) cap_logits_kernel<<<grid, 256, 0, st>>>(bi, in_row_stride, bo, out_row_stride, cols, cap, inv);
  else if (in_dtype == kBf16 && out_dtype == kF32) cap_logits_kernel<<<grid, 256, 0, st>>>(bi, in_row_stride, fo, out_row_stride, cols, cap, inv);
  else if (in_dtype == kF32 && out_dtype == kBf16) cap_logits_kernel<<<grid, 256, 0, st>>>(fi, in_row_stride, bo, out_row_stride, cols, cap, inv);
  else if (in_dtype == kF32 && out_dtype == kF32) cap_logits_kernel<<<grid, 256, 0, st>>>(fi, in_row_stride, fo, out_row_stride, cols, cap, inv);
  else return kInvalidArgument;
  return cudaGetLastError() == cudaSuccess ? kOk : kLaunchFailed;
}
