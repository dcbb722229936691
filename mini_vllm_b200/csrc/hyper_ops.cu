// Hyper-connections: the residual stream as `streams` fp32 copies X [rows, streams, width], and the activation of its feed-forward.
//
// hyper_norm_kernel, one CTA per row, between two sublayers:
//   X_t <- sum_s mix[s, t] X_s + out[t] y        (the sublayer that has run; all streams at once from the old ones)
//   u    = sum_s in[s] X_s                        (the next sublayer; in == nullptr: the plain sum, in front of the head)
//   h    = norm(u) * weight, in `groups` equal consecutive parts, each over its own root mean square
// or, in front of the first sublayer, X_t <- table[ids] + pos_table[positions] for every t.  The streams are read once and written once
// (roofline: HBM, rows * width * (8 * streams + 2 * sizeof(T)) bytes).
//
// poly_norm_kernel: a N(z) + b N(z^2) + c N(z^3) + e over a row, N(v) = v / rms(v); the row waits in shared memory for its three sums.
#include "chunk_common.cuh"
#include "host_util.cuh"
#include "mini_vllm_b200.h"

namespace mvb {

struct HyperParams {
  float* x;                     // [rows, streams, width]
  const void* y; int64_t y_stride;              // sublayer output, or the embedding table
  const int64_t *ids, *positions;               // lookup form
  const void* pos_table; int64_t vocab, max_positions;
  const float *mix, *out_w, *in_w;              // [streams, streams] from, to; [streams]; [streams]
  const void* weight;
  void* h;
  const int32_t* row_ends;      // nullptr, or: output row r comes from source row row_ends[r + 1] - 1 and x is left alone
  int width, streams, groups;
  float eps;
  int* dev_status;
};

// SP: streams rounded up to a power of two
template <class T, int V, int SP>
__global__ void __launch_bounds__(512) hyper_norm_kernel(const HyperParams p) {
  extern __shared__ __align__(16) float sm[];
  const int nvec = p.width / V, nt = blockDim.x, tid = threadIdx.x, S = p.streams;
  float* u_s = sm;                               // [width]
  float* part = u_s + p.width;                   // [nvec] sums of squares
  float* rstd = part + nvec;                     // [groups]
  __shared__ float mix[SP][SP], out_w[SP], in_w[SP];
  const int out_row = blockIdx.x, row = p.row_ends != nullptr ? p.row_ends[out_row + 1] - 1 : out_row;
  if (row < 0) return;
  const bool lookup = p.ids != nullptr;
  for (int i = tid; i < SP * SP; i += nt) {
    const int s = i / SP, t = i % SP;
    mix[s][t] = !lookup && s < S && t < S ? p.mix[s * S + t] : 0.f;
  }
  for (int i = tid; i < SP; i += nt) {
    out_w[i] = !lookup && i < S ? p.out_w[i] : (i < S ? 1.f : 0.f);
    in_w[i] = i < S ? (p.in_w != nullptr ? p.in_w[i] : 1.f) : 0.f;
  }
  const T* yrow = static_cast<const T*>(p.y) + static_cast<int64_t>(row) * p.y_stride;
  const T* prow = nullptr;
  if (lookup) {
    int64_t id = p.ids[row], pos = p.positions[row];
    if (id < 0 || id >= p.vocab || pos < 0 || pos >= p.max_positions) {
      if (tid == 0) report(p.dev_status, kDevBadPosition, row);
      id = pos = 0;
    }
    yrow = static_cast<const T*>(p.y) + id * p.y_stride;
    prow = static_cast<const T*>(p.pos_table) + pos * p.width;
  }
  float* xrow = p.x + static_cast<int64_t>(row) * S * p.width;
  __syncthreads();
  for (int i = tid; i < nvec; i += nt) {
    float y[V], u[V], x[SP][V];
    load_vec<T, V>(yrow + i * V, y);
    if (!lookup) {
#pragma unroll
      for (int s = 0; s < SP; ++s)
        if (s < S) load_f32<V>(xrow + static_cast<int64_t>(s) * p.width + i * V, x[s]);
    } else {
      float e[V];
      load_vec<T, V>(prow + i * V, e);
#pragma unroll
      for (int j = 0; j < V; ++j) y[j] += e[j];
    }
#pragma unroll
    for (int j = 0; j < V; ++j) u[j] = 0.f;
#pragma unroll
    for (int t = 0; t < SP; ++t) {
      if (t >= S) continue;
      float n[V];
#pragma unroll
      for (int j = 0; j < V; ++j) n[j] = out_w[t] * y[j];
      if (!lookup) {
#pragma unroll
        for (int s = 0; s < SP; ++s)
          if (s < S) {
#pragma unroll
            for (int j = 0; j < V; ++j) n[j] = fmaf(mix[s][t], x[s][j], n[j]);
          }
      }
      if (p.row_ends == nullptr) store_f32<V>(xrow + static_cast<int64_t>(t) * p.width + i * V, n);
#pragma unroll
      for (int j = 0; j < V; ++j) u[j] = fmaf(in_w[t], n[j], u[j]);
    }
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < V; ++j) ss += u[j] * u[j];
    part[i] = ss;
    store_f32<V>(u_s + i * V, u);
  }
  __syncthreads();
  const int per = nvec / p.groups, warp = tid >> 5, lane = tid & 31;
  for (int g = warp; g < p.groups; g += nt >> 5) {
    float ss = 0.f;
    for (int i = lane; i < per; i += 32) ss += part[g * per + i];
    ss = warp_sum(ss);
    if (lane == 0) rstd[g] = 1.f / sqrtf(ss * p.groups / static_cast<float>(p.width) + p.eps);
  }
  __syncthreads();
  T* hrow = static_cast<T*>(p.h) + static_cast<int64_t>(out_row) * p.width;
  for (int i = tid; i < nvec; i += nt) {
    float u[V], w[V];
    load_f32<V>(u_s + i * V, u);
    load_vec<T, V>(static_cast<const T*>(p.weight) + i * V, w);
    const float r = rstd[i / per];
#pragma unroll
    for (int j = 0; j < V; ++j) w[j] *= u[j] * r;
    store_vec<T, V>(hrow + i * V, w);
  }
}

template <class T, int V, int SP>
static int launch_hyper_sp(const HyperParams& p, int rows, cudaStream_t st) {
  const int nvec = p.width / V;
  int nt = (nvec + 31) / 32 * 32;
  if (nt > 512) nt = 512;
  const size_t smem = (static_cast<size_t>(p.width) + nvec + p.groups) * sizeof(float);
  if (smem > 200 * 1024) return kUnsupportedShape;
  struct Tag {};
  const int rc = opt_in_dynamic_smem<Tag>(reinterpret_cast<const void*>(&hyper_norm_kernel<T, V, SP>), smem);
  if (rc != kOk) return rc;
  hyper_norm_kernel<T, V, SP><<<rows, nt, smem, st>>>(p);
  return cudaGetLastError() == cudaSuccess ? kOk : kLaunchFailed;
}
template <class T, int V>
static int launch_hyper_v(const HyperParams& p, int rows, cudaStream_t st) {
  if (p.streams <= 1) return launch_hyper_sp<T, V, 1>(p, rows, st);
  if (p.streams <= 2) return launch_hyper_sp<T, V, 2>(p, rows, st);
  if (p.streams <= 4) return launch_hyper_sp<T, V, 4>(p, rows, st);
  if (p.streams <= 8) return launch_hyper_sp<T, V, 8>(p, rows, st);
  if (p.streams <= 16) return launch_hyper_sp<T, V, 16>(p, rows, st);
  return kUnsupportedShape;
}
template <class T>
static int launch_hyper(const HyperParams& p, int rows, cudaStream_t st) {
  constexpr int V = kVec<T>;
  const bool vec = (p.width / p.groups) % V == 0 && p.y_stride % V == 0 && is_aligned(p.x, 16) && is_aligned(p.y, 16) &&
                   is_aligned(p.pos_table, 16) && is_aligned(p.weight, 16) && is_aligned(p.h, 16);
  return vec ? launch_hyper_v<T, V>(p, rows, st) : launch_hyper_v<T, 1>(p, rows, st);
}

// ---- activation --------------------------------------------------------------------------------------------
template <class T, int V>
__global__ void __launch_bounds__(512) poly_norm_kernel(const T* __restrict__ z, int64_t z_stride, T* __restrict__ out, int64_t out_stride,
                                                        int cols, int pad_cols, const float* __restrict__ act, float eps) {
  extern __shared__ __align__(16) uint8_t raw[];
  T* z_s = reinterpret_cast<T*>(raw);
  __shared__ float sums[3][16];
  const int tid = threadIdx.x, nt = blockDim.x, warp = tid >> 5, lane = tid & 31, nvec = cols / V;
  const T* zrow = z + blockIdx.x * z_stride;
  T* orow = out + blockIdx.x * out_stride;
  float s[3] = {0.f, 0.f, 0.f};
  for (int i = tid; i < nvec; i += nt) {
    float v[V];
    load_vec<T, V>(zrow + i * V, v);
    store_vec<T, V>(z_s + i * V, v);             // (exact: the values came in this type)
#pragma unroll
    for (int j = 0; j < V; ++j) {
      const float q = v[j] * v[j];
      s[0] += q; s[1] = fmaf(q, q, s[1]); s[2] = fmaf(q * q, q, s[2]);
    }
  }
#pragma unroll
  for (int k = 0; k < 3; ++k) {
    s[k] = warp_sum(s[k]);
    if (lane == 0) sums[k][warp] = s[k];
  }
  __syncthreads();
  float r[3];
#pragma unroll
  for (int k = 0; k < 3; ++k) {
    float t = 0.f;
    for (int w = 0; w < nt / 32; ++w) t += sums[k][w];
    r[k] = act[k] / sqrtf(t / static_cast<float>(cols) + eps);
  }
  const float e = act[3];
  for (int i = tid; i < nvec; i += nt) {
    float v[V];
    load_vec<T, V>(z_s + i * V, v);
#pragma unroll
    for (int j = 0; j < V; ++j) v[j] = fmaf(v[j], fmaf(v[j], fmaf(v[j], r[2], r[1]), r[0]), e);
    store_vec<T, V>(orow + i * V, v);
  }
  for (int i = cols + tid; i < pad_cols; i += nt) orow[i] = from_f<T>(0.f);
}

template <class T>
static int launch_poly(const void* z, int64_t zs, void* out, int64_t os, int rows, int cols, int pad, const float* act, float eps, cudaStream_t st) {
  constexpr int V = kVec<T>;
  const bool vec = cols % V == 0 && zs % V == 0 && os % V == 0 && is_aligned(z, 16) && is_aligned(out, 16);
  const int nvec = vec ? cols / V : cols;
  // about four vectors per thread
  int nt = ((nvec + 3) / 4 + 31) / 32 * 32;
  if (nt < 128) nt = 128;
  if (nt > 512) nt = 512;
  const size_t smem = (static_cast<size_t>(cols) * sizeof(T) + 15) / 16 * 16;
  if (smem > 200 * 1024) return kUnsupportedShape;
  struct VecTag {};
  struct OneTag {};
  int rc;
  if (vec) {
    rc = opt_in_dynamic_smem<VecTag>(reinterpret_cast<const void*>(&poly_norm_kernel<T, V>), smem);
    if (rc == kOk) poly_norm_kernel<T, V><<<rows, nt, smem, st>>>(static_cast<const T*>(z), zs, static_cast<T*>(out), os, cols, pad, act, eps);
  } else {
    rc = opt_in_dynamic_smem<OneTag>(reinterpret_cast<const void*>(&poly_norm_kernel<T, 1>), smem);
    if (rc == kOk) poly_norm_kernel<T, 1><<<rows, nt, smem, st>>>(static_cast<const T*>(z), zs, static_cast<T*>(out), os, cols, pad, act, eps);
  }
  if (rc != kOk) return rc;
  return cudaGetLastError() == cudaSuccess ? kOk : kLaunchFailed;
}

}  // namespace mvb

static int run_hyper(int dtype, mvb::HyperParams& p, int rows, void* stream) {
  using namespace mvb;
  if (!p.x || !p.y || !p.weight || !p.h || rows < 0 || p.width <= 0 || p.streams <= 0 || p.groups <= 0 || p.width % p.groups != 0)
    return kInvalidArgument;
  if (dtype != kBf16 && dtype != kF32) return kInvalidArgument;
  if (rows == 0) return kOk;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return dtype == kBf16 ? launch_hyper<__nv_bfloat16>(p, rows, st) : launch_hyper<float>(p, rows, st);
}

extern "C" int mvb_hyper_embed_norm(int dtype, const int64_t* ids, const int64_t* positions, const void* table, int64_t vocab,
                                    const void* pos_table, int64_t max_positions, float* x, const float* in_weights, const void* weight,
                                    void* h, int rows, int width, int streams, int groups, float eps, int32_t* dev_status, void* stream) {
  using namespace mvb;
  if (!ids || !positions || !pos_table || vocab <= 0 || max_positions <= 0) return kInvalidArgument;
  HyperParams p{};
  p.x = x; p.y = table; p.y_stride = width; p.ids = ids; p.positions = positions; p.pos_table = pos_table; p.vocab = vocab;
  p.max_positions = max_positions; p.in_w = in_weights; p.weight = weight; p.h = h;
  p.width = width; p.streams = streams; p.groups = groups; p.eps = eps; p.dev_status = dev_status;
  return run_hyper(dtype, p, rows, stream);
}

extern "C" int mvb_hyper_norm(int dtype, float* x, const void* y, int64_t y_row_stride, const float* mix, const float* out_weights,
                              const float* in_weights, const void* weight, void* h, const int32_t* row_ends, int rows, int width,
                              int streams, int groups, float eps, void* stream) {
  using namespace mvb;
  if (!mix || !out_weights) return kInvalidArgument;
  HyperParams p{};
  p.x = x; p.y = y; p.y_stride = y_row_stride; p.mix = mix; p.out_w = out_weights; p.in_w = in_weights; p.weight = weight; p.h = h;
  p.row_ends = row_ends; p.width = width; p.streams = streams; p.groups = groups; p.eps = eps;
  return run_hyper(dtype, p, rows, stream);
}

extern "C" int mvb_poly_norm(int dtype, const void* z, int64_t z_row_stride, void* out, int64_t out_row_stride, int rows, int cols,
                             int out_cols, const float* act, float eps, void* stream) {
  using namespace mvb;
  if (!z || !out || !act || rows < 0 || cols <= 0 || out_cols < cols || (dtype != kBf16 && dtype != kF32)) return kInvalidArgument;
  if (rows == 0) return kOk;
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return dtype == kBf16 ? launch_poly<__nv_bfloat16>(z, z_row_stride, out, out_row_stride, rows, cols, out_cols, act, eps, st)
                        : launch_poly<float>(z, z_row_stride, out, out_row_stride, rows, cols, out_cols, act, eps, st);
}
