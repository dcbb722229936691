// Attention and rotation for what the tensor-core kernels do not take: fp32 activations, head sizes above 256, more than
// eight query heads per KV head.  Same contracts (paged pool or dense K/V, causal with an optional window and kept first tokens, score
// cap, bias by distance, sinks, head gates, output factor), any head size that is a multiple of 4 and at most 1024.
//
// One warp per (token, query head): a key's scores are a warp-wide dot product, four keys at a time, with an online
// softmax in fp32; K and V rows are read coalesced.  Scores use the accurate tanh / exp.
#include "dtype.cuh"
#include "host_util.cuh"
#include "mini_vllm_b200.h"
#include "rope_any.cuh"

namespace mvb {

struct AnyAttnParams {
  const void* q; int64_t q_stride;
  const void* k; int64_t k_stride;        // token-row strides of dense K / V; of a pool slot with a block table
  const void* v; int64_t v_stride;
  int64_t kv_rows;
  const int32_t* block_table; int64_t table_stride; int table_width, block_size;
  const int32_t* cu_q;                     // nullptr: row t is sequence t
  const int32_t* cu_k;                     // dense K/V only
  const int64_t* positions;
  const int32_t* cache_seqlens;            // nullptr, or: a sequence of length 0 (a padding row) gives zeros
  void* out; int64_t out_stride;
  int num_seqs, tokens, hq, group, d;
  float scale, cap, inv_cap, out_scale;
  int window_left;
  const float* sinks; const float* slopes;  // see mvb_attn_extras
  const void* head_gate; int64_t gate_stride;
  int keep_first;
  int* dev_status;
};

template <class T, int E>                   // E elements of a head per lane
__global__ void __launch_bounds__(128) any_attn_kernel(const AnyAttnParams p) {
  const int64_t w = (static_cast<int64_t>(blockIdx.x) * 128 + threadIdx.x) >> 5;
  const int lane = threadIdx.x & 31;
  const int t = static_cast<int>(w / p.hq), h = static_cast<int>(w % p.hq);
  if (t >= p.tokens) return;
  const int s = seq_of_row(p.cu_q, p.num_seqs, t), kvh = h / p.group;
  const int64_t pos = p.positions[t];
  const bool empty = p.cache_seqlens != nullptr && p.cache_seqlens[s] <= 0;
  float q[E], o[E];
#pragma unroll
  for (int e = 0; e < E; ++e) {
    const int i = e * 32 + lane;
    q[e] = i < p.d ? to_f(static_cast<const T*>(p.q)[t * p.q_stride + static_cast<int64_t>(h) * p.d + i]) : 0.f;
    o[e] = 0.f;
  }
  float m = -INFINITY, l = 0.f;
  if (p.sinks != nullptr) { m = p.sinks[h]; l = 1.f; }        // a key without a value
  const float slope = p.slopes != nullptr ? p.slopes[h] : 0.f;
  const int64_t lo = p.window_left >= 0 && pos > p.window_left ? pos - p.window_left : 0;
  for (int64_t j0 = p.keep_first > 0 ? 0 : lo; j0 <= pos && !empty; j0 += 4) {
    if (j0 >= p.keep_first && j0 < lo) j0 = lo;              // past the kept first tokens: on to the window
    int64_t row[4];
    float x[4];
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      const int64_t j = j0 + u;
      row[u] = -1;
      if (j <= pos && (j >= lo || j < p.keep_first)) {
        if (p.block_table != nullptr) {
          const int64_t col = j / p.block_size;
          const int blk = col < p.table_width ? p.block_table[s * p.table_stride + col] : -1;
          row[u] = blk < 0 ? -1 : static_cast<int64_t>(blk) * p.block_size + j % p.block_size;
        } else {
          row[u] = p.cu_k[s] + j;
        }
        if (row[u] < 0 || row[u] >= p.kv_rows) {
          if (lane == 0) report(p.dev_status, kDevBadBlock, s);
          row[u] = -1;
        }
      }
      float dot = 0.f;
      if (row[u] >= 0) {
        const T* kr = static_cast<const T*>(p.k) + row[u] * p.k_stride + static_cast<int64_t>(kvh) * p.d;
#pragma unroll
        for (int e = 0; e < E; ++e) {
          const int i = e * 32 + lane;
          if (i < p.d) dot = fmaf(q[e], to_f(kr[i]), dot);
        }
      }
      x[u] = dot;
    }
#pragma unroll
    for (int u = 0; u < 4; ++u) {
#pragma unroll
      for (int off = 16; off > 0; off >>= 1) x[u] += __shfl_xor_sync(0xffffffffu, x[u], off);
      x[u] *= p.scale;
      if (p.cap > 0.f) x[u] = p.cap * tanhf(x[u] * p.inv_cap);
      x[u] -= slope * static_cast<float>(pos - (j0 + u));
      if (row[u] < 0) x[u] = -INFINITY;
    }
    const float mn = fmaxf(fmaxf(fmaxf(x[0], x[1]), fmaxf(x[2], x[3])), m);
    if (mn == -INFINITY) continue;
    const float alpha = expf(m - mn);
    l *= alpha;
#pragma unroll
    for (int e = 0; e < E; ++e) o[e] *= alpha;
#pragma unroll
    for (int u = 0; u < 4; ++u) {
      if (row[u] < 0) continue;
      const float pr = expf(x[u] - mn);
      l += pr;
      const T* vr = static_cast<const T*>(p.v) + row[u] * p.v_stride + static_cast<int64_t>(kvh) * p.d;
#pragma unroll
      for (int e = 0; e < E; ++e) {
        const int i = e * 32 + lane;
        if (i < p.d) o[e] = fmaf(pr, to_f(vr[i]), o[e]);
      }
    }
    m = mn;
  }
  float inv = l > 0.f ? p.out_scale / l : 0.f;
  if (p.head_gate != nullptr) inv *= sigmoid_f(to_f(static_cast<const T*>(p.head_gate)[t * p.gate_stride + h]));
#pragma unroll
  for (int e = 0; e < E; ++e) {
    const int i = e * 32 + lane;
    if (i < p.d) static_cast<T*>(p.out)[t * p.out_stride + static_cast<int64_t>(h) * p.d + i] = from_f<T>(o[e] * inv);
  }
}

template <class T>
static int launch_any_attn(const AnyAttnParams& p, cudaStream_t st) {
  const int64_t blocks = (static_cast<int64_t>(p.tokens) * p.hq * 32 + 127) / 128;
  if (blocks > 0x7fffffffLL) return kUnsupportedShape;
  const unsigned g = static_cast<unsigned>(blocks);
  if (p.d <= 128) any_attn_kernel<T, 4><<<g, 128, 0, st>>>(p);
  else if (p.d <= 256) any_attn_kernel<T, 8><<<g, 128, 0, st>>>(p);
  else if (p.d <= 512) any_attn_kernel<T, 16><<<g, 128, 0, st>>>(p);
  else if (p.d <= 1024) any_attn_kernel<T, 32><<<g, 128, 0, st>>>(p);
  else return kUnsupportedShape;
  return cudaGetLastError() == cudaSuccess ? kOk : kLaunchFailed;
}

// fp32 form of the rotation + cache write: element i < d/2 of a head pairs with i + d/2, angles from the table
// [max_pos, d] = cos | sin; V is copied.  One thread per pair.
struct RopeF32Params {
  float* q; int64_t q_stride; float* k; int64_t k_stride; const float* v; int64_t v_stride;
  const int64_t* positions; const float* cos_sin; int64_t max_pos; const int32_t* slot_mapping;
  float *k_cache, *v_cache; int64_t num_slots;
  int tokens, hq, hkv, d, k_in_place;
  int* dev_status;
};

__global__ void __launch_bounds__(256) rope_kv_f32_kernel(const RopeF32Params p) {
  const int half = p.d / 2, per_tok = (p.hq + 2 * p.hkv) * half;
  const int64_t i = static_cast<int64_t>(blockIdx.x) * 256 + threadIdx.x;
  const int64_t t = i / per_tok;
  if (t >= p.tokens) return;
  const int r = static_cast<int>(i % per_tok), head = r / half, j = r % half;
  int64_t slot = p.slot_mapping != nullptr ? p.slot_mapping[t] : -1;
  if (slot >= p.num_slots) { report(p.dev_status, kDevBadSlot, static_cast<int>(t)); slot = -1; }
  if (head >= p.hq + p.hkv) {                                       // V
    const int vh = head - p.hq - p.hkv;
    if (slot < 0) return;
    const float* src = p.v + t * p.v_stride + static_cast<int64_t>(vh) * p.d;
    float* dst = p.v_cache + (slot * p.hkv + vh) * p.d;
    dst[j] = src[j]; dst[j + half] = src[j + half];
    return;
  }
  const bool is_q = head < p.hq;
  float* row = is_q ? p.q + t * p.q_stride + static_cast<int64_t>(head) * p.d : p.k + t * p.k_stride + static_cast<int64_t>(head - p.hq) * p.d;
  const int64_t pos = p.positions[t];
  if (pos < 0 || pos >= p.max_pos) { report(p.dev_status, kDevBadPosition, static_cast<int>(t)); return; }
  const float c = p.cos_sin[pos * p.d + j], s = p.cos_sin[pos * p.d + half + j];
  const float a = row[j], b = row[j + half];
  const float lo = a * c - b * s, hi = b * c + a * s;
  if (is_q || p.k_in_place) { row[j] = lo; row[j + half] = hi; }
  if (!is_q && slot >= 0) {
    float* dst = p.k_cache + (slot * p.hkv + head - p.hq) * p.d;
    dst[j] = lo; dst[j + half] = hi;
  }
}

// The same with any pairing size and a norm behind it: a head is rotated (cos_sin may be nullptr) and, with norm_dim > 0, divided by the
// root mean square of its norm_dim used coordinates (the others are zero padding).  One warp per (token, head), the head in registers;
// any even size up to 1024, either dtype.  v may be nullptr with hkv = 0 (only q is turned).
template <class T, int E>                   // E pairs per lane
__global__ void __launch_bounds__(128) rope_any_kernel(const RopeAnyParams p) {
  const int64_t w = (static_cast<int64_t>(blockIdx.x) * 128 + threadIdx.x) >> 5;
  const int lane = threadIdx.x & 31, heads = p.hq + 2 * p.hkv, half = p.d / 2;
  const int64_t t = w / heads;
  const int head = static_cast<int>(w % heads);
  if (t >= p.tokens) return;
  int64_t slot = p.slot_mapping != nullptr ? p.slot_mapping[t] : -1;
  if (slot >= p.num_slots) { if (lane == 0) report(p.dev_status, kDevBadSlot, static_cast<int>(t)); slot = -1; }
  if (head >= p.hq + p.hkv) {                                       // V
    const int vh = head - p.hq - p.hkv;
    if (slot < 0) return;
    const T* src = static_cast<const T*>(p.v) + t * p.v_stride + static_cast<int64_t>(vh) * p.d;
    T* dst = static_cast<T*>(p.v_cache) + (slot * p.hkv + vh) * p.d;
    for (int i = lane; i < p.d; i += 32) dst[i] = src[i];
    return;
  }
  const bool is_q = head < p.hq;
  T* row = is_q ? static_cast<T*>(p.q) + t * p.q_stride + static_cast<int64_t>(head) * p.d
                : static_cast<T*>(p.k) + t * p.k_stride + static_cast<int64_t>(head - p.hq) * p.d;
  const int64_t pos = p.cos_sin != nullptr ? p.positions[t] : 0;
  if (p.cos_sin != nullptr && (pos < 0 || pos >= p.max_pos)) {
    if (lane == 0) report(p.dev_status, kDevBadPosition, static_cast<int>(t));
    return;
  }
  float lo[E], hi[E], ss = 0.f;
#pragma unroll
  for (int e = 0; e < E; ++e) {
    const int i = e * 32 + lane;
    lo[e] = hi[e] = 0.f;
    if (i >= half) continue;
    const float a = to_f(row[i]), b = to_f(row[i + half]);
    const float c = p.cos_sin != nullptr ? p.cos_sin[pos * p.d + i] : 1.f, s = p.cos_sin != nullptr ? p.cos_sin[pos * p.d + half + i] : 0.f;
    lo[e] = a * c - b * s;
    hi[e] = b * c + a * s;
    ss += lo[e] * lo[e] + hi[e] * hi[e];
  }
  float r = 1.f;
  if (p.norm_dim > 0) {
#pragma unroll
    for (int off = 16; off > 0; off >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, off);
    r = 1.f / sqrtf(ss / static_cast<float>(p.norm_dim) + p.eps);
  }
  T* dst = !is_q && slot >= 0 ? static_cast<T*>(p.k_cache) + (slot * p.hkv + head - p.hq) * p.d : nullptr;
#pragma unroll
  for (int e = 0; e < E; ++e) {
    const int i = e * 32 + lane;
    if (i >= half) continue;
    const T x = from_f<T>(lo[e] * r), y = from_f<T>(hi[e] * r);
    if (is_q || p.k_in_place) { row[i] = x; row[i + half] = y; }
    if (dst != nullptr) { dst[i] = x; dst[i + half] = y; }
  }
}

template <class T>
int launch_rope_any(const RopeAnyParams& p, cudaStream_t st) {
  const int64_t blocks = (static_cast<int64_t>(p.tokens) * (p.hq + 2 * p.hkv) * 32 + 127) / 128;
  if (blocks > 0x7fffffffLL || p.d % 2 != 0) return kUnsupportedShape;
  const unsigned g = static_cast<unsigned>(blocks);
  if (p.d <= 128) rope_any_kernel<T, 2><<<g, 128, 0, st>>>(p);
  else if (p.d <= 256) rope_any_kernel<T, 4><<<g, 128, 0, st>>>(p);
  else if (p.d <= 1024) rope_any_kernel<T, 16><<<g, 128, 0, st>>>(p);
  else return kUnsupportedShape;
  return cudaGetLastError() == cudaSuccess ? kOk : kLaunchFailed;
}

}  // namespace mvb

extern "C" int mvb_any_attn_ext(int dtype, const void* q, int64_t q_row_stride, const void* k, int64_t k_row_stride, const void* v,
                            int64_t v_row_stride, int64_t kv_rows, const int32_t* block_table, int64_t table_stride,
                            int table_width, int block_size, const int32_t* cu_seqlens_q, const int32_t* cu_seqlens_k,
                            const int64_t* positions, const int32_t* cache_seqlens, int num_seqs, int num_tokens,
                            int num_q_heads, int num_kv_heads, int head_dim, float scale, int window_left, float softcap,
                            float out_scale, const mvb_attn_extras* extras, void* out, int64_t out_row_stride, int32_t* dev_status, void* stream) {
  using namespace mvb;
  if (!q || !k || !v || !positions || !out || num_seqs < 0 || num_tokens < 0 || kv_rows <= 0) return kInvalidArgument;
  if (num_q_heads <= 0 || num_kv_heads <= 0 || num_q_heads % num_kv_heads != 0 || head_dim <= 0) return kInvalidArgument;
  if (extras != nullptr && extras->keep_first < 0) return kInvalidArgument;
  if (!(softcap >= 0.f) || (dtype != kBf16 && dtype != kF32)) return kInvalidArgument;
  if (block_table != nullptr ? (block_size <= 0 || table_width <= 0) : cu_seqlens_k == nullptr) return kInvalidArgument;
  if (cu_seqlens_q == nullptr && num_seqs != num_tokens) return kInvalidArgument;
  if (num_tokens == 0 || num_seqs == 0) return kOk;
  const AnyAttnParams p{q, q_row_stride, k, k_row_stride, v, v_row_stride, kv_rows, block_table, table_stride, table_width,
                        block_size, cu_seqlens_q, cu_seqlens_k, positions, cache_seqlens, out, out_row_stride, num_seqs,
                        num_tokens, num_q_heads, num_q_heads / num_kv_heads, head_dim, scale, softcap,
                        softcap > 0.f ? 1.f / softcap : 0.f, out_scale, window_left, extras ? extras->sinks : nullptr,
                        extras ? extras->slopes : nullptr, extras ? extras->head_gate : nullptr,
                        extras ? extras->head_gate_row_stride : 0, extras && window_left >= 0 ? extras->keep_first : 0, dev_status};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return dtype == kBf16 ? launch_any_attn<__nv_bfloat16>(p, st) : launch_any_attn<float>(p, st);
}

extern "C" int mvb_any_attn(int dtype, const void* q, int64_t q_row_stride, const void* k, int64_t k_row_stride, const void* v,
                            int64_t v_row_stride, int64_t kv_rows, const int32_t* block_table, int64_t table_stride,
                            int table_width, int block_size, const int32_t* cu_seqlens_q, const int32_t* cu_seqlens_k,
                            const int64_t* positions, const int32_t* cache_seqlens, int num_seqs, int num_tokens,
                            int num_q_heads, int num_kv_heads, int head_dim, float scale, int window_left, float softcap,
                            float out_scale, void* out, int64_t out_row_stride, int32_t* dev_status, void* stream) {
  return mvb_any_attn_ext(dtype, q, q_row_stride, k, k_row_stride, v, v_row_stride, kv_rows, block_table, table_stride, table_width,
                          block_size, cu_seqlens_q, cu_seqlens_k, positions, cache_seqlens, num_seqs, num_tokens, num_q_heads,
                          num_kv_heads, head_dim, scale, window_left, softcap, out_scale, nullptr, out, out_row_stride, dev_status, stream);
}

extern "C" int mvb_rope_kv_write_f32(float* q, int64_t q_row_stride, float* k, int64_t k_row_stride, const float* v,
                                     int64_t v_row_stride, const int64_t* positions, const float* cos_sin, int64_t max_pos,
                                     const int32_t* slot_mapping, float* k_cache, float* v_cache, int64_t num_slots,
                                     int num_tokens, int num_q_heads, int num_kv_heads, int head_dim, int k_in_place,
                                     int32_t* dev_status, void* stream) {
  using namespace mvb;
  if (!q || !k || !v || !positions || !cos_sin || num_tokens < 0 || num_q_heads <= 0 || num_kv_heads <= 0 || head_dim <= 0)
    return kInvalidArgument;
  if (head_dim % 2 != 0) return kUnsupportedShape;
  if (slot_mapping != nullptr && (k_cache == nullptr || v_cache == nullptr || num_slots <= 0)) return kInvalidArgument;
  if (num_tokens == 0) return kOk;
  const RopeF32Params p{q, q_row_stride, k, k_row_stride, v, v_row_stride, positions, cos_sin, max_pos, slot_mapping,
                        k_cache, v_cache, num_slots, num_tokens, num_q_heads, num_kv_heads, head_dim, k_in_place, dev_status};
  const int64_t threads = static_cast<int64_t>(num_tokens) * (num_q_heads + 2 * num_kv_heads) * (head_dim / 2);
  const int64_t blocks = (threads + 255) / 256;
  if (blocks > 0x7fffffffLL) return kUnsupportedShape;
  rope_kv_f32_kernel<<<static_cast<unsigned>(blocks), 256, 0, static_cast<cudaStream_t>(stream)>>>(p);
  return cudaGetLastError() == cudaSuccess ? kOk : kLaunchFailed;
}

extern "C" int mvb_rope_norm_kv_write(int dtype, void* q, int64_t q_row_stride, void* k, int64_t k_row_stride, const void* v,
                                      int64_t v_row_stride, const int64_t* positions, const float* cos_sin, int64_t max_pos,
                                      const int32_t* slot_mapping, void* k_cache, void* v_cache, int64_t num_slots, int num_tokens,
                                      int num_q_heads, int num_kv_heads, int head_dim, int k_in_place, int norm_dim, float eps,
                                      int32_t* dev_status, void* stream) {
  using namespace mvb;
  if (!q || num_tokens < 0 || num_q_heads <= 0 || num_kv_heads < 0 || head_dim <= 0 || norm_dim < 0) return kInvalidArgument;
  if (num_kv_heads > 0 && (!k || !v)) return kInvalidArgument;
  if (dtype != kBf16 && dtype != kF32) return kInvalidArgument;
  if (cos_sin != nullptr && positions == nullptr) return kInvalidArgument;
  if (num_kv_heads == 0) slot_mapping = nullptr;
  if (slot_mapping != nullptr && (k_cache == nullptr || v_cache == nullptr || num_slots <= 0)) return kInvalidArgument;
  if (num_tokens == 0) return kOk;
  const RopeAnyParams p{q, q_row_stride, k, k_row_stride, v, v_row_stride, positions, cos_sin, max_pos, slot_mapping, k_cache, v_cache,
                        num_slots, num_tokens, num_q_heads, num_kv_heads, head_dim, k_in_place, norm_dim, eps, dev_status};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  if (dtype == kF32) return launch_rope_any<float>(p, st);
  const int rc = rope_norm_bf16(p, st);
  return rc != kUnsupportedShape ? rc : launch_rope_any<__nv_bfloat16>(p, st);
}
