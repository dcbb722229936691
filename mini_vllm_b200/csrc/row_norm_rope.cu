// Norm over the whole row of queries (and of keys), rotation and paged KV-cache write in one pass, with an optional norm of every
// value head.
//
//   q <- rotate(q / rms(q) * wq)     the root mean square over the token's heads * dim used coordinates, before they are heads
//   k <- rotate(k / rms(k) * wk)     likewise
//   v <- v / rms(v)                  per head over v_dim used coordinates, no weight (v_dim 0: v as it is)
//
// Without weights q and k are rotated only.
//
// q is updated in place, k and v go to the cache slot and, where asked, back to their place.  What a head is padded with is zero and
// its weights are too; rotated pairs are (i, i + D/2).  fp32 throughout, one rounding at the end.
//
// row_rope_kernel (bf16, heads of 128 or 256): a CTA per token; a task is a 16-byte chunk of the first half of a head with its partner
// in the second half, held in registers from the sums to the store, so everything is read and written once.
// row_rope_any_kernel: any even head size and dtype, a warp per head, the row read twice (the second time from L1/L2).
//
// Roofline: HBM, (Hq + 2 Hkv) * D * 2 bytes read and written per token.
#include "chunk_common.cuh"
#include "host_util.cuh"
#include "mini_vllm_b200.h"

namespace mvb {

struct RowRopeParams {
  void* q; int64_t q_stride; void* k; int64_t k_stride; void* v; int64_t v_stride;
  const void *q_weight, *k_weight;             // [heads * d], or both nullptr
  int q_dim, k_dim, v_dim;                     // used coordinates: of the rows, of a value head
  const int64_t* positions; const float* cos_sin; int64_t max_pos; const int32_t* slot_mapping;
  void *k_cache, *v_cache; int64_t num_slots;
  int tokens, hq, hkv, d, kv_in_place;
  float eps;
  int* dev_status;
};

__device__ __forceinline__ int64_t row_slot(const RowRopeParams& p, int t) {
  int64_t slot = p.slot_mapping != nullptr ? p.slot_mapping[t] : -1;
  if (slot >= p.num_slots || slot < -1) {
    if (threadIdx.x == 0) report(p.dev_status, kDevBadSlot, t);
    slot = -1;
  }
  return slot;
}
// sums of a and b over the block
__device__ __forceinline__ void block_sums(float& a, float& b) {
  __shared__ float part[2][32];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
  a = warp_sum(a); b = warp_sum(b);
  if (lane == 0) { part[0][warp] = a; part[1][warp] = b; }
  __syncthreads();
  a = warp_sum(lane < warps ? part[0][lane] : 0.f);
  b = warp_sum(lane < warps ? part[1][lane] : 0.f);
}

// PPH: chunk pairs per head (8: 128, 16: 256); heads of q, then k, then v
template <int ITEMS, int PPH>
__global__ void __launch_bounds__(512) row_rope_kernel(const RowRopeParams p) {
  constexpr int D = PPH * 16;
  const int t = blockIdx.x, nt = blockDim.x, q_tasks = p.hq * PPH, k_end = q_tasks + p.hkv * PPH, tasks = k_end + p.hkv * PPH;
  __nv_bfloat16 *q = static_cast<__nv_bfloat16*>(p.q) + t * p.q_stride, *k = static_cast<__nv_bfloat16*>(p.k) + t * p.k_stride,
                *v = static_cast<__nv_bfloat16*>(p.v) + t * p.v_stride;
  // chunk c of a head lies at 8 c and D/2 + 8 c
  auto place = [&](int task) {
    __nv_bfloat16* row = task < q_tasks ? q : task < k_end ? k : v;
    const int local = task < q_tasks ? task : task < k_end ? task - q_tasks : task - k_end;
    return row + local / PPH * D + local % PPH * 8;
  };
  const int64_t slot = row_slot(p, t), pos = p.cos_sin != nullptr ? p.positions[t] : 0;
  uint4 lo[ITEMS], hi[ITEMS];
#pragma unroll
  for (int j = 0; j < ITEMS; ++j) {
    const int task = threadIdx.x + j * nt;
    lo[j] = hi[j] = make_uint4(0u, 0u, 0u, 0u);
    if (task < tasks) {
      const __nv_bfloat16* at = place(task);
      lo[j] = *reinterpret_cast<const uint4*>(at);
      hi[j] = *reinterpret_cast<const uint4*>(at + D / 2);
    }
  }
  if (p.cos_sin != nullptr && (pos < 0 || pos >= p.max_pos)) {                   // (the whole block)
    if (threadIdx.x == 0) report(p.dev_status, kDevBadPosition, t);
    return;
  }
  float qs = 0.f, ks = 0.f, own[ITEMS];
#pragma unroll
  for (int j = 0; j < ITEMS; ++j) {
    const int task = threadIdx.x + j * nt;
    const uint32_t w[8] = {lo[j].x, lo[j].y, lo[j].z, lo[j].w, hi[j].x, hi[j].y, hi[j].z, hi[j].w};
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) { const float a = bf16_lo(w[i]), b = bf16_hi(w[i]); ss += a * a + b * b; }
    if (task < q_tasks) qs += ss; else if (task < k_end) ks += ss;
    // (a head's chunks are PPH neighbouring lanes)
#pragma unroll
    for (int off = 1; off < PPH; off <<= 1) ss += __shfl_xor_sync(0xffffffffu, ss, off);
    own[j] = ss;
  }
  block_sums(qs, ks);
  const float q_r = 1.f / sqrtf(qs / static_cast<float>(p.q_dim) + p.eps), k_r = 1.f / sqrtf(ks / static_cast<float>(p.k_dim) + p.eps);
  const int c = threadIdx.x % PPH * 8;                                           // (nt is a multiple of PPH: the same in every task)
  float cs[8], sn[8];
#pragma unroll
  for (int i = 0; i < 8; ++i) { cs[i] = 1.f; sn[i] = 0.f; }
  if (p.cos_sin != nullptr) {
    const float* tab = p.cos_sin + pos * D + c;
#pragma unroll
    for (int i = 0; i < 8; i += 4) {
      *reinterpret_cast<float4*>(cs + i) = *reinterpret_cast<const float4*>(tab + i);
      *reinterpret_cast<float4*>(sn + i) = *reinterpret_cast<const float4*>(tab + D / 2 + i);
    }
  }
#pragma unroll
  for (int j = 0; j < ITEMS; ++j) {
    const int task = threadIdx.x + j * nt;
    if (task >= tasks) continue;
    uint32_t *a = reinterpret_cast<uint32_t*>(&lo[j]), *b = reinterpret_cast<uint32_t*>(&hi[j]);
    const bool is_q = task < q_tasks, is_v = task >= k_end;
    if (is_v) {
      if (p.v_dim > 0) {
        const float r = 1.f / sqrtf(own[j] / static_cast<float>(p.v_dim) + p.eps);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
          a[i] = pack_bf16(bf16_lo(a[i]) * r, bf16_hi(a[i]) * r);
          b[i] = pack_bf16(bf16_lo(b[i]) * r, bf16_hi(b[i]) * r);
        }
      }
    } else {
      const int local = is_q ? task : task - q_tasks;
      const __nv_bfloat16* w = static_cast<const __nv_bfloat16*>(is_q ? p.q_weight : p.k_weight) + local / PPH * D + c;
      constexpr uint32_t ONES = 0x3f803f80u;
      uint4 wl = make_uint4(ONES, ONES, ONES, ONES), wh = wl;
      if (p.q_weight != nullptr) { wl = *reinterpret_cast<const uint4*>(w); wh = *reinterpret_cast<const uint4*>(w + D / 2); }
      const uint32_t *wa = reinterpret_cast<const uint32_t*>(&wl), *wb = reinterpret_cast<const uint32_t*>(&wh);
      const float r = p.q_weight == nullptr ? 1.f : is_q ? q_r : k_r;
#pragma unroll
      for (int i = 0; i < 4; ++i) {
        const float u0 = bf16_lo(a[i]) * r * bf16_lo(wa[i]), u1 = bf16_hi(a[i]) * r * bf16_hi(wa[i]);
        const float v0 = bf16_lo(b[i]) * r * bf16_lo(wb[i]), v1 = bf16_hi(b[i]) * r * bf16_hi(wb[i]);
        a[i] = pack_bf16(u0 * cs[2 * i] - v0 * sn[2 * i], u1 * cs[2 * i + 1] - v1 * sn[2 * i + 1]);
        b[i] = pack_bf16(v0 * cs[2 * i] + u0 * sn[2 * i], v1 * cs[2 * i + 1] + u1 * sn[2 * i + 1]);
      }
    }
    if (is_q || p.kv_in_place) {
      __nv_bfloat16* at = place(task);
      *reinterpret_cast<uint4*>(at) = lo[j];
      *reinterpret_cast<uint4*>(at + D / 2) = hi[j];
    }
    if (!is_q && slot >= 0) {
      const int local = is_v ? task - k_end : task - q_tasks;
      __nv_bfloat16* at = static_cast<__nv_bfloat16*>(is_v ? p.v_cache : p.k_cache) + (slot * p.hkv + local / PPH) * D + c;
      *reinterpret_cast<uint4*>(at) = lo[j];
      *reinterpret_cast<uint4*>(at + D / 2) = hi[j];
    }
  }
}

template <class T>
__global__ void __launch_bounds__(256) row_rope_any_kernel(const RowRopeParams p) {
  const int t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, half = p.d / 2;
  T *q = static_cast<T*>(p.q) + t * p.q_stride, *k = static_cast<T*>(p.k) + t * p.k_stride, *v = static_cast<T*>(p.v) + t * p.v_stride;
  const int64_t slot = row_slot(p, t), pos = p.cos_sin != nullptr ? p.positions[t] : 0;
  if (p.cos_sin != nullptr && (pos < 0 || pos >= p.max_pos)) {
    if (threadIdx.x == 0) report(p.dev_status, kDevBadPosition, t);
    return;
  }
  float qs = 0.f, ks = 0.f;
  for (int i = threadIdx.x; i < p.hq * p.d; i += 256) { const float x = to_f(q[i]); qs += x * x; }
  for (int i = threadIdx.x; i < p.hkv * p.d; i += 256) { const float x = to_f(k[i]); ks += x * x; }
  block_sums(qs, ks);                            // (a barrier: nothing is overwritten before everyone has read)
  const float q_r = 1.f / sqrtf(qs / static_cast<float>(p.q_dim) + p.eps), k_r = 1.f / sqrtf(ks / static_cast<float>(p.k_dim) + p.eps);
  for (int head = warp; head < p.hq + 2 * p.hkv; head += 8) {
    const bool is_q = head < p.hq, is_v = head >= p.hq + p.hkv;
    const int local = is_q ? head : is_v ? head - p.hq - p.hkv : head - p.hq;
    T* row = (is_q ? q : is_v ? v : k) + static_cast<int64_t>(local) * p.d;
    T* cache = !is_q && slot >= 0 ? static_cast<T*>(is_v ? p.v_cache : p.k_cache) + (slot * p.hkv + local) * p.d : nullptr;
    const bool back = is_q || p.kv_in_place;
    if (is_v) {
      float r = 1.f;
      if (p.v_dim > 0) {
        float ss = 0.f;
        for (int i = lane; i < p.d; i += 32) { const float x = to_f(row[i]); ss += x * x; }
        r = 1.f / sqrtf(warp_sum(ss) / static_cast<float>(p.v_dim) + p.eps);
      }
      for (int i = lane; i < p.d; i += 32) {
        const T x = p.v_dim > 0 ? from_f<T>(to_f(row[i]) * r) : row[i];
        if (back) row[i] = x;
        if (cache != nullptr) cache[i] = x;
      }
      continue;
    }
    const T* w = static_cast<const T*>(is_q ? p.q_weight : p.k_weight) + static_cast<int64_t>(local) * p.d;
    const bool plain = p.q_weight == nullptr;
    const float r = plain ? 1.f : is_q ? q_r : k_r;
    for (int i = lane; i < half; i += 32) {
      const float a = to_f(row[i]) * r * (plain ? 1.f : to_f(w[i])), b = to_f(row[i + half]) * r * (plain ? 1.f : to_f(w[i + half]));
      const float cs = p.cos_sin != nullptr ? p.cos_sin[pos * p.d + i] : 1.f, sn = p.cos_sin != nullptr ? p.cos_sin[pos * p.d + half + i] : 0.f;
      const T x = from_f<T>(a * cs - b * sn), y = from_f<T>(b * cs + a * sn);
      if (back) { row[i] = x; row[i + half] = y; }
      if (cache != nullptr) { cache[i] = x; cache[i + half] = y; }
    }
  }
}

template <int PPH>
static int launch_row_rope(const RowRopeParams& p, cudaStream_t st) {
  const int tasks = (p.hq + 2 * p.hkv) * PPH;
  // many tokens: small blocks with more loads in flight per thread; few: the shortest path for each
  const int items = p.tokens >= 1024 ? (tasks <= 128 ? 2 : 4) : tasks <= 384 ? 1 : tasks <= 1024 ? 2 : 4;
  const int nt = ((tasks + items - 1) / items + 31) / 32 * 32;
  if (nt > 512) return kUnsupportedShape;
  if (items == 1) row_rope_kernel<1, PPH><<<p.tokens, nt, 0, st>>>(p);
  else if (items == 2) row_rope_kernel<2, PPH><<<p.tokens, nt, 0, st>>>(p);
  else row_rope_kernel<4, PPH><<<p.tokens, nt, 0, st>>>(p);
  return cudaGetLastError() == cudaSuccess ? kOk : kLaunchFailed;
}

}  // namespace mvb

extern "C" int mvb_row_norm_rope_kv_write(int dtype, void* q, int64_t q_row_stride, void* k, int64_t k_row_stride, void* v,
                                          int64_t v_row_stride, const void* q_weight, const void* k_weight, int q_dim, int k_dim, int v_dim,
                                          float eps, const int64_t* positions, const float* cos_sin, int64_t max_pos,
                                          const int32_t* slot_mapping, void* k_cache, void* v_cache, int64_t num_slots, int num_tokens,
                                          int num_q_heads, int num_kv_heads, int head_dim, int kv_in_place, int32_t* dev_status,
                                          void* stream) {
  using namespace mvb;
  if (!q || !k || !v || (q_weight == nullptr) != (k_weight == nullptr) || num_tokens < 0 || num_q_heads <= 0 || num_kv_heads <= 0 || head_dim <= 0) return kInvalidArgument;
  if (q_dim <= 0 || k_dim <= 0 || v_dim < 0 || (dtype != kBf16 && dtype != kF32)) return kInvalidArgument;
  if (cos_sin != nullptr && positions == nullptr) return kInvalidArgument;
  if (slot_mapping != nullptr && (k_cache == nullptr || v_cache == nullptr || num_slots <= 0)) return kInvalidArgument;
  if (head_dim % 2 != 0) return kUnsupportedShape;
  if (num_tokens == 0) return kOk;
  const RowRopeParams p{q, q_row_stride, k, k_row_stride, v, v_row_stride, q_weight, k_weight, q_dim, k_dim, v_dim, positions, cos_sin,
                        max_pos, slot_mapping, k_cache, v_cache, num_slots, num_tokens, num_q_heads, num_kv_heads, head_dim, kv_in_place,
                        eps, dev_status};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  const bool vec = q_row_stride % 8 == 0 && k_row_stride % 8 == 0 && v_row_stride % 8 == 0 && is_aligned(q, 16) && is_aligned(k, 16) &&
                   is_aligned(v, 16) && is_aligned(q_weight, 16) && is_aligned(k_weight, 16) && is_aligned(k_cache, 16) &&
                   is_aligned(v_cache, 16) && is_aligned(cos_sin, 16);
  int rc = kUnsupportedShape;
  if (dtype == kBf16 && vec && head_dim == 128) rc = launch_row_rope<8>(p, st);
  else if (dtype == kBf16 && vec && head_dim == 256) rc = launch_row_rope<16>(p, st);
  if (rc != kUnsupportedShape) return rc;
  if (dtype == kBf16) row_rope_any_kernel<__nv_bfloat16><<<num_tokens, 256, 0, st>>>(p);
  else row_rope_any_kernel<float><<<num_tokens, 256, 0, st>>>(p);
  return cudaGetLastError() == cudaSuccess ? kOk : kLaunchFailed;
}
