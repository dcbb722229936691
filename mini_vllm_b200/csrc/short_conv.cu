// Depthwise causal convolution over a few taps, with bias and, where asked, SiLU, on a packed ragged batch with carried inputs.
//
//   out[t, c] = silu(bias[c] + sum_j w[j, c] u[t - j, c])
//
// The last `copies` channels may also be written a second time, behind the others (for a mixer that rotates one copy in place).
//
// The taps - 1 inputs in front of a step's tokens come from the sequence's state slot ([slots, taps - 1, channels], row
// taps - 1 - d = the input d tokens before the step), zeros before the start of the sequence; afterwards the slot holds the
// last taps - 1 inputs again.  A thread owns four channels and walks a run of tokens with the window in
// registers, so every input is read once.  A step in which every sequence brings one token (cu == nullptr) reads and
// rewrites its slots in the same kernel; a ragged step writes them in a second small kernel, because the tokens that read
// the old inputs and those that leave the new ones may be worked on by different CTAs.
//
// Roofline: HBM, 2 * channels * sizeof(T) bytes per token.
#include "dtype.cuh"
#include "host_util.cuh"
#include "mini_vllm_b200.h"

namespace mvb {

// V elements as they lie in memory
template <class T, int V> struct alignas(sizeof(T) * V) RawVec { T v[V]; };
template <class T, int V> __device__ __forceinline__ void get(const T* p, float (&out)[V]) {
  const RawVec<T, V> r = *reinterpret_cast<const RawVec<T, V>*>(p);
#pragma unroll
  for (int i = 0; i < V; ++i) out[i] = to_f(r.v[i]);
}
template <class T, int V> __device__ __forceinline__ void put(T* p, const float (&in)[V]) {
  RawVec<T, V> r;
#pragma unroll
  for (int i = 0; i < V; ++i) r.v[i] = from_f<T>(in[i]);
  *reinterpret_cast<RawVec<T, V>*>(p) = r;
}

struct ConvParams {
  const void* u; int64_t u_stride;
  const void* w;                 // [taps, channels], row j weighs the input j tokens back
  const void* bias;              // [channels] or nullptr
  void* out; int64_t out_stride;
  void* state;                   // [slots, taps - 1, channels] or nullptr (nothing carried)
  const int32_t* slots;          // [num_seqs]
  int64_t num_slots;
  const int32_t* cu;             // [num_seqs + 1] or nullptr
  const int64_t* positions;      // [tokens]
  int num_seqs, tokens, channels, taps;
  int silu, copies;
  int* dev_status;
};

constexpr int kConvRun = 16;     // tokens a thread walks

__device__ __forceinline__ int64_t conv_slot(const ConvParams& p, int s) {
  if (p.state == nullptr) return -1;
  const int64_t slot = p.slots[s];
  if (slot >= p.num_slots) { report(p.dev_status, kDevBadSlot, s); return -1; }
  return slot;
}

template <class T, int V, int TAPS>
__global__ void __launch_bounds__(128, TAPS <= 4 ? 7 : 1) short_conv_kernel(const ConvParams p) {
  const int c = (blockIdx.y * 128 + threadIdx.x) * V;
  if (c >= p.channels) return;
  const int t_begin = blockIdx.x * (p.cu == nullptr ? 1 : kConvRun);
  const int t_end = p.cu == nullptr ? t_begin + 1 : min(t_begin + kConvRun, p.tokens);
  const T* u = static_cast<const T*>(p.u) + c;
  T* out = static_cast<T*>(p.out) + c;
  const int taps = p.taps, C = p.channels;
  float w[TAPS][V], bias[V];
#pragma unroll
  for (int i = 0; i < V; ++i) bias[i] = 0.f;
  if (p.bias != nullptr) get<T, V>(static_cast<const T*>(p.bias) + c, bias);
#pragma unroll
  for (int j = 0; j < TAPS; ++j) {
#pragma unroll
    for (int i = 0; i < V; ++i) w[j][i] = 0.f;
    if (j < taps) get<T, V>(static_cast<const T*>(p.w) + static_cast<int64_t>(j) * C + c, w[j]);
  }

  float hist[TAPS][V];                                       // hist[j]: the input j tokens back (hist[0]: this token's)
  int s = seq_of_row(p.cu, p.num_seqs, t_begin);
  int begin = p.cu == nullptr ? t_begin : p.cu[s], end = p.cu == nullptr ? t_begin + 1 : p.cu[s + 1];
  bool fill = true;
  for (int t = t_begin; t < t_end;) {
    while (t >= end) {                                       // (a sequence may bring no token)
      ++s; begin = end; end = p.cu[s + 1]; fill = true;
    }
    if (fill) {
      fill = false;
      const int64_t pos = p.positions[t];
      const int64_t slot = conv_slot(p, s);
#pragma unroll
      for (int j = 1; j < TAPS; ++j) {
#pragma unroll
        for (int i = 0; i < V; ++i) hist[j][i] = 0.f;
        if (j >= taps || pos - j < 0) continue;
        if (t - j >= begin) get<T, V>(u + (t - j) * p.u_stride, hist[j]);
        else if (slot >= 0)
          get<T, V>(static_cast<const T*>(p.state) + (slot * (taps - 1) + (taps - 1 - (j - (t - begin)))) * C + c, hist[j]);
      }
    }
    // the rest of this run inside the sequence, B tokens at a time so that B loads are in flight
    constexpr int B = 4;
    const int stop = min(t_end, end);
    for (; t < stop; t += B) {
      RawVec<T, V> in[B];
#pragma unroll
      for (int m = 0; m < B; ++m)
        if (t + m < stop) in[m] = *reinterpret_cast<const RawVec<T, V>*>(u + (t + m) * p.u_stride);
#pragma unroll
      for (int m = 0; m < B; ++m) {
        if (t + m >= stop) break;
        float acc[V];
#pragma unroll
        for (int i = 0; i < V; ++i) { hist[0][i] = to_f(in[m].v[i]); acc[i] = bias[i]; }
#pragma unroll
        for (int j = TAPS - 1; j >= 0; --j)
#pragma unroll
          for (int i = 0; i < V; ++i) acc[i] = fmaf(w[j][i], hist[j][i], acc[i]);
#pragma unroll
        for (int i = 0; i < V; ++i)
          if (p.silu) acc[i] = acc[i] * fast_rcp(1.f + fast_exp2(acc[i] * -1.4426950408889634f));
        put<T, V>(out + (t + m) * p.out_stride, acc);
        if (c >= C - p.copies) put<T, V>(out + (t + m) * p.out_stride + p.copies, acc);
        if (p.cu == nullptr) {                               // the slot's rows are this thread's alone
          const int64_t slot = conv_slot(p, s);
          if (slot >= 0) {
#pragma unroll
            for (int j = 0; j < TAPS; ++j)
              if (j < taps - 1) put<T, V>(static_cast<T*>(p.state) + (slot * (taps - 1) + (taps - 2 - j)) * C + c, hist[j]);
          }
        }
#pragma unroll
        for (int j = TAPS - 1; j > 0; --j)
#pragma unroll
          for (int i = 0; i < V; ++i) hist[j][i] = hist[j - 1][i];
      }
    }
    t = stop;
  }
}

// the slot's new rows: the last taps - 1 inputs of the sequence, some of them possibly from before the step
template <class T, int V, int TAPS>
__global__ void __launch_bounds__(128) conv_state_kernel(const ConvParams p) {
  const int c = (blockIdx.y * 128 + threadIdx.x) * V, s = blockIdx.x;
  if (c >= p.channels) return;
  const int begin = p.cu[s], n = p.cu[s + 1] - begin, taps = p.taps;
  const int64_t slot = conv_slot(p, s);
  if (n <= 0 || slot < 0) return;
  T* st = static_cast<T*>(p.state) + slot * (taps - 1) * p.channels + c;
  const int64_t next = p.positions[begin] + n;               // position of the sequence's next token
  float v[TAPS][V];
#pragma unroll
  for (int d = 1; d < TAPS; ++d) {                           // everything read before anything is written
#pragma unroll
    for (int i = 0; i < V; ++i) v[d][i] = 0.f;
    if (d >= taps || next - d < 0) continue;
    if (n - d >= 0) get<T, V>(static_cast<const T*>(p.u) + (begin + n - d) * p.u_stride + c, v[d]);
    else get<T, V>(st + static_cast<int64_t>(taps - 1 - (d - n)) * p.channels, v[d]);
  }
#pragma unroll
  for (int d = 1; d < TAPS; ++d)
    if (d < taps) put<T, V>(st + static_cast<int64_t>(taps - 1 - d) * p.channels, v[d]);
}

template <class T, int V, int TAPS>
static int launch_conv_t(const ConvParams& p, cudaStream_t st) {
  const unsigned by = (p.channels / V + 127) / 128;
  if (by > 65535) return kUnsupportedShape;
  const dim3 grid(p.cu == nullptr ? p.tokens : (p.tokens + kConvRun - 1) / kConvRun, by);
  short_conv_kernel<T, V, TAPS><<<grid, 128, 0, st>>>(p);
  if (p.cu != nullptr && p.state != nullptr && p.taps > 1) conv_state_kernel<T, V, TAPS><<<dim3(p.num_seqs, by), 128, 0, st>>>(p);
  return cudaGetLastError() == cudaSuccess ? kOk : kLaunchFailed;
}

template <class T>
static int launch_conv(const ConvParams& p, cudaStream_t st) {
  constexpr int V = 4;                                       // (8 bf16 would double the registers and halve the warps)
  const bool vec = p.channels % V == 0 && p.copies % V == 0 && p.u_stride % V == 0 && p.out_stride % V == 0 && is_aligned(p.u, 16) &&
                   is_aligned(p.out, 16) && is_aligned(p.state, 16) && is_aligned(p.w, 16) && is_aligned(p.bias, 16);
  if (p.taps <= 4) return vec ? launch_conv_t<T, V, 4>(p, st) : launch_conv_t<T, 1, 4>(p, st);
  if (p.taps <= 8) return vec ? launch_conv_t<T, V, 8>(p, st) : launch_conv_t<T, 1, 8>(p, st);
  if (p.taps <= 32) return launch_conv_t<T, 1, 32>(p, st);
  return kUnsupportedShape;
}

}  // namespace mvb

extern "C" int mvb_short_conv(int dtype, const void* u, int64_t u_row_stride, const void* weight, const void* bias,
                                   void* out, int64_t out_row_stride, void* state, const int32_t* state_slots,
                                   int64_t num_slots, const int32_t* cu_seqlens_q, const int64_t* positions, int num_seqs,
                                   int num_tokens, int channels, int taps, int silu, int copies, int32_t* dev_status, void* stream) {
  using namespace mvb;
  if (!u || !weight || !out || !positions || num_seqs < 0 || num_tokens < 0 || channels <= 0 || taps <= 0 || copies < 0 || copies > channels) return kInvalidArgument;
  if (state != nullptr && (state_slots == nullptr || num_slots <= 0)) return kInvalidArgument;
  if (cu_seqlens_q == nullptr && num_seqs != num_tokens) return kInvalidArgument;
  if (dtype != kBf16 && dtype != kF32) return kInvalidArgument;
  if (num_tokens == 0 || num_seqs == 0) return kOk;
  const ConvParams p{u, u_row_stride, weight, bias, out, out_row_stride, taps > 1 ? state : nullptr, state_slots, num_slots,
                     cu_seqlens_q, positions, num_seqs, num_tokens, channels, taps, silu, copies, dev_status};
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  return dtype == kBf16 ? launch_conv<__nv_bfloat16>(p, st) : launch_conv<float>(p, st);
}

extern "C" int mvb_short_conv_silu(int dtype, const void* u, int64_t u_row_stride, const void* weight, const void* bias,
                                   void* out, int64_t out_row_stride, void* state, const int32_t* state_slots,
                                   int64_t num_slots, const int32_t* cu_seqlens_q, const int64_t* positions, int num_seqs,
                                   int num_tokens, int channels, int taps, int32_t* dev_status, void* stream) {
  return mvb_short_conv(dtype, u, u_row_stride, weight, bias, out, out_row_stride, state, state_slots, num_slots, cu_seqlens_q, positions,
                        num_seqs, num_tokens, channels, taps, 1, 0, dev_status, stream);
}
