// Arguments of the rotation with a norm behind it, shared by its two kernels: head by head for any size and dtype (any_attn.cu), by
// 16-byte chunks for the bf16 head sizes of the tensor-core kernels (rope_kv_write.cu).
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

namespace mvb {

struct RopeAnyParams {
  void* q; int64_t q_stride; void* k; int64_t k_stride; const void* v; int64_t v_stride;
  const int64_t* positions; const float* cos_sin; int64_t max_pos; const int32_t* slot_mapping;
  void *k_cache, *v_cache; int64_t num_slots;
  int tokens, hq, hkv, d, k_in_place, norm_dim;
  float eps;
  int* dev_status;
};

int rope_norm_bf16(const RopeAnyParams& p, cudaStream_t st);          // kUnsupportedShape: not a size or an alignment of that kernel

}  // namespace mvb
