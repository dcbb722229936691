// Entry points of the prefill attention (the kernel itself: prefill_attn.cuh).
#include "prefill_attn.cuh"

// rows of q that one work item covers: the two query tiles of an item are two heads of a GQA group over the same 128
// rows when the group allows it, else two consecutive 128-row tiles of one head (head_dim 128); one tile for head_dim 256
static int prefill_item_rows(int num_q_heads, int num_kv_heads, int head_dim) {
  if (num_q_heads <= 0 || num_kv_heads <= 0 || num_q_heads % num_kv_heads != 0) return mvb::kInvalidArgument;
  if (head_dim == 256) return 128;
  if (head_dim != 128) return mvb::kUnsupportedShape;
  return ((num_q_heads / num_kv_heads) % 2 == 0) ? 128 : 256;
}

static int prefill_attn_impl(const void* q, int64_t q_row_stride, const void* k, int64_t k_row_stride, const void* v,
                             int64_t v_row_stride, int64_t kv_rows, const int32_t* cu_seqlens_q,
                             const int32_t* cu_seqlens_k, const int32_t* block_table, int64_t table_stride,
                             int block_size, int num_seqs, int total_q, int max_seqlen_q, int num_q_heads,
                             int num_kv_heads, int head_dim, float scale, int window_left, void* out,
                             int64_t out_row_stride, const int32_t* items, int num_items, float softcap,
                             float out_scale, const mvb_attn_extras* extras, int32_t* dev_status, void* stream) {
  using namespace mvb;
  if (!(softcap >= 0.f)) return kInvalidArgument;
  if (extras != nullptr && (extras->keep_first < 0 || softcap > 0.f)) return kUnsupportedShape;
  if (!q || !k || !v || !cu_seqlens_q || !cu_seqlens_k || !out) return kInvalidArgument;
  if (num_seqs <= 0 || total_q < 0 || max_seqlen_q < 0 || kv_rows <= 0) return kInvalidArgument;
  if (num_q_heads <= 0 || num_kv_heads <= 0 || num_q_heads % num_kv_heads != 0) return kInvalidArgument;
  if (head_dim != 128 && head_dim != 256) return kUnsupportedShape;
  if (block_table != nullptr && block_size <= 0) return kInvalidArgument;
  if (kv_rows > 0x7fffffffLL || num_seqs > 65535 || num_q_heads > 65535) return kUnsupportedShape;
  if (items != nullptr && num_items < 0) return kInvalidArgument;
  if (total_q == 0 || max_seqlen_q == 0 || (items != nullptr && num_items == 0)) return kOk;
  if ((out_row_stride % 8) != 0 || !is_aligned(out, 16)) return kMisaligned;

  const PrefillOperands op{q, k, v, q_row_stride, k_row_stride, v_row_stride, kv_rows, total_q, num_q_heads, num_kv_heads};

  PrefillParams p;
  p.cu_q = cu_seqlens_q; p.cu_k = cu_seqlens_k; p.block_table = block_table; p.table_stride = table_stride;
  p.block_size = block_size; p.kv_rows = kv_rows; p.num_seqs = num_seqs; p.hq = num_q_heads;
  p.group = num_q_heads / num_kv_heads;
  p.pair_heads = 0;
  const float kLog2e = 1.4426950408889634f;
  const bool cap = softcap > 0.f;
  p.scale_log2 = cap ? 1.f : scale * kLog2e;
  p.cap_in = cap ? 2.f * scale * kLog2e / softcap : 0.f;
  p.cap_log2 = softcap * kLog2e;
  p.out_scale = out_scale;
  p.window_left = window_left;
  p.out = static_cast<__nv_bfloat16*>(out); p.out_stride = out_row_stride;
  p.dev_status = dev_status;
  p.items = items; p.num_items = num_items;
  p.sinks = p.slopes = nullptr; p.head_gate = nullptr; p.gate_stride = 0; p.keep_first = 0;
  if (extras != nullptr) {
    p.sinks = extras->sinks; p.slopes = extras->slopes;
    p.head_gate = static_cast<const __nv_bfloat16*>(extras->head_gate); p.gate_stride = extras->head_gate_row_stride;
    p.keep_first = window_left >= 0 ? extras->keep_first : 0;
    if (p.slopes != nullptr) { p.cap_in = p.scale_log2; p.scale_log2 = 1.f; }      // the bias is added to scaled scores
  }
  cudaStream_t st = static_cast<cudaStream_t>(stream);
  // The list form pays when the grid would be mostly empty indices (a ragged batch).  When the list fills the
  // grid - sequences of about one length - both forms take the items in the same order and the grid form,
  // which reads no list, measured 2-3 % faster: run that one (a complete list gives identical results).
  bool list = false;
  if (items != nullptr) {
    const int rows = prefill_item_rows(num_q_heads, num_kv_heads, head_dim);
    const int64_t grid_items = static_cast<int64_t>(num_seqs) * ((max_seqlen_q + rows - 1) / rows);
    list = static_cast<int64_t>(num_items) * 100 < grid_items * 85;
  }
  if (extras != nullptr) return launch_prefill_ext(op, p, head_dim, list, max_seqlen_q, st);
  if (!cap) return launch_prefill_form<0>(op, p, head_dim, list, max_seqlen_q, st);
  return p.cap_log2 <= 50.f ? launch_prefill_form<1>(op, p, head_dim, list, max_seqlen_q, st)
                            : launch_prefill_form<2>(op, p, head_dim, list, max_seqlen_q, st);
}

extern "C" int mvb_prefill_attn(const void* q, int64_t q_row_stride, const void* k, int64_t k_row_stride,
                                const void* v, int64_t v_row_stride, int64_t kv_rows,
                                const int32_t* cu_seqlens_q, const int32_t* cu_seqlens_k,
                                const int32_t* block_table, int64_t table_stride, int block_size, int num_seqs,
                                int total_q, int max_seqlen_q, int num_q_heads, int num_kv_heads, int head_dim,
                                float scale, int window_left, void* out, int64_t out_row_stride,
                                int32_t* dev_status, void* stream) {
  return prefill_attn_impl(q, q_row_stride, k, k_row_stride, v, v_row_stride, kv_rows, cu_seqlens_q, cu_seqlens_k,
                           block_table, table_stride, block_size, num_seqs, total_q, max_seqlen_q, num_q_heads,
                           num_kv_heads, head_dim, scale, window_left, out, out_row_stride, nullptr, 0, 0.f, 1.f,
                           nullptr, dev_status, stream);
}

extern "C" int mvb_prefill_item_rows(int num_q_heads, int num_kv_heads, int head_dim) {
  return prefill_item_rows(num_q_heads, num_kv_heads, head_dim);
}

extern "C" int mvb_prefill_attn_items(const void* q, int64_t q_row_stride, const void* k, int64_t k_row_stride,
                                      const void* v, int64_t v_row_stride, int64_t kv_rows,
                                      const int32_t* cu_seqlens_q, const int32_t* cu_seqlens_k,
                                      const int32_t* block_table, int64_t table_stride, int block_size, int num_seqs,
                                      int total_q, int max_seqlen_q, int num_q_heads, int num_kv_heads, int head_dim,
                                      float scale, int window_left, void* out, int64_t out_row_stride,
                                      const int32_t* items, int num_items, int32_t* dev_status, void* stream) {
  if (items == nullptr) return mvb::kInvalidArgument;
  return prefill_attn_impl(q, q_row_stride, k, k_row_stride, v, v_row_stride, kv_rows, cu_seqlens_q, cu_seqlens_k,
                           block_table, table_stride, block_size, num_seqs, total_q, max_seqlen_q, num_q_heads,
                           num_kv_heads, head_dim, scale, window_left, out, out_row_stride, items, num_items, 0.f, 1.f,
                           nullptr, dev_status, stream);
}

extern "C" int mvb_prefill_attn_capped(const void* q, int64_t q_row_stride, const void* k, int64_t k_row_stride,
                                       const void* v, int64_t v_row_stride, int64_t kv_rows,
                                       const int32_t* cu_seqlens_q, const int32_t* cu_seqlens_k,
                                       const int32_t* block_table, int64_t table_stride, int block_size, int num_seqs,
                                       int total_q, int max_seqlen_q, int num_q_heads, int num_kv_heads, int head_dim,
                                       float scale, int window_left, void* out, int64_t out_row_stride,
                                       const int32_t* items, int num_items, float softcap, float out_scale,
                                       int32_t* dev_status, void* stream) {
  return prefill_attn_impl(q, q_row_stride, k, k_row_stride, v, v_row_stride, kv_rows, cu_seqlens_q, cu_seqlens_k,
                           block_table, table_stride, block_size, num_seqs, total_q, max_seqlen_q, num_q_heads,
                           num_kv_heads, head_dim, scale, window_left, out, out_row_stride, items, num_items, softcap,
                           out_scale, nullptr, dev_status, stream);
}

extern "C" int mvb_prefill_attn_ext(const void* q, int64_t q_row_stride, const void* k, int64_t k_row_stride, const void* v,
                                    int64_t v_row_stride, int64_t kv_rows, const int32_t* cu_seqlens_q, const int32_t* cu_seqlens_k,
                                    const int32_t* block_table, int64_t table_stride, int block_size, int num_seqs, int total_q,
                                    int max_seqlen_q, int num_q_heads, int num_kv_heads, int head_dim, float scale, int window_left,
                                    void* out, int64_t out_row_stride, const int32_t* items, int num_items, float out_scale,
                                    const mvb_attn_extras* extras, int32_t* dev_status, void* stream) {
  if (extras == nullptr) return mvb::kInvalidArgument;
  return prefill_attn_impl(q, q_row_stride, k, k_row_stride, v, v_row_stride, kv_rows, cu_seqlens_q, cu_seqlens_k, block_table,
                           table_stride, block_size, num_seqs, total_q, max_seqlen_q, num_q_heads, num_kv_heads, head_dim, scale,
                           window_left, out, out_row_stride, items, num_items, 0.f, out_scale, extras, dev_status, stream);
}
