/*
 * C ABI of libmini_vllm_b200.so: the B200 (sm_100a) kernels for mini-vllm's ragged
 * continuous-batching attention path.
 *
 * Conventions for every entry point
 *   - All data pointers are DEVICE pointers owned by the caller (typically PyTorch tensors
 *     kept alive until the stream reaches the launch).  Nothing here allocates, frees,
 *     synchronises or throws; work is enqueued on `stream` (a cudaStream_t passed as void*).
 *   - Return value: 0 on success, a negative mvb_status for an argument error found on the
 *     host (nothing is launched in that case).
 *   - `dev_status` (optional, may be NULL) is a device int32[4] the caller zeroes; a kernel
 *     that meets an out-of-range slot / block id / position, or whose bounded wait runs out,
 *     records {code, detail, block, thread} there, skips the access and carries on.
 *   - bf16 tensors are passed as void*; the last dimension (head_dim) is contiguous and
 *     heads are contiguous (stride head_dim); only the token (row) stride is free.
 *   - KV pool layout per layer: [num_blocks, block_size, num_kv_heads, head_dim] bf16,
 *     contiguous, the layout the reference allocates in
 *     minivllm/executor/executor.py:51-60.  A slot is block_id * block_size + offset.
 *
 * Reference citations are paths inside w4096/mini-vllm.
 */
#ifndef MINI_VLLM_B200_H_
#define MINI_VLLM_B200_H_

#include <stddef.h>
#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

enum mvb_status {
  MVB_OK = 0,
  MVB_INVALID_ARGUMENT = -1,
  MVB_UNSUPPORTED_SHAPE = -2,
  MVB_LAUNCH_FAILED = -3,
  MVB_TENSOR_MAP_FAILED = -4,
  MVB_MISALIGNED = -5,
  MVB_NO_DRIVER_ENTRY = -6,
  MVB_SCRATCH_TOO_SMALL = -7
};

/* Library ABI version (bumped when a signature changes). */
int mvb_abi_version(void);
/* Human-readable name of a status code. */
const char* mvb_status_string(int status);

/*
 * Self-test of the kernels' bounded waits.  (No counterpart in the reference.)
 * Every wait inside the attention kernels is an mbarrier wait with an iteration limit; when it runs out
 * the kernel records {4 = wait timeout, detail, block, thread} in dev_status and returns instead of
 * hanging.  This entry runs that same wait, with `limit` polls (1..65536), on a barrier nothing arrives
 * at, so the status path can be exercised without disturbing a real kernel: after the stream has drained
 * dev_status[0] == 4 and dev_status[1] == limit.
 */
int mvb_selftest_wait_timeout(int32_t* dev_status, int limit, void* stream);

/*
 * Prefill batch packing on the device.
 * Replaces Executor._build_prefill_input (minivllm/executor/executor.py:81-127) and
 * Executor._build_block_table (:156-163): from per-sequence facts it expands
 *   input_ids[t], positions[t] = cached + i, slot_mapping[t] = blocks[pos/bs]*bs + pos%bs,
 *   cu_seqlens_q / cu_seqlens_k (exclusive prefix sums, int32 [num_seqs+1]) and, when
 *   block_table != NULL, the [num_seqs, table_width] table right-padded with -1.
 * Inputs (device int32): seq_len[num_seqs] (full length n), cached_len[num_seqs],
 *   blk_off[num_seqs+1] (exclusive prefix sum of per-sequence block counts),
 *   blocks_flat[blk_off[num_seqs]], new_tokens[num_tokens] (the uncached suffixes, concatenated).
 * A token whose block index is beyond its sequence's block list (warm-up requests own no
 * blocks, executor.py:62-78) gets slot -1.
 */
int mvb_pack_prefill(const int32_t* seq_len, const int32_t* cached_len, const int32_t* blk_off,
                     const int32_t* blocks_flat, const int32_t* new_tokens, int num_seqs, int num_tokens,
                     int table_width, int block_size, int64_t* input_ids, int64_t* positions,
                     int32_t* slot_mapping, int32_t* cu_seqlens_q, int32_t* cu_seqlens_k, int32_t* block_table,
                     int32_t* dev_status, void* stream);

/*
 * Decode batch packing on the device, written straight into (slices of) the CUDA-graph
 * runner's static buffers.
 * Replaces Executor._build_decode_input (minivllm/executor/executor.py:130-153) and the staging
 * copies of CudaGraphRunner.replay (minivllm/executor/graph.py:64-70).
 * For row b < num_seqs: input_ids = token, positions = n-1, cache_seqlens = n,
 *   slot = last_block*bs + (n - (nblk-1)*bs) - 1, block_table[b, :table_width] = blocks, pad -1.
 * Rows num_seqs..padded_seqs-1 are padding: input_ids 0, positions 0, slot -1, cache_seqlens 0,
 *   block table row -1.
 * The token of row b is prev_sampled[src_index[b]] when prev_sampled != NULL and
 * src_index[b] >= 0 (the previous step's sampler output, still on the device), else
 * host_tokens[b].
 * block_table has row stride table_stride (>= table_width) elements.
 */
int mvb_pack_decode(const int32_t* seq_len, const int32_t* blk_off, const int32_t* blocks_flat,
                    const int32_t* host_tokens, const int64_t* prev_sampled, const int32_t* src_index,
                    int num_seqs, int padded_seqs, int table_width, int64_t table_stride, int block_size,
                    int64_t* input_ids, int64_t* positions, int32_t* slot_mapping, int32_t* cache_seqlens,
                    int32_t* block_table, int32_t* dev_status, void* stream);

/*
 * Fused rotary embedding + paged KV-cache write.
 * Replaces RotaryEmbedding.forward (minivllm/models/layers/rotary.py:49-71) followed by
 * store_kvcache (minivllm/models/layers/attention.py:13-43).
 *   q [num_tokens, num_q_heads, head_dim] bf16, row stride q_row_stride elements: rotated in place.
 *   k [num_tokens, num_kv_heads, head_dim]: rotated; written to k_cache at slot_mapping[t]
 *     (skipped when the slot is -1 or slot_mapping == NULL) and, if k_in_place != 0, back into k.
 *   v: copied to v_cache at the same slot.
 *   cos_sin [max_pos, head_dim] fp32 = cat(cos, sin) as built by rotary.py:32-47; NULL disables
 *     the rotation (plain store_kvcache).  Arithmetic is fp32 with separately rounded products,
 *     one rounding to bf16, so results are bit-identical to the eager reference.
 * head_dim must be a multiple of 16; k_cache/v_cache may be NULL only with slot_mapping NULL.
 */
int mvb_rope_kv_write(void* q, int64_t q_row_stride, void* k, int64_t k_row_stride, const void* v,
                      int64_t v_row_stride, const int64_t* positions, const float* cos_sin, int64_t max_pos,
                      const int32_t* slot_mapping, void* k_cache, void* v_cache, int64_t num_slots,
                      int num_tokens, int num_q_heads, int num_kv_heads, int head_dim, int k_in_place,
                      int32_t* dev_status, void* stream);

/*
 * Per-head RMSNorm of q and k + rotary embedding + paged KV-cache write in one kernel.
 * Replaces the q_norm / k_norm / rotary_embedding / store_kvcache sequence of the model call-sites
 * (minivllm/models/models/qwen3.py:89-94, minivllm/models/models/gemma3.py:97-102).
 *   q, k, v are read where the projection left them (views of the packed qkv output are fine: only
 *   the row strides matter).  Each head row is normalised in fp32,
 *     y = x * rsqrt(mean(x^2) + eps) * w          (unit_offset == 0, nn.RMSNorm, qwen3.py:64-65)
 *     y = x * rsqrt(mean(x^2) + eps) * (1 + w)    (unit_offset != 0, gemma3.py:12-24)
 *   rounded to bf16 as the stand-alone norm would, rotated like mvb_rope_kv_write, and written: q in
 *   place, k to the cache slot (and in place if k_in_place), v to the cache slot.
 *   q_weight, k_weight: bf16 [head_dim].  head_dim / 16 must be a power of two (<= 32).
 * Results equal the unfused sequence up to the summation order of the squares (at most one bf16 ulp
 * on a few elements); use mvb_rope_kv_write where bit-exact KV contents are required.
 */
int mvb_qk_norm_rope_kv_write(void* q, int64_t q_row_stride, void* k, int64_t k_row_stride, const void* v,
                              int64_t v_row_stride, const void* q_weight, const void* k_weight, float eps,
                              int unit_offset, const int64_t* positions, const float* cos_sin, int64_t max_pos,
                              const int32_t* slot_mapping, void* k_cache, void* v_cache, int64_t num_slots,
                              int num_tokens, int num_q_heads, int num_kv_heads, int head_dim, int k_in_place,
                              int32_t* dev_status, void* stream);

/*
 * Paged decode attention (one query token per sequence), split along the context.
 * Replaces flash_attn_with_kvcache as called at minivllm/models/layers/attention.py:90-91.
 *
 * mvb_decode_workspace_bytes: size of the caller-supplied workspace for up to max_seqs rows.
 * mvb_decode_plan: one small launch per step (the plan depends only on cache_seqlens and the
 *   window, so every layer of a step shares it) that balances 16-token tiles over the
 *   persistent grid and records it in the workspace.
 * mvb_decode_attn: q [num_seqs, num_q_heads, head_dim] -> out (same shape, bf16).  Key j of
 *   sequence b is visible iff max(0, n-1-window_left) <= j < n with n = cache_seqlens[b]
 *   (window_left < 0: no window).  Rows with n == 0 (graph padding, graph.py:66-69) give zeros.
 *   Grid and pointers do not depend on data, so the launch sequence can be captured in a
 *   CUDA graph.  block_table is [num_seqs, table_width] with row stride table_stride.
 *   Supported: head_dim 128 or 256; num_q_heads/num_kv_heads <= 8; num_kv_heads in {1,2,4} or a
 *   multiple of 8 (head_dim 128) / 4 (head_dim 256); block_size a multiple of 16.
 *   The plan must have been made for the same cache_seqlens, window and head shape.
 */
size_t mvb_decode_workspace_bytes(int max_seqs, int num_q_heads, int head_dim);
int mvb_decode_plan(const int32_t* cache_seqlens, int num_seqs, int window_left, int num_q_heads,
                    int num_kv_heads, int head_dim, void* workspace, size_t workspace_bytes, void* stream);
/* Same plan, and the first block id of every CTA's range is looked up here once per step instead of by
 * every layer's attention kernel in front of its first TMA load (the table must be the one passed to
 * mvb_decode_attn). */
int mvb_decode_plan_with_table(const int32_t* cache_seqlens, const int32_t* block_table, int64_t table_stride,
                               int block_size, int num_seqs, int window_left, int num_q_heads, int num_kv_heads,
                               int head_dim, void* workspace, size_t workspace_bytes, void* stream);
int mvb_decode_attn(const void* q, int64_t q_row_stride, const void* k_cache, const void* v_cache,
                    int64_t num_blocks, int block_size, const int32_t* cache_seqlens,
                    const int32_t* block_table, int64_t table_stride, int table_width, int num_seqs,
                    int num_q_heads, int num_kv_heads, int head_dim, float scale, int window_left, void* out,
                    int64_t out_row_stride, void* workspace, size_t workspace_bytes, int32_t* dev_status,
                    void* stream);

/*
 * Decode attention for callers that cannot provide a workspace.  (No counterpart in the reference,
 * which lets PyTorch allocate whatever its attention library needs.)
 *
 * Meant for users who must not, or cannot, allocate device memory around this call: a process whose
 * GPU memory is fully parcelled out at start-up, a thin binding that can only pass on buffers it was
 * given, or a latency-critical loop that has to stay clear of cudaMalloc and its device-wide
 * synchronisation.  It computes exactly what mvb_decode_plan followed by mvb_decode_attn compute, but
 * keeps the plan, the partial results and the arrival counters in a MVB_STATIC_SCRATCH_BYTES array
 * that is part of the library image: each GPU that loads the library holds that memory until the
 * process ends.  Inputs and outputs are still the caller's.
 *
 *   - Limit: the scratch needed for (num_seqs, num_q_heads, head_dim) must fit the 8 MiB array.
 *     That covers 16 or 32 query heads of dimension 128 (or 4 to 16 of dimension 256) with
 *     thousands of sequences; 64 heads x 128 does not fit.  Larger requests return
 *     MVB_SCRATCH_TOO_SMALL and launch nothing.
 *   - The first call on each device looks up the array's device address; make that first call
 *     outside any stream capture.  No call allocates or frees memory.
 *   - All calls on a device share the one array.  Each call re-plans and clears what has to start
 *     at zero, so earlier contents do not matter, but two calls whose kernels overlap on the GPU
 *     (different streams) would race on it: keep them ordered.
 */
#define MVB_STATIC_SCRATCH_BYTES (8u << 20)
int mvb_decode_attn_static(const void* q, int64_t q_row_stride, const void* k_cache, const void* v_cache,
                           int64_t num_blocks, int block_size, const int32_t* cache_seqlens,
                           const int32_t* block_table, int64_t table_stride, int table_width, int num_seqs,
                           int num_q_heads, int num_kv_heads, int head_dim, float scale, int window_left,
                           void* out, int64_t out_row_stride, int32_t* dev_status, void* stream);

/*
 * Causal varlen prefill attention on the tcgen05 tensor cores.
 * Replaces flash_attn_varlen_func as called at minivllm/models/layers/attention.py:84-87.
 *   q [total_q, num_q_heads, head_dim]; sequence s owns rows cu_seqlens_q[s]..cu_seqlens_q[s+1].
 *   block_table == NULL: k, v are dense [total_k, num_kv_heads, head_dim] (row strides
 *     k_row_stride / v_row_stride; kv_rows = total_k) sliced by cu_seqlens_k.
 *   block_table != NULL: k, v are the paged pool (kv_rows = num_blocks*block_size slots,
 *     both row strides = num_kv_heads*head_dim) and keys 0..k_len-1 of sequence s are gathered
 *     through row s of the table (the prefix-cache case, attention.py:79-83).
 *   Query i of a sequence sits at position p = k_len - q_len + i and sees keys
 *   max(0, p - window_left) <= j <= p.
 * Supported: head_dim 128 or 256, any GQA ratio; with a block table, block_size a multiple of 128
 * (head_dim 128) or of 64 (head_dim 256), the kernel's KV tile, so that a tile never straddles blocks.
 */
int mvb_prefill_attn(const void* q, int64_t q_row_stride, const void* k, int64_t k_row_stride, const void* v,
                     int64_t v_row_stride, int64_t kv_rows, const int32_t* cu_seqlens_q, const int32_t* cu_seqlens_k,
                     const int32_t* block_table, int64_t table_stride, int block_size, int num_seqs,
                     int total_q, int max_seqlen_q, int num_q_heads, int num_kv_heads, int head_dim,
                     float scale, int window_left, void* out, int64_t out_row_stride, int32_t* dev_status,
                     void* stream);

/*
 * The same launch with its work given as a list.  (No counterpart in the reference.)
 *   items: int32 [num_items, 2] on the device, one (sequence, query block) pair per work item; query block b of a
 *   sequence is its rows b*R .. b*R+R-1 with R = mvb_prefill_item_rows(...) (128 or 256, a property of the head
 *   layout).  The list must hold every query block of every sequence exactly once (rows of a block that is not
 *   listed are not written); its order is the order in which the GPU takes the work, so the caller lists the blocks
 *   with the most visible keys first.  Entries outside the batch are skipped.  num_items <= 65535.
 * Without the list mvb_prefill_attn launches a block index for every (sequence, block rank) up to the longest
 * sequence's block count; on a ragged batch most of those are empty and each costs a round trip to hand out
 * (config 3's prefill batch: 1920 indices for 872 items, 140 us; with the list, longest first: 112 us).
 * The host knows the lengths when it packs the step (Executor._build_prefill_input, executor.py:81-127), which is
 * where the list is built; results are bit-identical to mvb_prefill_attn.  A list that fills at least 85 % of
 * the grid (sequences of about one length) is not read: the grid form is run, which is then the faster one.
 */
int mvb_prefill_item_rows(int num_q_heads, int num_kv_heads, int head_dim);
int mvb_prefill_attn_items(const void* q, int64_t q_row_stride, const void* k, int64_t k_row_stride, const void* v,
                           int64_t v_row_stride, int64_t kv_rows, const int32_t* cu_seqlens_q,
                           const int32_t* cu_seqlens_k, const int32_t* block_table, int64_t table_stride,
                           int block_size, int num_seqs, int total_q, int max_seqlen_q, int num_q_heads,
                           int num_kv_heads, int head_dim, float scale, int window_left, void* out,
                           int64_t out_row_stride, const int32_t* items, int num_items, int32_t* dev_status,
                           void* stream);

/*
 * Fused temperature / top-k / Gumbel-max sampler over the vocabulary.
 * Replaces Sampler.forward (minivllm/models/layers/sampler.py:9-31).
 *   logits [num_rows, vocab] bf16 (row stride in elements) -> out int64 [num_rows].
 *   top_k == NULL and top_p == NULL: greedy argmax of logits / temperature (lowest index wins ties), the
 *     reference's path when no top-k/top-p is requested (sampler.py:31).
 *   top_k != NULL or top_p != NULL: row r keeps every logit >= its top_k[r]-th largest
 *     (top_k[r] <= 0 keeps all), then, if top_p[r] < 1, the most likely of those until their
 *     softmax(logit / temperature) mass reaches top_p[r] (tokens tied with the last one are kept);
 *     it adds Gumbel noise from Philox4x32-10 keyed by (seed, offset, r, column) to
 *     logit / temperature and returns the argmax.  temperatures may be NULL (all 1).
 *   scatter_table/scatter_index (both or neither): the token of row r is also stored at
 *     scatter_table[scatter_index[r]], a per-request table the next decode packing reads its input
 *     tokens from (mvb_pack_decode's prev_sampled/src_index), so the sampled ids never have to visit
 *     the host between steps (the reference syncs on .tolist() every step, executor.py:193-195).
 */
int mvb_sample(const void* logits, int64_t row_stride, int num_rows, int vocab, const float* temperatures,
               const int32_t* top_k, const float* top_p, uint64_t seed, uint64_t offset, int64_t* out,
               int64_t* scatter_table, const int32_t* scatter_index, int32_t* dev_status, void* stream);

/*
 * lm_head and greedy sampling in one kernel: out[r] = argmax_n bf16(sum_k hidden_states[r, k] * weight[n, k]),
 * the lowest column winning ties.
 * Replaces, for requests without top-k / top-p (the reference's argmax path), logits = lm_head(hidden_states)
 * (minivllm/models/models/qwen3.py:215-219, gemma3.py:258-262) followed by Sampler.forward's
 * torch.argmax (minivllm/models/layers/sampler.py:31): a tcgen05 GEMM whose epilogue rounds each accumulator to
 * bf16 - the logit the unfused path would have stored - and keeps only the best (value, column) per row, so the
 * [num_rows, vocab] logits are never written or read back.  A positive temperature does not change an argmax
 * and is not needed here.
 *   hidden_states [num_rows, hidden] bf16 (row stride in elements), weight [vocab, hidden] bf16 (the lm_head /
 *   tied embedding matrix as stored); hidden a multiple of 64; rows 16-byte aligned.
 *   scratch: mvb_lm_head_argmax_scratch_bytes(max rows) bytes of device memory that the caller zeroes ONCE; every
 *   call leaves it zeroed again.  Calls that share a scratch must not overlap on the GPU.
 *   scatter_table / scatter_index as for mvb_sample.
 * Accumulation is fp32 in the tensor cores' order, which is not cuBLAS's: a logit can round to the neighbouring
 * bf16 value, so the token may differ from the unfused path where the two best logits are within one bf16 step.
 */
size_t mvb_lm_head_argmax_scratch_bytes(int max_rows);
int mvb_lm_head_argmax(const void* hidden_states, int64_t x_row_stride, const void* weight, int64_t w_row_stride,
                       int num_rows, int hidden, int vocab, int64_t* out, int64_t* scatter_table,
                       const int32_t* scatter_index, void* scratch, size_t scratch_bytes, int32_t* dev_status,
                       void* stream);

/*
 * Decoder-layer glue around the attention path.  A decode step of a small model is bound by the number
 * of kernels it launches, so the elementwise chains the models run between their GEMMs are fused.
 *
 * mvb_act_mul: out[t, i] = act(gate_up[t, i]) * gate_up[t, intermediate + i] on a packed
 *   [rows, 2 * intermediate] projection; act = SiLU (minivllm/models/models/qwen3.py:117-121) or
 *   tanh-GELU (gelu_tanh != 0, minivllm/models/models/gemma3.py:122-128).  The activation is rounded
 *   to bf16 before the product, as the unfused sequence rounds it.
 * mvb_add_rmsnorm: the residual update and the next RMSNorm of a decoder layer in one pass over a row:
 *     y' = y                       (y_weight == NULL; qwen3.py:146-155)
 *     y' = rmsnorm(y, y_weight)    (Gemma's post-attention / post-feedforward norm, gemma3.py:157-170)
 *     x  = bf16(x + y')            (in place, x is [rows, hidden] contiguous)
 *     out = rmsnorm(x, weight)     (the following input / post-attention / pre-feedforward / final norm)
 *   rmsnorm(v, w) = v * rsqrt(mean(v^2) + eps) * w, or * (1 + w) when unit_offset != 0, in fp32.
 *   hidden must be a multiple of 8 and at most 8192.
 * mvb_add_rmsnorm_last_tokens: the same residual add and norm, but only for the LAST token of every sequence of
 *   a packed prefill batch, gathered by the kernel itself: output row r is computed from source row
 *   cu_seqlens_q[r + 1] - 1, which is the row the reference picks with last_indices = cu_seqlens_q[1:] - 1
 *   (minivllm/models/models/qwen3.py:215-217, gemma3.py:258-260) AFTER running the final norm over every token.
 *   x is read only (the residual stream is not needed after the final norm); out is [num_seqs, hidden].
 */
int mvb_add_rmsnorm_last_tokens(const void* x, const void* y, int64_t y_row_stride, const void* y_weight,
                                const void* weight, void* out, const int32_t* cu_seqlens_q, int num_seqs, int hidden,
                                float eps, int unit_offset, void* stream);
int mvb_act_mul(const void* gate_up, int64_t in_row_stride, void* out, int64_t out_row_stride, int rows,
                int intermediate, int gelu_tanh, void* stream);
int mvb_add_rmsnorm(void* x, const void* y, int64_t y_row_stride, const void* y_weight, const void* weight,
                    void* out, int rows, int hidden, float eps, int unit_offset, void* stream);

/*
 * Attention with capped scores, for models whose scores pass c tanh(s / c) before the softmax (softcap = c > 0; 0 = none)
 * and mixers whose output carries a constant factor (out_scale; 1 = none).  Otherwise mvb_prefill_attn_items (items may be
 * NULL here: the grid form) and mvb_decode_attn.  The cap is computed to a few fp32 ulps of c.
 */
int mvb_prefill_attn_capped(const void* q, int64_t q_row_stride, const void* k, int64_t k_row_stride, const void* v,
                            int64_t v_row_stride, int64_t kv_rows, const int32_t* cu_seqlens_q,
                            const int32_t* cu_seqlens_k, const int32_t* block_table, int64_t table_stride,
                            int block_size, int num_seqs, int total_q, int max_seqlen_q, int num_q_heads,
                            int num_kv_heads, int head_dim, float scale, int window_left, void* out,
                            int64_t out_row_stride, const int32_t* items, int num_items, float softcap, float out_scale,
                            int32_t* dev_status, void* stream);
int mvb_decode_attn_capped(const void* q, int64_t q_row_stride, const void* k_cache, const void* v_cache,
                           int64_t num_blocks, int block_size, const int32_t* cache_seqlens, const int32_t* block_table,
                           int64_t table_stride, int table_width, int num_seqs, int num_q_heads, int num_kv_heads,
                           int head_dim, float scale, int window_left, void* out, int64_t out_row_stride, void* workspace,
                           size_t workspace_bytes, float softcap, float out_scale, int32_t* dev_status, void* stream);

/*
 * What attention may have beyond a window and a cap; every field is optional (NULL / 0).
 *   sinks [num_q_heads]   one more logit per head, as it is, in the softmax's denominator only
 *   slopes [num_q_heads]  slope * (query position - key position) is taken off a scaled score
 *   head_gate             [tokens, num_q_heads] in the activations' type: a head's output is multiplied by sigmoid(gate)
 *   keep_first            with a window: keys at positions below it stay visible
 * The _ext entry points are the ones above with it (no score cap beside it, except in mvb_any_attn_ext).  A plan for kept first tokens
 * comes from mvb_decode_plan_ext with the same keep_first.
 */
typedef struct {
  const float* sinks;
  const float* slopes;
  const void* head_gate;
  int64_t head_gate_row_stride;
  int keep_first;
} mvb_attn_extras;
int mvb_prefill_attn_ext(const void* q, int64_t q_row_stride, const void* k, int64_t k_row_stride, const void* v, int64_t v_row_stride,
                         int64_t kv_rows, const int32_t* cu_seqlens_q, const int32_t* cu_seqlens_k, const int32_t* block_table,
                         int64_t table_stride, int block_size, int num_seqs, int total_q, int max_seqlen_q, int num_q_heads,
                         int num_kv_heads, int head_dim, float scale, int window_left, void* out, int64_t out_row_stride,
                         const int32_t* items, int num_items, float out_scale, const mvb_attn_extras* extras, int32_t* dev_status,
                         void* stream);
int mvb_decode_plan_ext(const int32_t* cache_seqlens, const int32_t* block_table, int64_t table_stride, int block_size, int num_seqs,
                        int window_left, int keep_first, int num_q_heads, int num_kv_heads, int head_dim, void* workspace,
                        size_t workspace_bytes, void* stream);
int mvb_decode_attn_ext(const void* q, int64_t q_row_stride, const void* k_cache, const void* v_cache, int64_t num_blocks, int block_size,
                        const int32_t* cache_seqlens, const int32_t* block_table, int64_t table_stride, int table_width, int num_seqs,
                        int num_q_heads, int num_kv_heads, int head_dim, float scale, int window_left, void* out, int64_t out_row_stride,
                        void* workspace, size_t workspace_bytes, float out_scale, const mvb_attn_extras* extras, int32_t* dev_status,
                        void* stream);

/*
 * The entry points below take dtype 0 (activations, weights and K/V in bf16) or 1 (fp32); the arithmetic between loads and
 * stores is fp32 in both.  A "ragged step" has cu_seqlens_q [num_seqs + 1]; with cu_seqlens_q == NULL every sequence
 * brings one token and row t is sequence t.  positions [num_tokens] are absolute; a sequence whose first token of the
 * step has position 0 starts from a zero state whatever its slot holds, so slots need no clearing.  state_slots
 * [num_seqs] picks a sequence's slot, negative = no state is read or kept (padding rows, warm-up).
 *
 * mvb_any_attn: attention of any head size (<= 1024), group size and dtype, one warp per (token, head), for what the
 *   tensor-core kernels do not take.  block_table == NULL: dense K/V rows cu_seqlens_k[s] + j (row strides); else a pool of
 *   kv_rows slots (k_row_stride = v_row_stride = num_kv_heads * head_dim).  cache_seqlens (optional): rows of length 0 give 0.
 * mvb_rope_kv_write_f32: mvb_rope_kv_write for fp32 activations and pools.
 * mvb_rope_norm_kv_write: the same in either dtype, with a norm behind the rotation: norm_dim > 0 divides every q and k head by
 *   sqrt(mean(x^2) + eps), the mean over norm_dim coordinates (what a head is padded with is zero).  cos_sin == NULL: no rotation;
 *   num_kv_heads == 0: q alone (k, v and the caches may be NULL).
 */
int mvb_any_attn(int dtype, const void* q, int64_t q_row_stride, const void* k, int64_t k_row_stride, const void* v,
                 int64_t v_row_stride, int64_t kv_rows, const int32_t* block_table, int64_t table_stride, int table_width,
                 int block_size, const int32_t* cu_seqlens_q, const int32_t* cu_seqlens_k, const int64_t* positions,
                 const int32_t* cache_seqlens, int num_seqs, int num_tokens, int num_q_heads, int num_kv_heads, int head_dim,
                 float scale, int window_left, float softcap, float out_scale, void* out, int64_t out_row_stride,
                 int32_t* dev_status, void* stream);
int mvb_any_attn_ext(int dtype, const void* q, int64_t q_row_stride, const void* k, int64_t k_row_stride, const void* v,
                     int64_t v_row_stride, int64_t kv_rows, const int32_t* block_table, int64_t table_stride, int table_width,
                     int block_size, const int32_t* cu_seqlens_q, const int32_t* cu_seqlens_k, const int64_t* positions,
                     const int32_t* cache_seqlens, int num_seqs, int num_tokens, int num_q_heads, int num_kv_heads, int head_dim,
                     float scale, int window_left, float softcap, float out_scale, const mvb_attn_extras* extras, void* out,
                     int64_t out_row_stride, int32_t* dev_status, void* stream);
int mvb_rope_norm_kv_write(int dtype, void* q, int64_t q_row_stride, void* k, int64_t k_row_stride, const void* v, int64_t v_row_stride,
                           const int64_t* positions, const float* cos_sin, int64_t max_pos, const int32_t* slot_mapping, void* k_cache,
                           void* v_cache, int64_t num_slots, int num_tokens, int num_q_heads, int num_kv_heads, int head_dim,
                           int k_in_place, int norm_dim, float eps, int32_t* dev_status, void* stream);
int mvb_rope_kv_write_f32(float* q, int64_t q_row_stride, float* k, int64_t k_row_stride, const float* v,
                          int64_t v_row_stride, const int64_t* positions, const float* cos_sin, int64_t max_pos,
                          const int32_t* slot_mapping, float* k_cache, float* v_cache, int64_t num_slots, int num_tokens,
                          int num_q_heads, int num_kv_heads, int head_dim, int k_in_place, int32_t* dev_status, void* stream);

/*
 * Glue around an fp32 residual stream x [rows, width].  rmsnorm(v, w) = v * rsqrt(mean(v^2) + eps) * w.
 * mvb_residual_norm: x += (y_weight ? rmsnorm(y, y_weight) : y) in place; out = rmsnorm(x, weight).  row_ends != NULL: output
 *   row r is computed from source row row_ends[r + 1] - 1 and x is left as it is.
 * mvb_embed_norm: x[r] = table[ids[r]]; out = rmsnorm(x, weight).
 * mvb_residual_norm_pair, mvb_embed_norm_pair: for layers whose two sublayers read the same stream through norms of their own: out =
 *   rmsnorm(x, weight), out2 = rmsnorm(x, weight2) (both optional together).  The looked-up row is multiplied by scale; the stream of
 *   row r also gets extra[extra_index[r, j]], j < num_extra (rows of routed experts), added in that order.
 * mvb_glu: g = min(gate, limit), u = clamp(up, -limit, limit), out = g sigmoid(alpha g) (u + offset) on a packed
 *   [rows, 2 * intermediate] projection, times sigmoid(row_gate[row]) where there is one.  mvb_clamped_glu: offset 1.
 * mvb_residual_norm_pair_ext: the stream of row r also gets own_weights[r] (fp32; NULL: nothing) times row r of `own`, and an extra
 *   index of -1 adds nothing.
 * mvb_xielu: act[0] z^2 + z / 2 for z > 0, act[1] (e^z - 1 - z) + z / 2 for z <= 0 (act: fp32, on the device).
 * mvb_cap_logits: out = cap tanh(in / cap) (cap == 0: a copy), each side bf16 or fp32.
 * mvb_argmax_f32: the greedy token of fp32 logits (lowest column wins ties); scatter_* as for mvb_sample.
 */
int mvb_argmax_f32(const float* logits, int64_t row_stride, int rows, int cols, int64_t* out, int64_t* scatter_table,
                   const int32_t* scatter_index, void* stream);
int mvb_residual_norm(int dtype, float* x, const void* y, int64_t y_row_stride, const void* y_weight, const void* weight,
                      void* out, const int32_t* row_ends, int rows, int width, float eps, void* stream);
int mvb_embed_norm(int dtype, const int64_t* ids, const void* table, int64_t vocab, float* x, const void* weight, void* out,
                   int rows, int width, float eps, int32_t* dev_status, void* stream);
int mvb_residual_norm_pair(int dtype, float* x, const void* y, int64_t y_row_stride, const void* extra, int64_t extra_row_stride,
                           int64_t extra_rows, const int32_t* extra_index, int num_extra, const void* weight, void* out,
                           const void* weight2, void* out2, const int32_t* row_ends, int rows, int width, float eps, int32_t* dev_status,
                           void* stream);
int mvb_residual_norm_pair_ext(int dtype, float* x, const void* y, int64_t y_row_stride, const void* extra, int64_t extra_row_stride,
                               int64_t extra_rows, const int32_t* extra_index, int num_extra, const void* own, int64_t own_row_stride,
                               const float* own_weights, const void* weight, void* out, const void* weight2, void* out2,
                               const int32_t* row_ends, int rows, int width, float eps, int32_t* dev_status, void* stream);
int mvb_xielu(int dtype, const void* in, int64_t in_row_stride, void* out, int64_t out_row_stride, int rows, int cols, const float* act,
              void* stream);
int mvb_embed_norm_pair(int dtype, const int64_t* ids, const void* table, int64_t vocab, float scale, float* x, const void* weight,
                        void* out, const void* weight2, void* out2, int rows, int width, float eps, int32_t* dev_status, void* stream);
int mvb_glu(int dtype, const void* gate_up, int64_t in_row_stride, void* out, int64_t out_row_stride, int rows, int intermediate,
            float limit, float alpha, float offset, const void* row_gate, int64_t gate_row_stride, void* stream);
int mvb_clamped_glu(int dtype, const void* gate_up, int64_t in_row_stride, void* out, int64_t out_row_stride, int rows,
                    int intermediate, float limit, float alpha, void* stream);
int mvb_cap_logits(int in_dtype, int out_dtype, const void* in, int64_t in_row_stride, void* out, int64_t out_row_stride,
                   int rows, int cols, float cap, void* stream);

/*
 * Recurrent mixers with per-sequence state slots.
 * mvb_short_conv: mvb_short_conv_silu with the SiLU optional, and the last `copies` channels written a second time, right behind the
 *   others.
 * mvb_short_conv_silu: out[t, c] = silu(bias[c] + sum_j weight[j, c] u[t - j, c]), j < taps <= 32; inputs from before the
 *   step come from state [num_slots, taps - 1, channels] (dtype; oldest input first), which is then brought up to date.
 * mvb_selective_scan: S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c u_c B_n, out_c = (sum_n S[c, n] C_n + D_c u_c) silu(z_c),
 *   dt = softplus(raw + dt_bias).  a_log2e [channels, state_stride] = A * log2(e), zero past num_states; state [num_slots,
 *   channels, state_stride] fp32; state_stride a multiple of 4, num_states <= 256.
 * mvb_gated_delta: per head S <- g * S, e = beta (v - S^T k), S <- S + k e^T, o = S^T q, with q, k made unit vectors
 *   (1e-6 inside the root; q times q_scale), g = exp(-exp_a softplus(a + dt_bias)) per key channel, beta = sigmoid(b);
 *   out = o / rms(o) * norm_weight * sigmoid(gate) * out_scale.  Head h reads q/k head h / (heads / kv_heads).  q, k
 *   [tokens, kv_heads, dim], v [tokens, heads, vdim] share one row stride; dim <= 256.  state [num_slots, heads, dim,
 *   vdim rounded up to 4] fp32.  scratch: mvb_gated_delta_scratch_bytes(...) bytes.
 */
int mvb_short_conv(int dtype, const void* u, int64_t u_row_stride, const void* weight, const void* bias, void* out,
                   int64_t out_row_stride, void* state, const int32_t* state_slots, int64_t num_slots, const int32_t* cu_seqlens_q,
                   const int64_t* positions, int num_seqs, int num_tokens, int channels, int taps, int silu, int copies,
                   int32_t* dev_status, void* stream);
int mvb_short_conv_silu(int dtype, const void* u, int64_t u_row_stride, const void* weight, const void* bias, void* out,
                        int64_t out_row_stride, void* state, const int32_t* state_slots, int64_t num_slots,
                        const int32_t* cu_seqlens_q, const int64_t* positions, int num_seqs, int num_tokens, int channels,
                        int taps, int32_t* dev_status, void* stream);
int mvb_selective_scan(int dtype, const void* u, int64_t u_row_stride, const void* dt, int64_t dt_row_stride, const void* z,
                       int64_t z_row_stride, const void* b, const void* c, int64_t bc_row_stride, const float* dt_bias,
                       const float* a_log2e, const float* d, void* out, int64_t out_row_stride, float* state,
                       const int32_t* state_slots, int64_t num_slots, const int32_t* cu_seqlens_q, const int64_t* positions,
                       int num_seqs, int num_tokens, int channels, int num_states, int state_stride, int32_t* dev_status,
                       void* stream);
size_t mvb_gated_delta_scratch_bytes(int dtype, int num_tokens, int num_seqs, int heads, int kv_heads, int dim, int vdim,
                                     int ragged);
int mvb_gated_delta(int dtype, const void* q, const void* k, const void* v, int64_t qkv_row_stride, const void* a,
                    int64_t a_row_stride, const void* b, int64_t b_row_stride, const void* gate, int64_t gate_row_stride,
                    const float* exp_a, const float* dt_bias, const float* norm_weight, void* out, int64_t out_row_stride,
                    float* state, const int32_t* state_slots, int64_t num_slots, const int32_t* cu_seqlens_q,
                    const int64_t* positions, int num_seqs, int num_tokens, int heads, int kv_heads, int dim, int vdim,
                    float q_scale, float eps, float out_scale, void* scratch, size_t scratch_bytes, int32_t* dev_status,
                    void* stream);

/*
 * Linear attention with decay (per-sequence state slots as above): per head S <- D S + w k v^T, o = S^T q, then
 * out = o / rms(o) * norm_weight * gate function.  q, k [tokens, heads, dim], v [tokens, heads, vdim] share one row stride; q is
 * multiplied by q_scale; dim <= 256; state [num_slots, heads, dim, vdim rounded up to 4] fp32.
 * mvb_gated_linear: D = diag(sigmoid(decay + decay_bias)^inv_tau) per key channel (decay [tokens, heads * dim]), w = 1; SiLU gate;
 *   norm_weight [vdim].
 * mvb_mlstm: log gates i = cap tanh((input + input_bias) / cap), f = log sigmoid(cap tanh((forget + forget_bias) / cap)) per head; with
 *   the running maximum m' = max(f + m, i) (m from 0): D = e^{f + m - m'}, w = e^{i - m'}; n <- D n + w k; o over
 *   max(|n . q|, e^{-m'}) + 1e-6; sigmoid gate; norm_weight [heads * vdim].  normaliser [num_slots, heads, dim], maximum
 *   [num_slots, heads] fp32.
 * scratch: mvb_linear_attn_scratch_bytes(...) bytes (exp_gates: 1 for mvb_mlstm; ragged: cu_seqlens_q != NULL).
 */
size_t mvb_linear_attn_scratch_bytes(int dtype, int num_tokens, int num_seqs, int heads, int dim, int vdim, int exp_gates, int ragged);
int mvb_gated_linear(int dtype, const void* q, const void* k, const void* v, int64_t qkv_row_stride, const void* decay,
                     int64_t decay_row_stride, const float* decay_bias, float inv_tau, const void* gate, int64_t gate_row_stride,
                     const float* norm_weight, void* out, int64_t out_row_stride, float* state, const int32_t* state_slots,
                     int64_t num_slots, const int32_t* cu_seqlens_q, const int64_t* positions, int num_seqs, int num_tokens, int heads,
                     int dim, int vdim, float q_scale, float eps, void* scratch, size_t scratch_bytes, int32_t* dev_status, void* stream);
int mvb_mlstm(int dtype, const void* q, const void* k, const void* v, int64_t qkv_row_stride, const void* forget,
              int64_t forget_row_stride, const float* forget_bias, const void* input, int64_t input_row_stride, const float* input_bias,
              float cap, const void* gate, int64_t gate_row_stride, const float* norm_weight, void* out, int64_t out_row_stride,
              float* state, float* normaliser, float* maximum, const int32_t* state_slots, int64_t num_slots,
              const int32_t* cu_seqlens_q, const int64_t* positions, int num_seqs, int num_tokens, int heads, int dim, int vdim,
              float q_scale, float eps, void* scratch, size_t scratch_bytes, int32_t* dev_status, void* stream);

/*
 * Hyper-connected residual streams x [rows, streams, width] fp32; norms in `groups` equal consecutive parts of a row.
 * mvb_hyper_embed_norm: every stream = table[ids] + pos_table[positions]; h = norm(sum_s in[s] x_s) * weight.
 * mvb_hyper_norm: x_t <- sum_s mix[s, t] x_s + out[t] y; h = norm(sum_s in[s] x_s) * weight (in NULL: the plain sum).  row_ends != NULL:
 *   output row r comes from source row row_ends[r + 1] - 1 and x is left as it is.  streams <= 16.
 * mvb_poly_norm: out = a N(z) + b N(z^2) + c N(z^3) + e over the row's `cols` values, N(v) = v / sqrt(mean(v^2) + eps), act = {a, b, c,
 *   e} on the device; columns cols..out_cols-1 become 0.
 */
int mvb_hyper_embed_norm(int dtype, const int64_t* ids, const int64_t* positions, const void* table, int64_t vocab,
                         const void* pos_table, int64_t max_positions, float* x, const float* in_weights, const void* weight, void* h,
                         int rows, int width, int streams, int groups, float eps, int32_t* dev_status, void* stream);
int mvb_hyper_norm(int dtype, float* x, const void* y, int64_t y_row_stride, const float* mix, const float* out_weights,
                   const float* in_weights, const void* weight, void* h, const int32_t* row_ends, int rows, int width, int streams,
                   int groups, float eps, void* stream);
int mvb_poly_norm(int dtype, const void* z, int64_t z_row_stride, void* out, int64_t out_row_stride, int rows, int cols, int out_cols,
                  const float* act, float eps, void* stream);

/*
 * Attention over a cached latent (pool [num_blocks, block_size, width], one row per token for all heads).
 * mvb_latent_norm: q_out = rmsnorm(q) [tokens, q_pad] and, with c != NULL, c_out = rmsnorm(c) [tokens, c_pad], also into
 *   cache[slot_mapping[t]] (slots < 0: not written; cache NULL: no cache); columns behind q_cols / c_cols become 0.
 * mvb_gather_latents: the contexts cu_seqlens_k describes as dense rows.
 * mvb_gate_mul: out = o * sigmoid(gate).
 * mvb_latent_decode: one query row per sequence in the absorbed form: out[b, h] = softmax(scale q[b, h] . c) c, bf16; width one of 64,
 *   128, 192, 256, 384, 512; block_size a multiple of 64.  The workspace (mvb_decode_workspace_bytes(num_seqs, num_heads, width)) must
 *   hold the plan of mvb_latent_decode_plan for the same cache_seqlens.
 */
int mvb_latent_norm(int dtype, const void* q, int64_t q_row_stride, const void* q_weight, void* q_out, int q_cols, int q_pad,
                    const void* c, int64_t c_row_stride, const void* c_weight, void* c_out, int c_cols, int c_pad, void* cache,
                    const int32_t* slot_mapping, int64_t num_slots, int num_tokens, float eps, int32_t* dev_status, void* stream);
int mvb_gather_latents(const void* cache, int64_t num_slots, int row_bytes, const int32_t* block_table, int64_t table_stride,
                       int table_width, int block_size, const int32_t* cu_seqlens_k, int num_seqs, int num_rows, void* out,
                       int32_t* dev_status, void* stream);
int mvb_gate_mul(int dtype, const void* o, int64_t o_row_stride, const void* gate, int64_t gate_row_stride, void* out,
                 int64_t out_row_stride, int rows, int cols, void* stream);
int mvb_latent_decode_plan(const int32_t* cache_seqlens, const int32_t* block_table, int64_t table_stride, int block_size, int num_seqs,
                           int num_heads, int width, void* workspace, size_t workspace_bytes, void* stream);
int mvb_latent_decode(const void* q, int64_t q_row_stride, int64_t q_head_stride, const void* cache, int64_t num_blocks, int block_size,
                      const int32_t* cache_seqlens, const int32_t* block_table, int64_t table_stride, int table_width, int num_seqs,
                      int num_heads, int width, float scale, void* out, int64_t out_row_stride, int64_t out_head_stride, void* workspace,
                      size_t workspace_bytes, int32_t* dev_status, void* stream);

/*
 * Mixture of experts.  Group sizes stay on the device.
 * mvb_moe_route: the `top` largest of fp32 logits [num_tokens, num_experts <= 1024] per token (ids, and weights = sigmoid(logit)), each
 *   row's number among its expert's (ranks), every expert's first row in sorted order (offsets [num_experts + 1]), and row tiles
 *   (expert, first row, rows, 0) of at most block_rows rows; their number is tile_offsets[num_experts].  counters [num_experts + 1] must
 *   be zero and is left zero.  max_tiles >= num_tokens * top / block_rows + min(num_experts, num_tokens * top).
 * mvb_moe_route_ext: scores are the softmax over all num_experts + num_identity outputs (softmax != 0) or sigmoids; the choice is by score
 *   + correction [outputs] (NULL: the score), the weight is the score times weight_scale.  The outputs behind the experts are identity
 *   experts: rank -1, no row; their weights are added up per token in identity_weights [num_tokens].
 * mvb_moe_gather: rows of h in sorted order (none, and slot -1, for a rank of -1); slots [num_tokens, top] and row_weights [num_tokens * top] come with it.
 * mvb_moe_gemm: per expert, out rows = weight [num_experts, m, k] times x rows; gated: weight [num_experts, 2, m, k] (gate, up) and
 *   y = g sigmoid(alpha g) (u + offset), g = min(w gate, limit), u = clamp(w up, -limit, limit), w = row_weights (NULL: 1); gated == 2: w multiplies y instead
 *   of gate and up.  block_rows
 *   32, 64 or 128 (fp32: 64, w_row_stride = k), as in the tiles.
 */
int mvb_moe_route(const float* logits, int64_t logits_row_stride, int num_tokens, int num_experts, int top, int block_rows, int max_tiles,
                  int32_t* counters, int32_t* ids, float* weights, int32_t* ranks, int32_t* offsets, int32_t* tile_offsets,
                  int32_t* tiles, void* stream);
int mvb_moe_route_ext(const float* logits, int64_t logits_row_stride, int num_tokens, int num_experts, int num_identity, int top, int softmax,
                      const float* correction, float weight_scale, int block_rows, int max_tiles, int32_t* counters, int32_t* ids,
                      float* weights, int32_t* ranks, int32_t* offsets, int32_t* tile_offsets, int32_t* tiles, float* identity_weights,
                      void* stream);
int mvb_moe_gather(int dtype, const void* h, int64_t h_row_stride, const int32_t* ids, const float* weights, const int32_t* ranks,
                   const int32_t* offsets, void* out, int64_t out_row_stride, int32_t* slots, float* row_weights, int num_tokens, int top,
                   int width, void* stream);
int mvb_moe_gemm(int dtype, const void* x, int64_t x_row_stride, int64_t num_rows, const void* weight, int64_t w_row_stride,
                 int num_experts, int m, int k, int gated, float limit, float alpha, float offset, const float* row_weights,
                 const int32_t* num_tiles, const int32_t* tiles, int max_tiles, int block_rows, void* out, int64_t out_row_stride,
                 int32_t* dev_status, void* stream);

/*
 * mvb_state_space: per head, S <- e^(a dt) S + dt B x^T, y = S^T C + D x, dt = softplus(raw + dt_bias); head h uses the B and C of group
 *   h / (heads / groups).  x [num_tokens, heads, vdim], b and c [num_tokens, groups, num_states <= 256] with one row stride; fp32
 *   dt_bias, a_log2e (= a log2(e), a <= 0) and d [heads]; state fp32 [num_slots, heads, num_states, vdim rounded up to 4]; scratch of
 *   mvb_state_space_scratch_bytes (often 0).  longest: tokens of the step's longest sequence, by which a ragged step decides whether to
 *   cut sequences into segments (0: never).
 * mvb_gated_group_norm: out = u / rms(u) * weight with u = y silu(z), the root mean square over each of `groups` equal consecutive parts
 *   of a row of `width`.
 * mvb_row_norm_rope_kv_write: q and k are divided by the root mean square of their whole row (q_dim, k_dim used coordinates) and
 *   multiplied by q_weight, k_weight [heads * head_dim] (both NULL: neither), then rotated (cos_sin NULL: not); v is divided by the root mean square of each
 *   head's v_dim used coordinates (0: not).  q in place; k and v to their cache slots and, with kv_in_place, in place too.
 */
int mvb_state_space(int dtype, const void* x, const void* b, const void* c, int64_t xbc_row_stride, const void* dt, int64_t dt_row_stride,
                    const float* dt_bias, const float* a_log2e, const float* d, void* y, int64_t y_row_stride, float* state,
                    const int32_t* state_slots, int64_t num_slots, const int32_t* cu_seqlens_q, const int64_t* positions, int num_seqs,
                    int num_tokens, int longest, int heads, int groups, int num_states, int vdim, void* scratch, size_t scratch_bytes,
                    int32_t* dev_status, void* stream);
size_t mvb_state_space_scratch_bytes(int dtype, int num_tokens, int num_seqs, int longest, int heads, int num_states, int vdim, int ragged);
int mvb_gated_group_norm(int dtype, const void* y, int64_t y_row_stride, const void* z, int64_t z_row_stride, const float* weight, void* out,
                         int64_t out_row_stride, int rows, int width, int groups, float eps, void* stream);
int mvb_row_norm_rope_kv_write(int dtype, void* q, int64_t q_row_stride, void* k, int64_t k_row_stride, void* v, int64_t v_row_stride,
                               const void* q_weight, const void* k_weight, int q_dim, int k_dim, int v_dim, float eps,
                               const int64_t* positions, const float* cos_sin, int64_t max_pos, const int32_t* slot_mapping, void* k_cache,
                               void* v_cache, int64_t num_slots, int num_tokens, int num_q_heads, int num_kv_heads, int head_dim,
                               int kv_in_place, int32_t* dev_status, void* stream);

#ifdef __cplusplus
}
#endif
#endif /* MINI_VLLM_B200_H_ */
