// The prefill attention with sinks, kept first tokens, a bias by distance and head gates: instantiations of their own, so that the
// plain kernel carries none of it and the two compile side by side.
#include "prefill_attn.cuh"

namespace mvb {

int launch_prefill_ext(const PrefillOperands& op, const PrefillParams& p, int head_dim, bool list, int max_seqlen_q, cudaStream_t st) {
  return p.slopes != nullptr ? launch_prefill_form<4>(op, p, head_dim, list, max_seqlen_q, st)
                             : launch_prefill_form<3>(op, p, head_dim, list, max_seqlen_q, st);
}

}  // namespace mvb
