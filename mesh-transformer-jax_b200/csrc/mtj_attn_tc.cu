// The paged instance of the tensor-core attention (GPT-J, d_head 256); the kernel is in mtj_attn_tc.cuh.
#include "mtj_attn_tc.cuh"

namespace mtj {

cudaError_t launch_prefill_attn_tc(const void* map_q, const void* map_k, const void* map_v,
                                   const PrefillAttnTcArgs& a, cudaStream_t s) {
  if (a.M <= 0 || a.rows.Tc <= 0 || a.M % a.rows.Tc != 0 || a.d_head != 256) return cudaErrorInvalidValue;
  return launch_attn_tc<4, 4, kPagedHeads>(map_q, map_k, map_k, map_v, a, s);
}

}  // namespace mtj
