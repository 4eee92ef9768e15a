// Instances of the tensor-core attention over linear key / value matrices with a sliding window: latent attention
// in its expanded form, where a key row is [the head's own columns | columns all heads share] and both parts, like
// the value row, are padded to whole 64-column blocks (mtj_stack.cu builds the matrices).
#include "mtj_attn_tc.cuh"

namespace mtj {

int attn_tc_value_blocks(int vdim) { return vdim <= 64 ? 1 : vdim <= 128 ? 2 : vdim <= 256 ? 4 : 0; }
int attn_tc_key_blocks(int own_dim, int shared_dim) {
  const int n = (own_dim + 63) / 64 + (shared_dim + 63) / 64;
  return n <= 4 ? (n < 2 ? 2 : n) : 0;
}

cudaError_t launch_prefill_attn_tc_linear(const void* map_q, const void* map_k, const void* map_ks, const void* map_v,
                                          int key_blocks, int value_blocks, const PrefillAttnTcArgs& a, cudaStream_t s) {
  if (a.M <= 0 || a.rows.Tc <= 0 || a.M % a.rows.Tc != 0 || a.window <= 0 || a.hist < 0 || a.key_rows < a.hist + a.rows.Tc ||
      a.k_own < 0 || a.k_own > key_blocks)
    return cudaErrorInvalidValue;
  switch (key_blocks * 8 + value_blocks) {
    case 2 * 8 + 1: return launch_attn_tc<2, 1, kLinearRows>(map_q, map_k, map_ks, map_v, a, s);
    case 2 * 8 + 2: return launch_attn_tc<2, 2, kLinearRows>(map_q, map_k, map_ks, map_v, a, s);
    case 2 * 8 + 4: return launch_attn_tc<2, 4, kLinearRows>(map_q, map_k, map_ks, map_v, a, s);
    case 3 * 8 + 1: return launch_attn_tc<3, 1, kLinearRows>(map_q, map_k, map_ks, map_v, a, s);
    case 3 * 8 + 2: return launch_attn_tc<3, 2, kLinearRows>(map_q, map_k, map_ks, map_v, a, s);
    case 3 * 8 + 4: return launch_attn_tc<3, 4, kLinearRows>(map_q, map_k, map_ks, map_v, a, s);
    case 4 * 8 + 1: return launch_attn_tc<4, 1, kLinearRows>(map_q, map_k, map_ks, map_v, a, s);
    case 4 * 8 + 2: return launch_attn_tc<4, 2, kLinearRows>(map_q, map_k, map_ks, map_v, a, s);
    case 4 * 8 + 4: return launch_attn_tc<4, 4, kLinearRows>(map_q, map_k, map_ks, map_v, a, s);
    default: return cudaErrorInvalidValue;
  }
}

}  // namespace mtj
