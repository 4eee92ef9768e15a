// Instances of the tensor-core attention over paged rows: query heads in groups over key heads that lie side by side in
// the rows of the cache.  A head's 64-column blocks may reach into its neighbour's columns (and past the row's end,
// where TMA fills zeros): the queries are zero there, and output columns past the head's are not stored.
#include "mtj_attn_tc.cuh"

namespace mtj {

int attn_tc_grouped_blocks(int dim) { return dim <= 64 ? 1 : dim <= 128 ? 2 : dim <= 256 ? 4 : 0; }

cudaError_t launch_prefill_attn_tc_grouped(const void* map_q, const void* map_k, const void* map_v, int key_blocks,
                                           int value_blocks, const PrefillAttnTcArgs& a, cudaStream_t s) {
  if (a.M <= 0 || a.rows.Tc <= 0 || a.M % a.rows.Tc != 0 || a.window <= 0 || a.kv_group <= 0 || (a.k_cols & 7) || (a.v_ld & 7) ||
      a.k_cols <= 0 || a.v_ld < a.v_cols || a.rows.pos0_dev)
    return cudaErrorInvalidValue;
  switch (key_blocks * 8 + value_blocks) {
    case 1 * 8 + 1: return launch_attn_tc<1, 1, kPagedRows>(map_q, map_k, map_k, map_v, a, s);
    case 1 * 8 + 2: return launch_attn_tc<1, 2, kPagedRows>(map_q, map_k, map_k, map_v, a, s);
    case 1 * 8 + 4: return launch_attn_tc<1, 4, kPagedRows>(map_q, map_k, map_k, map_v, a, s);
    case 2 * 8 + 1: return launch_attn_tc<2, 1, kPagedRows>(map_q, map_k, map_k, map_v, a, s);
    case 2 * 8 + 2: return launch_attn_tc<2, 2, kPagedRows>(map_q, map_k, map_k, map_v, a, s);
    case 2 * 8 + 4: return launch_attn_tc<2, 4, kPagedRows>(map_q, map_k, map_k, map_v, a, s);
    case 4 * 8 + 1: return launch_attn_tc<4, 1, kPagedRows>(map_q, map_k, map_k, map_v, a, s);
    case 4 * 8 + 2: return launch_attn_tc<4, 2, kPagedRows>(map_q, map_k, map_k, map_v, a, s);
    case 4 * 8 + 4: return launch_attn_tc<4, 4, kPagedRows>(map_q, map_k, map_k, map_v, a, s);
    default: return cudaErrorInvalidValue;
  }
}

}  // namespace mtj
