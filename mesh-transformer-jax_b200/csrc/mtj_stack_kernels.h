// Launchers of the layer-stack kernels: row norms, latent attention, selective scan (internal to libmtj_b200).
//
// Positions.  A row m of a call sits at frame position rows.pos0 + m % Tc of sequence rows.b0 + m / Tc (RowMap); the
// position inside its own sequence, which these kernels use, is that minus pad[sequence].  Rows before the
// sequence's start (left padding of a batched prompt) have a negative own position: they store nothing in caches and
// states and give finite values.
#pragma once
#include "mtj_kernels.h"

namespace mtj {

template <typename K, typename... A>
cudaError_t launch_pdl(K kernel, dim3 grid, dim3 block, size_t smem, cudaStream_t s, bool pdl, A... args) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = grid;
  cfg.blockDim = block;
  cfg.dynamicSmemBytes = smem;
  cfg.stream = s;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = pdl ? 1 : 0;
  return cudaLaunchKernelEx(&cfg, kernel, args...);
}

// ---- mtj_stack_kernels.cu
// One row per block:  y = sum of the planes;  x += mult * RMSNorm(y) * w_post (y may be null);  then, of the new x:
// stats = (0, 1 / rms), xn = RMSNorm(x) * w_next in bf16, and cat = [x | x0] for the projection at the start of a pass.
struct ResidualNormArgs {
  float* x;                    // [M, ld]; columns d .. ld - 1 of every buffer here are zero
  int M, d, ld;
  const float* y;              // [planes, M, ld] or null
  int planes;
  const float* w_post;         // [ld]
  float mult, eps;
  float* stats;                // [M, 2] or null
  const float* w_next;         // [ld], with xn
  __nv_bfloat16* xn;           // [M, ld] or null
  const float* x0;             // [M, ld], with cat_*
  float* cat_f32;              // [M, 2 ld] or null
  __nv_bfloat16* cat_bf16;     // [M, 2 ld] or null
};
cudaError_t launch_residual_norm(const ResidualNormArgs& a, cudaStream_t s, bool pdl);
// One row per block:  x = LayerNorm(alpha * x + y) * w + b;  then xn = x in bf16, or, with w_next, the layer norm of the
// new x in bf16, and its (mean, 1 / deviation) into stats.  y == null: x stays, only what follows is done.
struct ResidualLayerNormArgs {
  float* x;                    // [M, ld]; columns d .. ld - 1 of every buffer here are zero
  int M, d, ld;
  const float* y;              // [M, ld] or null
  const float *w, *b;          // [ld]
  float alpha, eps;
  __nv_bfloat16* xn;           // [M, ld] or null
  const float *w_next, *b_next;  // [ld] or null
  float* stats;                // [M, 2] or null
};
cudaError_t launch_residual_layernorm(const ResidualLayerNormArgs& a, cudaStream_t s, bool pdl);
cudaError_t launch_gather_rows_bf16(const __nv_bfloat16* src, int ld, const int32_t* rows, int n, __nv_bfloat16* dst,
                                    cudaStream_t s);
// src [N, K] (bf16 or fp32) -> bf16 dst[(r0 + n / gin * gout + n % gin) * ld + (k < csplit ? k : k + cshift)]
cudaError_t launch_pack_rows(const void* src, int src_is_bf16, int N, int K, __nv_bfloat16* dst, int ld, int r0, int gin,
                             int gout, int csplit, int cshift, cudaStream_t s);
// fp32 dst[i] = -exp(src[i])
cudaError_t launch_neg_exp(const void* src, int src_is_bf16, int64_t n, float* dst, cudaStream_t s);
// src [N, K] -> fp32 dst [K, ld]
cudaError_t launch_transpose_f32(const void* src, int src_is_bf16, int N, int K, float* dst, int ld, cudaStream_t s);
// dst = src, n fp32 elements (a multiple of four)
cudaError_t launch_copy_rows(const float* src, float* dst, int64_t n, cudaStream_t s, bool pdl);

// ---- mtj_latent_attn.cu: attention over a cached latent (and one rotated key part) shared by all heads
struct LatentCache {
  void* pool;                  // [pages][kPageTokens][row_ld] bf16 or fp32: latent (kv_ld columns) | rotated part
  int f32;                     // element type of the pool
  const int32_t* page_table;   // [sequences][ring_pages]; ring slot of own position p: (p / kPageTokens) % ring_pages
  int ring_pages, row_ld, kv_ld;
};
struct LatentArgs {
  int M, heads, dim, rot, vdim, rank, window;
  float scale, eps;
  RowMap rows;
  const int32_t* pad;
  LatentCache cache;
  const float2* sincos;        // [positions][rot / 2] = (sin, cos)
  const float* p1;             // [M, ld_p1] fp32: q head by head [dim | rot], then latent | rotated part
  int ld_p1;
  const float* kv_norm;        // [rank]
  const __nv_bfloat16* w_uk;   // [heads * dim, kv_ld]
  const __nv_bfloat16* w_uv;   // [heads * vdim, kv_ld]
  // absorbed form (few rows, fp32 runs): q' = W_uk^T q, scores against the latent itself
  float* q_abs;                // [M, heads, row_ld], scaled
  int tensor_cores;            // bf16 queries and weights on the tensor cores are allowed
  int splits;                  // key ranges per row
  float* part_o;               // [M, heads, splits, kv_ld]
  float* part_ml;              // [M, heads, splits, 2]
  float* out;                  // [M, ld_out] or null
  __nv_bfloat16* out_bf16;     // [M, ld_out] or null
  int ld_out;
  // expanded form (many rows): operands of the tensor-core attention
  __nv_bfloat16* q_pack;       // [M, heads * 64 * key_blocks]
  int key_blocks, k_own;
  __nv_bfloat16* c_lin;        // [sequences * key_rows, kv_ld] latents of the history and the chunk
  __nv_bfloat16* kr_lin;       // [sequences * key_rows, kr_ld] their rotated parts, zero-padded
  int kr_ld, hist, key_rows, nseq;
};
// normalises and caches the latent, rotates and caches the key part, rotates and absorbs the queries
cudaError_t launch_latent_absorb(const LatentArgs& a, cudaStream_t s, bool pdl);
cudaError_t launch_latent_attn(const LatentArgs& a, cudaStream_t s, bool pdl);
// merges the key ranges and applies W_uv
cudaError_t launch_latent_out(const LatentArgs& a, cudaStream_t s, bool pdl);
// the same caching, with the queries packed for the tensor-core attention and the latents copied to c_lin / kr_lin;
// the second fills the history rows from the cache
cudaError_t launch_latent_pack(const LatentArgs& a, cudaStream_t s);
cudaError_t launch_latent_history(const LatentArgs& a, cudaStream_t s);
constexpr int kLatentMaxRank = 1024;
constexpr int kLatentBlocks = 592;       // most (rows x splits x head groups) a call spreads over beyond one per row
int latent_attn_splits(int M, int heads, int row_ld, int tensor_cores, int window);

// ---- mtj_grouped_attn.cu: softmax attention of query heads over shared key / value heads, causal or windowed
struct GroupedCache {
  void *k, *v;                 // [pages][kPageTokens][kv_heads * up8(dim)] | [..][kv_heads * up8(vdim)], bf16 or fp32
  int f32;
  const int32_t* page_table;   // [sequences][ring_pages]; ring slot of own position p: (p / kPageTokens) % ring_pages
  int ring_pages, k_ld, v_ld;
};
struct GroupedAttnArgs {
  int M, heads, kv_heads, dim, vdim, window;
  float scale, eps;
  float q_temp_coef;
  double q_temp_every;         // 0: no temperature
  RowMap rows;
  const int32_t* pad;
  GroupedCache cache;
  const float* p1;             // [M, ld_p1] q | k | v (only q where own_kv is 0)
  int ld_p1, own_kv;
  const float *q_norm, *k_norm;
  // queries, normed and scaled by the temperature: bf16 heads of q_cols columns, zero-padded, or fp32 heads of up8(dim)
  __nv_bfloat16* q_bf16;
  float* q_f32;
  int q_cols;
  int splits;                  // key ranges per row
  float* part_o;               // [M, heads, splits, vdim]
  float* part_ml;              // [M, heads, splits, 2]
  uint32_t* counters;          // [M * kv_heads * ceil(heads / kv_heads / 8)], zero between launches
  float* out;                  // [M, ld_out] or null
  __nv_bfloat16* out_bf16;     // [M, ld_out] or null
  int ld_out;
};
// norms the queries and keys, writes the queries and, into the cache, keys and values
cudaError_t launch_grouped_prep(const GroupedAttnArgs& a, cudaStream_t s, bool pdl);
// every row of the call by itself, from the cache
cudaError_t launch_grouped_attn(const GroupedAttnArgs& a, cudaStream_t s, bool pdl);
constexpr int kGroupedMaxDim = 512;
constexpr int kGroupedBlocks = 2368;     // most (rows x key heads x splits) a call spreads over beyond one per row and head
int grouped_attn_splits(int M, int heads, int kv_heads, int window);
int grouped_counters(int heads, int kv_heads);   // per row

// ---- mtj_matrix_state.cu: recurrences whose state is a matrix per head, keys x values
//   SSD    S <- exp(A dt) S + dt k v^T,  o = S^T q + D v, with dt = softplus(decay + decay_b) per head
//   delta  S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q, with unit k and q (q times q_scale),
//          g = exp(A softplus(decay + decay_b)) per head and key channel, beta = sigmoid
// the outputs' norm and gate: parts of part_n neighbouring columns, each by its own root mean square;
// gate_first: RMSNorm(y * silu(gate)) * w[column], else RMSNorm(y) * w[column within the part] * sigmoid(gate)
struct GatedNormArgs {
  int M, parts, part_n, gate_first;
  float eps;
  const float* y;              // [M, ld_y]
  int ld_y;
  const void* gate;            // [M, ld_gate], fp32 or bf16
  int gate_bf16, ld_gate;
  const float* w;
  float* out;                  // [M, ld_out] or null
  __nv_bfloat16* out_bf16;
  int ld_out;
};
struct MatrixStateArgs {
  int M, heads, key_heads, dim, vdim;
  int delta;
  RowMap rows;
  int nseq;
  const int32_t* pad;
  const void* u;               // [M, ld_u] convolved keys, queries and values at columns k0, q0, v0; fp32 or bf16
  int u_bf16, ld_u, q0, k0, v0;
  const float* decay;          // [M, ld_decay]
  int ld_decay;
  const float* decay_b;        // [heads] | [heads * dim]
  const float* A;              // [heads], negative
  const float* beta;           // [M, ld_beta], delta
  int ld_beta;
  const float* D;              // [heads], SSD
  float q_scale;
  float* state;                // [slots][heads][dim][vdim]
  float* out;                  // [M, ld_out]
  int ld_out;
  void* chunk_records;         // launch_matrix_chunks: nseq * ceil(Tc / kMatrixChunk) * matrix_chunk_bytes, 16-byte aligned
  uint32_t* dev_err;
};
// row by row
cudaError_t launch_matrix_scan(const MatrixStateArgs& a, cudaStream_t s, bool pdl);
// one row per sequence; with `norm`, if matrix_step_norms(a), the norm and gate of the outputs too (out is not written)
cudaError_t launch_matrix_step(const MatrixStateArgs& a, const GatedNormArgs* norm, cudaStream_t s, bool pdl);
bool matrix_step_ok(const MatrixStateArgs& a);      // sizes that kernel takes
bool matrix_step_norms(const MatrixStateArgs& a);
// ---- mtj_matrix_chunk.cu: the same over long prompts, in chunks on the tensor cores (bf16 operands)
constexpr int kMatrixChunk = 16;
int64_t matrix_chunk_bytes(int heads, int key_heads, int dim, int delta);     // of chunk_records, per chunk of a sequence
cudaError_t launch_matrix_chunks(const MatrixStateArgs& a, cudaStream_t s);
cudaError_t launch_gated_norm(const GatedNormArgs& a, cudaStream_t s, bool pdl);
constexpr int kMatrixMaxDim = 256;

// ---- mtj_ssm.cu: causal convolution and selective scan with carried state
struct SsmArgs {
  int M, inner, state, taps, dt_rank;
  RowMap rows;
  int nseq;                    // sequences in the call
  const int32_t* pad;
  const void* xz;              // [M, ld_xz] x | z (z at column z0), fp32 or bf16
  int xz_bf16, ld_xz, z0;
  const float* conv_w;         // [taps, ld_u]
  const float* conv_b;         // [ld_u]
  float* conv_state;           // [slots][taps - 1][ld_u]
  float* u;                    // [M, ld_u] or null
  __nv_bfloat16* u_bf16;       // [M, ld_u] or null
  int ld_u;
  const float* xp;             // [M, ld_xp] dt | B | C
  int ld_xp;
  // launch_ssm_split: xp_out (= xp) and dtr_bf16 [M, ld_dtr], its dt part, from [planes, M, dt_rank + 2 state]
  const float* xp_planes;
  int planes;
  float* xp_out;
  __nv_bfloat16* dtr_bf16;
  int ld_dtr;
  const float* dt_raw;         // [M, ld_u] W_dt dt, before the bias; null in a step: the step projects itself
  const __nv_bfloat16* w_dt;   // [inner, ld_wdt] (step)
  int ld_wdt;
  const float* dt_b;
  const float* A;              // [inner, state], negative
  const float* D;
  float* ssm_state;            // [slots][inner][state]
  float* out;                  // [M, ld_u] or null
  __nv_bfloat16* out_bf16;     // [M, ld_u] or null
};
// u = silu(conv(x) + b) for all rows, then the taps - 1 last inputs of every sequence into conv_state
cudaError_t launch_ssm_conv(const SsmArgs& a, cudaStream_t s, bool pdl);
cudaError_t launch_ssm_split(const SsmArgs& a, cudaStream_t s, bool pdl);
// the recurrence over the rows of every sequence, from and to ssm_state, with the gate
cudaError_t launch_ssm_scan(const SsmArgs& a, cudaStream_t s);
// one row per sequence: step size, recurrence and gate in one kernel
cudaError_t launch_ssm_step(const SsmArgs& a, cudaStream_t s, bool pdl);
constexpr int kSsmMaxState = 256;

}  // namespace mtj
