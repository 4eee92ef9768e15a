// Layer-stack models: a list of layers, each a mixer (latent attention with a sliding window, grouped attention, a
// selective state-space mixer, or a recurrence with a matrix state) and an optional feed-forward (SwiGLU or squared
// relu), with RMS norms before and after every sublayer or a layer norm behind every residual sum, and a block of layers
// that may run several times, each pass with caches and states of its own.  A layer may read the keys and values of an
// earlier one.  The handle (mtj_handle.h) holds what all families share: tokens, positions, sampler, step graph.
#pragma once
#include <array>
#include <map>
#include <string>
#include <tuple>
#include <vector>

#include "mtj_handle.h"
#include "mtj_stack_kernels.h"

namespace mtj {

class LayerStack {
 public:
  // validates the description; on success *out owns a copy of it
  static int32_t create(const mtj_config& cfg, const mtj_stack_desc& desc, int max_pos, LayerStack** out);

  void carve_weights(Carver& c);
  void carve_workspace(Carver& c);
  int32_t bind(mtj_handle* h, cudaStream_t s);          // after both carves: zeroes, tables, tensor maps, the leaf list
  int64_t leaves() const { return leaf_count_; }
  int32_t load_param(mtj_handle* h, const std::string& name, const void* src, int32_t dtype, int32_t ndim,
                     const int64_t* shape, cudaStream_t s);

  // Embedding and all layers for the M rows of `rows`; ids as in EmbedArgs.  hist: positions before the first row that
  // caches may hold (0: none).  decode: one row per sequence.  Leaves the residual stream ready for the logits calls.
  int32_t forward(mtj_handle* h, const uint32_t* ids, int ids_ld, const RowMap& id_rows, int M, const RowMap& rows, int hist,
                  bool decode, cudaStream_t s);
  // final norm + head of the rows of the last forward: contiguous rows, or rows named by a device array
  int32_t logits(mtj_handle* h, int row0, int n, float* out, bool decode, cudaStream_t s);
  int32_t logits_select(mtj_handle* h, const int32_t* rows_dev, int n, float* out, cudaStream_t s);
  int runs() const { return static_cast<int>(runs_.size()); }
  // residual stream after the last forward, [rows][row stride]
  const float* residual(int* ld) const { *ld = ld_; return x_; }
  // layer runs to execute (0 = all), for mtj_k_stack_residual
  int stop_after = 0;

 private:
  struct Linear {                      // bf16 [N, K], rows of ld elements, zero-padded
    __nv_bfloat16* w = nullptr;
    int N = 0, K = 0, ld = 0;
    TensorMap map;
    void shape(int n, int k) { N = n; K = k; ld = static_cast<int>(align_up(k, 8)); }
    void take(Carver& c) { w = c.take<__nv_bfloat16>(align_up(N, 8) * ld); }
  };
  struct Layer {
    mtj_layer_desc d;
    Linear in, out, gate_up, down;     // mixer input and output, feed-forward
    Linear x, dt;                      // mamba1; matrix state with key-channel decay: dt = its second decay projection
    Linear gate2;                      // the second projection of that mixer's output gate
    Linear up;                         // latent attention, expanded form: per head [W_uk, padded] then [W_uv, padded]
    __nv_bfloat16 *uk = nullptr, *uv = nullptr;
    float *norm1 = nullptr, *norm1b = nullptr, *norm2 = nullptr, *norm2b = nullptr, *kv_norm = nullptr;
    float *conv_w = nullptr, *conv_b = nullptr, *dt_b = nullptr, *A = nullptr, *D = nullptr;
    float *norm1_b = nullptr, *norm2_b = nullptr;      // biases of the layer norms
    float *q_norm = nullptr, *k_norm = nullptr;        // grouped attention
    float* mix_norm = nullptr;                         // matrix state: norm of the outputs
    float2* sincos = nullptr;
    int32_t* page_table = nullptr;
    int ring_pages = 0, kv_ld = 0, row_ld = 0, kr_ld = 0, ld_u = 0, ld_xp = 0;
    int key_blocks = 0, k_own = 0, value_blocks = 0;   // key_blocks == 0: sizes outside the tensor-core attention
    int k_cols = 0, v_cols = 0, q_cols = 0;            // grouped attention: columns per cached head, per query head
    // matrix state: channels of the convolution; columns of the input projection's output
    int channels = 0, x0 = 0, a0 = 0, g0 = 0, aux0 = 0, aux = 0;
    TensorMap map_q, map_k, map_kr, map_v;
  };
  struct Run {                         // one execution of a layer, with its own cache or state
    int layer;
    bool first;                        // first layer of a pass
    void* cache = nullptr;
    float *conv_state = nullptr, *ssm_state = nullptr;
    void *k_pool = nullptr, *v_pool = nullptr;         // grouped attention: own, or the run's that it reads
    const int32_t* page_table = nullptr;
    TensorMap map_k, map_v;
    int kv_run = -1;                   // run whose keys and values are used (itself: its index)
  };
  struct Pack {                        // source rows [src0, src0 + n) of a matrix -> packed rows of dst
    int src0, n;
    __nv_bfloat16* dst;
    int ld, r0, gin, gout, csplit, cshift;
  };
  struct Leaf {
    std::vector<int64_t> shape;
    int op;
    void* dst;                         // of the fp32 forms
    int ld;
    std::vector<Pack> packs;           // of kRows
    int64_t id;
  };
  // what follows a sublayer's projection on the few-row path
  struct Post {
    const float *w, *b;
    bool stats;
  };
  enum { kRows, kF32, kNegExp, kTransposeF32 };

  bool use_tc(const mtj_handle* h, int M, bool decode) const;
  const TensorMap* xmap(const __nv_bfloat16* buf, int K, int ld, int M);
  int32_t gemm(mtj_handle* h, GemvEpilogue epi, const Linear& l, const __nv_bfloat16* x, int M, float* out, int ld_out,
               __nv_bfloat16* out_bf16, int ld_bf16, bool decode, cudaStream_t s, int x_row0 = 0, int x_ld = 0, int f32_from = 0);
  int32_t gemm_planes(mtj_handle* h, const Linear& l, const __nv_bfloat16* x, int M, int* planes, bool decode, cudaStream_t s);
  int32_t gemv(mtj_handle* h, GemvEpilogue epi, const Linear& l, const float* x, int ldx, int M, const float* norm, float* out,
               int ld_out, const Post* post, bool pdl, cudaStream_t s, const int32_t* select = nullptr,
               const float* stats = nullptr);
  // a sublayer's input projection: of the normed residual stream, or of the stream itself
  int32_t project_in(mtj_handle* h, const Linear& l, const float* norm, int M, float* out, int ld_out, bool pdl, cudaStream_t s);
  int32_t grouped(mtj_handle* h, const Run& r, int M, const RowMap& rows, bool tc, bool decode, const Post& post, cudaStream_t s);
  int32_t matrix(mtj_handle* h, const Run& r, int M, const RowMap& rows, bool tc, bool decode, const Post& post, cudaStream_t s);
  int32_t mamba(mtj_handle* h, const Run& r, int M, const RowMap& rows, bool tc, bool decode, const Post& post, cudaStream_t s);
  int32_t latent(mtj_handle* h, const Run& r, int M, const RowMap& rows, int hist, bool tc, bool decode, const Post& post,
                 cudaStream_t s);
  int32_t add_leaf(const std::string& name, Leaf leaf);

  int d_ = 0, V_ = 0, ld_ = 0, R_ = 0, max_batch_ = 0, max_pos_ = 0;
  int loop_start_ = 0, loop_stop_ = 0, loop_times_ = 0;
  float mult_ = 1.f, eps_ = 0.f, embed_scale_ = 0.f, softcap_ = 0.f;
  bool post_ln_ = false;               // layer norms behind the residual sums; the sublayers read the stream itself
  bool f32_ = false;                   // 32-bit runs: fp32 activations and caches everywhere
  int tc_min_rows_ = 16;
  std::vector<Layer> layers_;
  std::vector<Run> runs_;
  Linear loop_in_, head_;
  __nv_bfloat16* embed_ = nullptr;
  float *final_norm_ = nullptr, *final_norm_b_ = nullptr, *zeros_ = nullptr;
  std::map<std::pair<double, int>, float2*> tables_;
  std::map<std::string, Leaf> leaf_map_;
  int64_t leaf_count_ = 0;
  char *w_begin_ = nullptr, *w_end_ = nullptr, *s_begin_ = nullptr, *s_end_ = nullptr;

  // workspace, sized for the widest layer
  int rows_a_ = 0, lin_rows_ = 0, ld_p1_ = 0, ld_act_ = 0;
  int64_t xp_planes_elems_ = 0;
  bool last_tc_ = false;
  float *x_ = nullptr, *x0_ = nullptr, *stats_ = nullptr, *cat_ = nullptr, *y_ = nullptr, *p1_ = nullptr, *u_ = nullptr, *xp_ = nullptr,
        *dt_raw_ = nullptr, *gate_raw_ = nullptr, *aux_ = nullptr, *mix_ = nullptr, *q_f32_ = nullptr, *act_ = nullptr, *xp_planes_ = nullptr, *q_abs_ = nullptr, *part_o_ = nullptr, *part_ml_ = nullptr;
  __nv_bfloat16 *xn_bf_ = nullptr, *cat_bf_ = nullptr, *xz_bf_ = nullptr, *u_bf_ = nullptr, *dtr_bf_ = nullptr, *act_bf_ = nullptr,
                *sel_bf_ = nullptr, *q_pack_ = nullptr, *c_lin_ = nullptr, *kr_lin_ = nullptr, *kv_lin_ = nullptr, *gate_bf_ = nullptr;
  char* chunk_records_ = nullptr;
  uint32_t *counters_ = nullptr, *attn_counters_ = nullptr;
  int ld_aux_ = 0, ld_mix_ = 0;
  std::map<std::tuple<const void*, int, int>, std::array<TensorMap, 3>> xmaps_;
};

}  // namespace mtj
