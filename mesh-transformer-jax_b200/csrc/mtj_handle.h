// The runtime object behind the C ABI, shared by the model families (mtj_model.cu: the entry points and the GPT-J
// layers; mtj_stack.cu: layer-stack models): error reporting, arena carving and the per-handle state.
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

#include <algorithm>
#include <string>
#include <vector>

#include "../../include/mtj_b200.h"
#include "mtj_comm.h"
#include "mtj_common.cuh"
#include "mtj_kernels.h"

extern "C" int32_t mtj_set_error(int32_t code, const char* msg);

namespace mtj {

class LayerStack;      // mtj_stack.h

inline int32_t fail(int32_t code, const std::string& msg) { return mtj_set_error(code, msg.c_str()); }

#define MTJ_CUDA(expr)                                                              \
  do {                                                                              \
    cudaError_t _e = (expr);                                                        \
    if (_e != cudaSuccess)                                                          \
      return fail(MTJ_ERR_CUDA, std::string(#expr) + ": " + cudaGetErrorString(_e)); \
  } while (0)

constexpr int kTcSplitMax = 8;      // split-K factor limit of the small-M out-projection
constexpr int kTcSplitRows = 128;
constexpr int kHiLoRows = 64;       // decode rows that can carry hi + lo activations
constexpr int kTpPipeMinRows = 128; // a chunk is cut in two for all-reduce overlap only if each half keeps this many rows

struct alignas(64) TensorMap { unsigned char bytes[128]; };   // a CUtensorMap

struct LayerWeights {
  __nv_bfloat16* w_in = nullptr;    // [3*dl + ffl, d]  rows: Q | K | V | FF-in
  float* b_ff = nullptr;            // [ffl]
  __nv_bfloat16* w_out = nullptr;   // [d, dl + ffl]    cols: attn vector | gelu(ff)
  float* b_out = nullptr;           // [d]
  float* ln_scale = nullptr;
  float* ln_offset = nullptr;
  TensorMap map_in, map_out;        // TMA views of w_in / w_out for the tensor-core path
  TensorMap map_k, map_v;           // TMA views of this layer's K / V pools as [pages*heads*64, d_head]
};

inline int64_t align_up(int64_t v, int64_t a) { return (v + a - 1) / a * a; }

// Bump allocator over a caller-provided arena; with base == nullptr it only sizes.
struct Carver {
  char* base;
  int64_t off = 0;
  explicit Carver(void* b) : base(static_cast<char*>(b)) {}
  template <typename T>
  T* take(int64_t count) {
    off = align_up(off, 256);
    T* p = base ? reinterpret_cast<T*>(base + off) : nullptr;
    off += count * static_cast<int64_t>(sizeof(T));
    return p;
  }
};

}  // namespace mtj

struct mtj_handle {
  mtj_config cfg;
  int L = 0, d = 0, n_heads = 0, heads = 0, dh = 0, rot = 0, V = 0, Vl = 0, seq = 0, W = 0, mp = 1, rank = 0, dl = 0, ffl = 0;
  int max_batch, max_gen, max_rows, ring_pages = 0, n_pages = 0, max_pos, max_splits = 0;

  // layer-stack families: their layers, caches and states (null: the GPT-J layers below)
  mtj::LayerStack* stack = nullptr;

  // weight arena
  __nv_bfloat16* emb_w = nullptr;
  float* emb_b = nullptr;
  std::vector<mtj::LayerWeights> layers;
  float* lnf_scale = nullptr;
  float* lnf_offset = nullptr;
  __nv_bfloat16* proj_w = nullptr;
  float* proj_b = nullptr;
  float2* sincos = nullptr;
  std::vector<uint8_t> leaf_loaded;   // one mark per parameter leaf (embedding 2, 10 per layer, projection 4)
  int64_t expected = 0;

  // workspace
  float* x = nullptr;
  float* stats = nullptr;
  float* q = nullptr;
  float* act2 = nullptr;
  float* part_o = nullptr;
  float* part_ml = nullptr;
  uint32_t* counters = nullptr;     // attention + gemv tickets (zeroed at bind)
  uint32_t* gemv_counters = nullptr;
  float* logits = nullptr;          // [max_batch, Vl] this shard's logits
  float* logits_all = nullptr;      // [max_batch, V]  (== logits when mp == 1)
  float* logits_gather = nullptr;   // [mp, max_batch, Vl] all-gather landing zone (mp > 1)
  float* part = nullptr;            // [max_rows, d] this shard's partial sums before the all-reduce (mp > 1)
  void* comm = nullptr;             // ncclComm_t over the "shard" axis
  // peer-memory all-reduce for small messages (decode); buffers are cudaMalloc'ed once at set-up
  // because they have to be exportable to the other ranks' processes
  bool p2p_ready = false;
  int p2p_rows = 0;                 // rows a data slot holds
  char* p2p_local = nullptr;        // [2 slots][p2p_rows * d] floats | flags | seq | ticket
  char* p2p_peer[mtj::kP2pMaxWorld] = {};
  size_t p2p_flag_off = 0;
  size_t p2p_recv_off = 0;          // push exchange of the persistent decode kernel
  size_t p2p_push_off = 0;          // receive area of the per-layer push all-reduce [2][mp][p2p_rows][d] floats
  size_t p2p_pflag_off = 0;         // its row flags [mp][p2p_rows]
  size_t p2p_amax_off = 0;          // greedy-token packets [2][mp][p2p_rows][2] uint2
  bool tp_token = true;             // decode at mp > 1: the greedy token is agreed on by pushing each rank's local
                                    // arg-max to all ranks instead of gathering the logits (MTJ_NO_TP_TOKEN=1: off)
  bool tp_push = false;             // batched decode at mp > 1: push all-reduce fused with the split-K reduction and
                                    // the LayerNorm; default: from 4 shards on (MTJ_TP_PUSH=0 / 1 overrides)
  bool xn_ready = false;            // the bf16 operand of the next projection has already been written
  bool tc_cluster_k = true;         // batched decode: split K over block clusters when tiles are few (MTJ_NO_CLUSTER_K=1: off)
  float* uniforms = nullptr;        // [max_batch, V] sampler inputs of the current step
  float* top_p = nullptr;           // [max_batch]
  float* temp = nullptr;            // [max_batch]
  void* sample_scratch = nullptr;
  // tensor-core path (many token rows): bf16 activation operands and their TMA views
  bool tc_ok = false;
  __nv_bfloat16* xn_bf16 = nullptr;   // [max_rows, d] LayerNorm output
  __nv_bfloat16* act_bf16 = nullptr;  // [max_rows, dl + ffl] attention vector | gelu(ff)
  mtj::TensorMap map_xn[3], map_act[3], map_proj, map_q;   // activation views with 32 / 64 / 128-row boxes
  mtj::TensorMap map_xn_wide, map_act_wide;   // 256-row boxes for the persistent GEMM
  __nv_bfloat16* q_bf16 = nullptr;    // [max_rows, dl] rotated queries for the tensor-core attention
  bool attn_tc_ok = false;
  // few-sequence decode: the bf16 rounding errors of the two activation operands (x = hi + lo), rows [0, kHiLoRows)
  __nv_bfloat16* xn_lo = nullptr;
  __nv_bfloat16* act_lo = nullptr;
  mtj::TensorMap map_xn_lo[2], map_act_lo[2];   // 32 / 64-row boxes
  bool hilo_ok = false;
  int tc_hilo_max_b = mtj::kHiLoRows;    // up to this many sequences the activations travel as hi + lo (mtj_config.hilo_max_batch)
  int wait_limit = 1 << 22;         // iteration limit of the bounded device-side waits (mtj_config.wait_limit)
  bool tc_wide_ok = false;   // persistent 128 x 256 GEMM for long chunks
  int tc_pair = 7;           // ... as block pairs on 256 x 256 tiles: bit 0 in-projection, 1 out-projection, 2 logits
                             // (MTJ_TC_PAIR=<mask> overrides, for measurement)
  bool mega_push = true;     // per-block push exchange inside the persistent decode kernel (MTJ_NO_MEGA_PUSH=1: slot protocol)
  float* tc_partial = nullptr;        // [kTcSplitMax, kTcSplitRows, d] split-K partial sums of small-M out-projections
  int eval_rows = 0;                // rows of logits materialised at a time by the loss path
  float* eval_logits = nullptr;     // [eval_rows, Vl]
  // loss path on the persistent GEMM: the logits are never stored, its epilogue leaves per (32-entry vocabulary
  // group, row) the max and the sum of exp, plus the target's logit
  int ce_groups = 0;
  int ce_rows = 0;                  // rows per launch of that GEMM: several 256-row token tiles, so that a block's
                                    // epilogues overlap its next tiles instead of ending the launch
  float* ce_gmax = nullptr;         // [ce_groups, ce_rows]
  float* ce_gsum = nullptr;
  float* ce_tlogit = nullptr;       // [ce_rows]
  uint8_t* ce_ghit = nullptr;       // [ce_rows]
  bool fused_ce = true;             // MTJ_NO_FUSED_CE=1: materialise the logits slice and run ce_partial instead
  float* ce_max = nullptr;          // [max_rows] local max, then global max
  float* ce_lmax = nullptr;         // [max_rows] copy of the local max (mp > 1)
  float* ce_sum = nullptr;          // [max_rows, 2]
  uint8_t* ce_hit = nullptr;        // [max_rows]
  uint32_t* tokens = nullptr;       // [max_batch] next decode input
  int32_t* cur = nullptr;           // absolute position of the next decode token
  int32_t* pad = nullptr;           // [max_batch]
  int32_t* key_limit = nullptr;     // [max_batch]
  int32_t* page_table = nullptr;    // [max_batch, ring_pages]
  int32_t* row_select = nullptr;    // [max_rows]
  uint32_t* dev_err = nullptr;
  uint32_t* rng_seed = nullptr;     // [2] key of the device generator that draws the sampler's uniforms
  int32_t* top_k = nullptr;         // [max_batch] the sampler's top_k, used while has_top_k
  bool has_top_k = false;
  __nv_bfloat16* kpool = nullptr;   // [L][n_pages][heads][kPageTokens][dh]
  __nv_bfloat16* vpool = nullptr;
  int64_t pool_layer_elems = 0;
  bool bound = false;

  // decode state
  std::vector<int32_t> host_pad;    // host copy of `pad` for the running batch
  int min_pad = 0;                  // smallest first-visible position over the running sequences
  // pages a sequence of the running batch holds at most right now (its window start to the decode position)
  int est_pages() const {
    const int cur = W + steps_done;
    const int start = std::max(min_pad, cur - W + 1);
    return cur / mtj::kPageTokens - start / mtj::kPageTokens + 1;
  }
  int batch = 0;
  bool prefilled = false;
  int steps_done = 0;
  int64_t launches = 0;
  bool use_pdl = true;
  int ks_inproj = 0, ks_out = 0, ks_logits = 0;   // K-split overrides (tuning; 0 = automatic)
  // decode of 1-4 sequences on one GPU: the whole step as one persistent kernel
  bool use_mega = true;
  bool mega_token = true;                  // greedy token picked inside the whole-step kernel (MTJ_NO_MEGA_TOKEN=1: separate kernel)
  mtj::MegaLayer* mega_layers = nullptr;   // device copy of the per-layer pointers
  uint32_t* mega_sync = nullptr;           // [5 L + 3] phase counters
  unsigned long long* mega_amax = nullptr; // [4] running maxima of the in-kernel greedy token
  unsigned long long* mega_trace = nullptr;  // [6 L + 3] phase time stamps (profiling read-out)
  bool mega_trace_on = false;
  // decode: attention runs on a side stream next to the FF half of the in-projection
  bool fork_attn = true;
  int mega_max_b = 1;               // sequences the whole-step decode kernel is used for (mtj_config.mega_max_batch, up to 4)
  int tc_decode_min_b = 2;          // from this many sequences on decode takes the tensor-core GEMM path (mtj_config.tc_decode_min_batch)
  bool tc_pdl = true;               // programmatic dependent launch on the tensor-core decode chain (MTJ_NO_TC_PDL=1: off)
  bool fork_pdl = false;            // let the out-projection start early although it also waits on the side stream
  cudaStream_t side_stream = nullptr;
  // tensor-parallel prefill / eval: two row chunks are in flight, the all-reduce of one (on comm_stream)
  // overlapping the layer of the other.  A view = one half of the row-indexed activation buffers.
  struct ActView {
    float *x, *stats, *part, *q;
    __nv_bfloat16 *xn_bf16, *act_bf16, *q_bf16;
    mtj::TensorMap map_xn[3], map_act[3], map_xn_wide, map_act_wide, map_q;
  };
  ActView views[2];
  bool views_ok = false;
  int view_rows[2] = {0, 0};
  cudaStream_t comm_stream = nullptr;
  cudaEvent_t ev_layer[2] = {nullptr, nullptr}, ev_reduced[2] = {nullptr, nullptr};
  bool tp_pipe = false;             // overlap the all-reduce of one chunk with the layer of the next; default: from 4
                                    // shards on (MTJ_TP_PIPE=0 / 1 overrides)
  void save_view(int i) {
    ActView& v = views[i];
    v.x = x; v.stats = stats; v.part = part; v.q = q; v.xn_bf16 = xn_bf16; v.act_bf16 = act_bf16; v.q_bf16 = q_bf16;
    for (int k = 0; k < 3; ++k) { v.map_xn[k] = map_xn[k]; v.map_act[k] = map_act[k]; }
    v.map_xn_wide = map_xn_wide; v.map_act_wide = map_act_wide; v.map_q = map_q;
  }
  void use_view(int i) {
    const ActView& v = views[i];
    x = v.x; stats = v.stats; part = v.part; q = v.q; xn_bf16 = v.xn_bf16; act_bf16 = v.act_bf16; q_bf16 = v.q_bf16;
    for (int k = 0; k < 3; ++k) { map_xn[k] = v.map_xn[k]; map_act[k] = v.map_act[k]; }
    map_xn_wide = v.map_xn_wide; map_act_wide = v.map_act_wide; map_q = v.map_q;
  }
  cudaEvent_t ev_fork = nullptr, ev_join = nullptr;

  // decode step captured once per batch size and replayed (the step counter,
  // tokens and page table live on the device, so the graph never changes)
  bool use_graph = true;
  cudaStream_t capture_stream = nullptr;
  cudaGraphExec_t graph_exec = nullptr;
  int graph_batch = 0;
  int graph_greedy = -1;
  int64_t graph_kernels = 0;

  // optional per-family kernel timing (mtj_profile_*): events around launches
  bool profile = false;
  std::vector<cudaEvent_t> ev_pool;
  size_t ev_used = 0;
  std::vector<std::pair<int, std::pair<size_t, size_t>>> ev_spans;   // (family, (start, stop))

  void prof_begin(int family, cudaStream_t s) {
    if (!profile || ev_used + 2 > ev_pool.size()) return;
    cudaEventRecord(ev_pool[ev_used], s);
    ev_spans.push_back({family, {ev_used, ev_used + 1}});
    ev_used += 2;
  }
  void prof_end(cudaStream_t s) {
    if (!profile || ev_spans.empty()) return;
    cudaEventRecord(ev_pool[ev_spans.back().second.second], s);
  }

  void carve_weights(mtj::Carver& c) {
    emb_w = c.take<__nv_bfloat16>(static_cast<int64_t>(Vl) * d);
    emb_b = c.take<float>(d);
    layers.resize(L);
    for (auto& lw : layers) {
      lw.w_in = c.take<__nv_bfloat16>(static_cast<int64_t>(3 * dl + ffl) * d);
      lw.b_ff = c.take<float>(ffl);
      lw.w_out = c.take<__nv_bfloat16>(static_cast<int64_t>(d) * (dl + ffl));
      lw.b_out = c.take<float>(d);
      lw.ln_scale = c.take<float>(d);
      lw.ln_offset = c.take<float>(d);
    }
    lnf_scale = c.take<float>(d);
    lnf_offset = c.take<float>(d);
    proj_w = c.take<__nv_bfloat16>(static_cast<int64_t>(Vl) * d);
    proj_b = c.take<float>(Vl);
    sincos = c.take<float2>(static_cast<int64_t>(max_pos) * (rot / 2));
  }

  // buffers of the step driver, the sampler and the loss, whatever the layers are
  void carve_common(mtj::Carver& c) {
    const int64_t R = max_rows;
    logits = c.take<float>(static_cast<int64_t>(std::max(max_batch, 1)) * Vl);
    logits_all = logits;
    uniforms = c.take<float>(static_cast<int64_t>(max_batch) * V);
    top_p = c.take<float>(max_batch);
    temp = c.take<float>(max_batch);
    sample_scratch = c.take<char>(mtj::sample_scratch_bytes(max_batch, V));
    eval_rows = static_cast<int>(std::min<int64_t>(R, 256));
    eval_logits = c.take<float>(static_cast<int64_t>(eval_rows) * Vl);
    ce_max = c.take<float>(R);
    ce_lmax = c.take<float>(R);
    ce_sum = c.take<float>(R * 2);
    ce_hit = c.take<uint8_t>(R);
    tokens = c.take<uint32_t>(max_batch);
    cur = c.take<int32_t>(4);
    pad = c.take<int32_t>(max_batch);
    key_limit = c.take<int32_t>(max_batch);
    row_select = c.take<int32_t>(R);
    dev_err = c.take<uint32_t>(4);
    rng_seed = c.take<uint32_t>(4);
    top_k = c.take<int32_t>(max_batch);
  }

  void carve_workspace(mtj::Carver& c) {
    const int64_t R = max_rows;
    carve_common(c);
    x = c.take<float>(R * d);
    stats = c.take<float>(R * 2);
    q = c.take<float>(R * dl);
    act2 = c.take<float>(R * (dl + ffl));
    part_o = c.take<float>(static_cast<int64_t>(max_batch) * heads * max_splits * dh);
    part_ml = c.take<float>(static_cast<int64_t>(max_batch) * heads * max_splits * 2);
    counters = c.take<uint32_t>(static_cast<int64_t>(max_batch) * heads);
    gemv_counters = c.take<uint32_t>(R);
    if (mp > 1) {
      logits_all = c.take<float>(static_cast<int64_t>(max_batch) * V);
      logits_gather = c.take<float>(static_cast<int64_t>(max_batch) * V);
      part = c.take<float>(R * d);
    }
    tc_partial = c.take<float>(static_cast<int64_t>(mtj::kTcSplitMax) * std::min<int64_t>(R, mtj::kTcSplitRows) * d);
    q_bf16 = c.take<__nv_bfloat16>(R * dl);
    xn_bf16 = c.take<__nv_bfloat16>(R * d);
    act_bf16 = c.take<__nv_bfloat16>(R * (dl + ffl));
    xn_lo = c.take<__nv_bfloat16>(std::min<int64_t>(R, mtj::kHiLoRows) * d);
    act_lo = c.take<__nv_bfloat16>(std::min<int64_t>(R, mtj::kHiLoRows) * (dl + ffl));
    ce_groups = 4 * ((Vl + 127) / 128);
    ce_rows = static_cast<int>(std::min<int64_t>(R, 1024));
    ce_gmax = c.take<float>(static_cast<int64_t>(ce_groups) * ce_rows);
    ce_gsum = c.take<float>(static_cast<int64_t>(ce_groups) * ce_rows);
    ce_tlogit = c.take<float>(ce_rows);
    ce_ghit = c.take<uint8_t>(ce_rows);
    mega_layers = c.take<mtj::MegaLayer>(L);
    mega_sync = c.take<uint32_t>(5 * L + 3);
    mega_amax = c.take<unsigned long long>(4);
    mega_trace = c.take<unsigned long long>(6 * L + 3);
    page_table = c.take<int32_t>(static_cast<int64_t>(max_batch) * ring_pages);
    pool_layer_elems = static_cast<int64_t>(n_pages) * heads * mtj::kPageTokens * dh;
    kpool = c.take<__nv_bfloat16>(pool_layer_elems * L);
    vpool = c.take<__nv_bfloat16>(pool_layer_elems * L);
  }

  mtj::KvCache kv(int layer) const {
    mtj::KvCache k;
    k.kpool = kpool + pool_layer_elems * layer;
    k.vpool = vpool + pool_layer_elems * layer;
    k.page_table = page_table;
    k.ring_pages = ring_pages;
    k.pad = pad;
    return k;
  }
};
