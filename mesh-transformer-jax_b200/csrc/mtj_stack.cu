// Host side of layer-stack models: description, weight layout, caches and states, and the kernel sequences.
//
// Two forms of every layer, as for GPT-J:
//   few rows (one sequence decoding, short portions) and 32-bit runs: fp32 activations through the weight-streaming
//     GEMV family -- RMSNorm in the prologue, SwiGLU / squared relu / norm + residual + next statistics in the
//     epilogue --, latent attention in its absorbed form, grouped attention row by row, one-row recurrences;
//   many rows, or several sequences decoding: bf16 operands through the tcgen05 GEMMs, attention on the tensor cores
//     (latent: expanded to per-head keys and values, or absorbed in decode), the scans over whole sequences.
// The residual stream, norms, scores, decays and states are fp32 in both.
#include "mtj_stack.h"

#include <math.h>
#include <stdlib.h>

namespace mtj {

namespace {
int up8(int64_t v) { return static_cast<int>(align_up(v, 8)); }
int up4(int v) { return (v + 3) & ~3; }
constexpr int kAbsorbRows = 256;       // rows of the absorbed attention's scratch
constexpr int kSelectGemvRows = 4;
constexpr int kChunkedRows = 2 * kMatrixChunk;   // rows of a sequence from which matrix-state mixers work in chunks
}  // namespace

int32_t LayerStack::create(const mtj_config& cfg, const mtj_stack_desc& desc, int max_pos, LayerStack** out) {
  if (desc.n_layers <= 0 || !desc.layers) return fail(MTJ_ERR_INVALID, "a stack needs layers");
  if (desc.loop_times < 0 || (desc.loop_times > 0 && (desc.loop_start < 0 || desc.loop_stop <= desc.loop_start ||
                                                      desc.loop_stop > desc.n_layers)))
    return fail(MTJ_ERR_INVALID, "loop must name a range of layers");
  LayerStack st;
  st.d_ = cfg.d_model;
  st.V_ = cfg.n_vocab;
  st.ld_ = up8(cfg.d_model);
  st.R_ = cfg.max_rows;
  st.max_batch_ = cfg.max_batch;
  st.max_pos_ = max_pos;
  st.loop_start_ = desc.loop_start;
  st.loop_stop_ = desc.loop_stop;
  st.loop_times_ = desc.loop_times;
  st.mult_ = desc.residual_mult;
  st.eps_ = desc.norm_eps;
  st.embed_scale_ = desc.embed_scale;
  st.softcap_ = desc.logit_softcap;
  if (desc.residual != MTJ_RESIDUAL_SANDWICH_RMS && desc.residual != MTJ_RESIDUAL_POST_LN) return fail(MTJ_ERR_UNSUPPORTED, "unknown residual form");
  st.post_ln_ = desc.residual == MTJ_RESIDUAL_POST_LN;
  if (st.post_ln_ && desc.loop_times > 0) return fail(MTJ_ERR_UNSUPPORTED, "loops are for the sandwich residual form");
  if (!(desc.logit_softcap >= 0.f)) return fail(MTJ_ERR_INVALID, "logit_softcap must not be negative");
  st.f32_ = desc.act_f32 != 0;
  if (desc.tc_min_rows > 0) st.tc_min_rows_ = desc.tc_min_rows;
  if (st.ld_ > 24576) return fail(MTJ_ERR_UNSUPPORTED, "width up to 24576");
  for (int i = 0; i < desc.n_layers; ++i) {
    Layer l;
    l.d = desc.layers[i];
    const mtj_layer_desc& m = l.d;
    const std::string at = "layer " + std::to_string(i) + ": ";
    if (m.ff < 0) return fail(MTJ_ERR_INVALID, at + "feed-forward width");
    if (m.mixer == MTJ_MIXER_LATENT_ATTENTION) {
      if (m.heads <= 0 || m.dim <= 0 || m.rot_dim < 0 || (m.rot_dim & 1) || m.vdim <= 0 || m.kv_rank <= 0 || m.window <= 0)
        return fail(MTJ_ERR_INVALID, at + "latent attention sizes");
      if (m.kv_rank > kLatentMaxRank || m.rot_dim > 1024 || m.dim > 1024)
        return fail(MTJ_ERR_UNSUPPORTED, at + "latent attention takes kv_rank, dim and rot_dim up to 1024");
      l.in.shape(m.heads * (m.dim + m.rot_dim) + m.kv_rank + m.rot_dim, st.d_);
      l.out.shape(st.d_, m.heads * m.vdim);
      l.kv_ld = up8(m.kv_rank);
      l.row_ld = l.kv_ld + up8(m.rot_dim);
      l.k_own = (m.dim + 63) / 64;
      l.value_blocks = attn_tc_value_blocks(m.vdim);
      l.key_blocks = l.value_blocks ? attn_tc_key_blocks(m.dim, m.rot_dim) : 0;
      if (l.key_blocks && !st.f32_) {
        l.kr_ld = 64 * std::max(1, l.key_blocks - l.k_own);
        l.up.shape(m.heads * 64 * (l.k_own + l.value_blocks), m.kv_rank);
      }
      const int window = std::min(m.window, max_pos);
      const int all = (max_pos + kPageTokens - 1) / kPageTokens;
      const int ring = (window - 1 + std::min(st.R_, max_pos) + kPageTokens - 1) / kPageTokens + 1;
      l.ring_pages = std::min(all, ring);
    } else if (m.mixer == MTJ_MIXER_MAMBA1) {
      if (m.inner <= 0 || m.state <= 0 || m.conv <= 0 || m.dt_rank <= 0) return fail(MTJ_ERR_INVALID, at + "state-space sizes");
      if (m.state > kSsmMaxState || m.conv > 64 || m.dt_rank > 8192)
        return fail(MTJ_ERR_UNSUPPORTED, at + "state-space mixers take state up to 256, conv up to 64, dt_rank up to 8192");
      l.in.shape(up8(m.inner) + m.inner, st.d_);      // x rows, zero rows up to a multiple of 8, z rows
      l.out.shape(st.d_, m.inner);
      l.x.shape(m.dt_rank + 2 * m.state, m.inner);
      l.dt.shape(m.inner, m.dt_rank);
      l.ld_u = up8(m.inner);
      l.ld_xp = up8(m.dt_rank + 2 * m.state);
    } else if (m.mixer == MTJ_MIXER_GROUPED_ATTENTION) {
      if (m.heads <= 0 || m.kv_heads <= 0 || m.heads % m.kv_heads || m.dim <= 0 || m.vdim <= 0)
        return fail(MTJ_ERR_INVALID, at + "attention sizes");
      if (m.dim > kGroupedMaxDim || m.vdim > kGroupedMaxDim) return fail(MTJ_ERR_UNSUPPORTED, at + "attention takes dim and vdim up to 512");
      if (!(m.q_temp_every >= 0.0)) return fail(MTJ_ERR_INVALID, at + "q_temp_every");
      if (m.kv_from >= 0) {
        const Layer* src = m.kv_from < i ? &st.layers_[m.kv_from] : nullptr;
        if (!src || src->d.mixer != MTJ_MIXER_GROUPED_ATTENTION || src->d.kv_from >= 0 || src->d.kv_heads != m.kv_heads ||
            src->d.dim != m.dim || src->d.vdim != m.vdim)
          return fail(MTJ_ERR_INVALID, at + "kv_from must name an earlier attention layer with keys and values of its own and the same head sizes");
      }
      l.in.shape(m.heads * m.dim + (m.kv_from >= 0 ? 0 : m.kv_heads * (m.dim + m.vdim)), st.d_);
      l.out.shape(st.d_, m.heads * m.vdim);
      l.k_cols = up8(m.dim);
      l.v_cols = up8(m.vdim);
      l.value_blocks = st.f32_ ? 0 : attn_tc_grouped_blocks(m.vdim);
      l.key_blocks = l.value_blocks ? attn_tc_grouped_blocks(m.dim) : 0;
      l.q_cols = l.key_blocks ? 64 * l.key_blocks : up8(m.dim);
      l.ring_pages = (max_pos + kPageTokens - 1) / kPageTokens;
    } else if (m.mixer == MTJ_MIXER_MATRIX_STATE_SSD || m.mixer == MTJ_MIXER_MATRIX_STATE_DELTA) {
      const bool ssd = m.mixer == MTJ_MIXER_MATRIX_STATE_SSD;
      if (m.heads <= 0 || m.kv_heads <= 0 || m.heads % m.kv_heads || m.vdim <= 0 || m.dim <= 0 || m.conv <= 0 ||
          (ssd ? m.norm_groups <= 0 || (m.heads * m.vdim) % m.norm_groups : m.decay_rank <= 0 || m.gate_rank <= 0))
        return fail(MTJ_ERR_INVALID, at + "matrix-state sizes");
      if (m.dim > kMatrixMaxDim || m.conv > 64) return fail(MTJ_ERR_UNSUPPORTED, at + "matrix states take key sizes up to 256, conv up to 64");
      const int inner = m.heads * m.vdim, keys = m.kv_heads * m.dim;
      l.channels = inner + 2 * keys;
      l.ld_u = up8(l.channels);
      if (ssd) {                                        // z | values, keys, queries | step sizes, each from a multiple of 8 on
        l.x0 = up8(inner);
        l.aux0 = l.x0 + l.ld_u;
      } else {                                          // queries, keys, values | decay rank | gate rank | update strengths
        l.a0 = l.ld_u;
        l.g0 = l.a0 + up8(m.decay_rank);
        l.aux0 = l.g0 + up8(m.gate_rank);
        l.dt.shape(m.heads * m.dim, m.decay_rank);
        l.gate2.shape(inner, m.gate_rank);
      }
      l.aux = m.heads;
      l.in.shape(l.aux0 + l.aux, st.d_);
      l.out.shape(st.d_, inner);
    } else {
      return fail(MTJ_ERR_UNSUPPORTED, at + "unknown mixer");
    }
    if (m.ff > 0) {
      if (m.ff_kind != MTJ_FF_SWIGLU && m.ff_kind != MTJ_FF_SQUARED_RELU) return fail(MTJ_ERR_UNSUPPORTED, at + "unknown feed-forward");
      l.gate_up.shape(m.ff_kind == MTJ_FF_SWIGLU ? 2 * m.ff : m.ff, st.d_);
      l.down.shape(st.d_, m.ff);
    }
    st.layers_.push_back(l);
  }
  auto add = [&](int from, int to, bool pass) {
    for (int i = from; i < to; ++i) {
      Run r;
      r.layer = i;
      r.first = pass && i == from;
      st.runs_.push_back(r);
    }
  };
  if (st.loop_times_ > 0) {
    add(0, st.loop_start_, false);
    for (int t = 0; t < st.loop_times_; ++t) add(st.loop_start_, st.loop_stop_, true);
    add(st.loop_stop_, desc.n_layers, false);
    st.loop_in_.shape(st.d_, 2 * st.ld_);           // [x, padded | x0, padded]
  } else {
    add(0, desc.n_layers, false);
  }
  for (size_t i = 0; i < st.runs_.size(); ++i) {
    const mtj_layer_desc& m = st.layers_[st.runs_[i].layer].d;
    st.runs_[i].kv_run = static_cast<int>(i);
    if (m.mixer != MTJ_MIXER_GROUPED_ATTENTION || m.kv_from < 0) continue;
    int src = static_cast<int>(i) - 1;                  // the latest run of that layer
    while (src >= 0 && st.runs_[src].layer != m.kv_from) --src;
    if (src < 0) return fail(MTJ_ERR_INVALID, "kv_from names a layer that has not run");
    st.runs_[i].kv_run = src;
  }
  st.head_.shape(st.V_, st.d_);
  *out = new LayerStack(st);
  return MTJ_OK;
}

void LayerStack::carve_weights(Carver& c) {
  w_begin_ = c.base ? c.base + c.off : nullptr;
  embed_ = c.take<__nv_bfloat16>(static_cast<int64_t>(V_) * d_);
  final_norm_ = c.take<float>(ld_);
  if (post_ln_) final_norm_b_ = c.take<float>(ld_);
  zeros_ = c.take<float>(ld_);
  head_.take(c);
  if (loop_times_ > 0) loop_in_.take(c);
  tables_.clear();
  for (Layer& l : layers_) {
    const mtj_layer_desc& m = l.d;
    l.norm1 = c.take<float>(ld_);
    (post_ln_ ? l.norm1_b : l.norm1b) = c.take<float>(ld_);
    l.in.take(c);
    l.out.take(c);
    if (m.mixer == MTJ_MIXER_LATENT_ATTENTION) {
      l.kv_norm = c.take<float>(l.kv_ld);
      l.uk = c.take<__nv_bfloat16>(static_cast<int64_t>(m.heads) * m.dim * l.kv_ld);
      l.uv = c.take<__nv_bfloat16>(static_cast<int64_t>(m.heads) * m.vdim * l.kv_ld);
      if (l.up.N) l.up.take(c);
      float2*& t = tables_[{m.rot_base, m.rot_dim}];
      if (!t) t = c.take<float2>(std::max<int64_t>(1, static_cast<int64_t>(max_pos_) * (m.rot_dim / 2)));
      l.sincos = t;
    } else if (m.mixer == MTJ_MIXER_GROUPED_ATTENTION) {
      l.q_norm = c.take<float>(m.heads * m.dim);
      if (m.kv_from < 0) l.k_norm = c.take<float>(m.kv_heads * m.dim);
    } else if (m.mixer == MTJ_MIXER_MATRIX_STATE_SSD || m.mixer == MTJ_MIXER_MATRIX_STATE_DELTA) {
      const bool ssd = m.mixer == MTJ_MIXER_MATRIX_STATE_SSD;
      if (!ssd) {
        l.dt.take(c);
        l.gate2.take(c);
      }
      l.conv_w = c.take<float>(static_cast<int64_t>(m.conv) * l.ld_u);
      l.conv_b = c.take<float>(l.ld_u);
      l.dt_b = c.take<float>(ssd ? m.heads : static_cast<int64_t>(m.heads) * m.dim);
      l.A = c.take<float>(m.heads);
      if (ssd) l.D = c.take<float>(m.heads);
      l.mix_norm = c.take<float>(ssd ? static_cast<int64_t>(m.heads) * m.vdim : m.vdim);
    } else {
      l.x.take(c);
      l.dt.take(c);
      l.conv_w = c.take<float>(static_cast<int64_t>(m.conv) * l.ld_u);
      l.conv_b = c.take<float>(l.ld_u);
      l.dt_b = c.take<float>(l.ld_u);
      l.A = c.take<float>(static_cast<int64_t>(m.inner) * m.state);
      l.D = c.take<float>(l.ld_u);
    }
    if (m.ff > 0) {
      l.norm2 = c.take<float>(ld_);
      (post_ln_ ? l.norm2_b : l.norm2b) = c.take<float>(ld_);
      l.gate_up.take(c);
      l.down.take(c);
    }
  }
  w_end_ = c.base ? c.base + c.off : nullptr;
}

void LayerStack::carve_workspace(Carver& c) {
  const int64_t R = R_;
  s_begin_ = c.base ? c.base + c.off : nullptr;
  rows_a_ = static_cast<int>(std::min<int64_t>(R, kAbsorbRows));
  int64_t p1 = 8, act = 8, u = 0, xp = 0, dtr = 0, xz = 0, qabs = 0, po = 0, ml = 0, qp = 0, cl = 0, kr = 0, kv = 0, hist = 0;
  int64_t dtw = 0, gate = 0, aux = 0, mix = 0, qf = 0, gpo = 0, gml = 0, cnt = 0, rec = 0;
  for (const Layer& l : layers_) {
    const mtj_layer_desc& m = l.d;
    p1 = std::max<int64_t>(p1, up8(l.in.N));
    act = std::max<int64_t>({act, l.out.ld, l.down.ld});
    if (m.mixer == MTJ_MIXER_MAMBA1) {
      u = std::max<int64_t>(u, l.ld_u);
      xp = std::max<int64_t>(xp, l.ld_xp);
      dtr = std::max<int64_t>(dtr, l.dt.ld);
      xz = std::max<int64_t>(xz, up8(l.in.N));
      dtw = std::max<int64_t>(dtw, l.ld_u);
    } else if (m.mixer == MTJ_MIXER_GROUPED_ATTENTION) {
      // the partial results of a call's rows: at most max(rows, kGroupedBlocks / (key heads)) rows times key ranges
      const int64_t rs = std::max<int64_t>(rows_a_, kGroupedBlocks / m.kv_heads + 1);
      gpo = std::max<int64_t>(gpo, rs * m.heads * m.vdim);
      gml = std::max<int64_t>(gml, rs * m.heads * 2);
      cnt = std::max<int64_t>(cnt, static_cast<int64_t>(rows_a_) * grouped_counters(m.heads, m.kv_heads));
      if (l.key_blocks) qp = std::max<int64_t>(qp, static_cast<int64_t>(m.heads) * l.q_cols);
      else qf = std::max<int64_t>(qf, static_cast<int64_t>(m.heads) * l.q_cols);
    } else if (m.mixer == MTJ_MIXER_MATRIX_STATE_SSD || m.mixer == MTJ_MIXER_MATRIX_STATE_DELTA) {
      u = std::max<int64_t>(u, l.ld_u);
      xz = std::max<int64_t>(xz, up8(l.in.N));
      aux = std::max<int64_t>(aux, up8(l.aux));
      mix = std::max<int64_t>(mix, l.out.ld);
      if (l.dt.N) dtw = std::max<int64_t>(dtw, up8(l.dt.N));
      rec = std::max(rec, matrix_chunk_bytes(m.heads, m.kv_heads, m.dim, m.mixer == MTJ_MIXER_MATRIX_STATE_DELTA));
      if (l.gate2.N) gate = std::max<int64_t>(gate, up8(l.gate2.N));
    } else {
      qabs = std::max<int64_t>(qabs, static_cast<int64_t>(m.heads) * l.row_ld);
      po = std::max<int64_t>(po, static_cast<int64_t>(m.heads) * l.kv_ld);
      ml = std::max<int64_t>(ml, m.heads);
      if (l.up.N) {
        qp = std::max<int64_t>(qp, static_cast<int64_t>(m.heads) * 64 * l.key_blocks);
        cl = std::max<int64_t>(cl, l.kv_ld);
        kr = std::max<int64_t>(kr, l.kr_ld);
        kv = std::max<int64_t>(kv, l.up.N);
        hist = std::max<int64_t>(hist, std::min(m.window, max_pos_) - 1);
      }
    }
  }
  ld_p1_ = static_cast<int>(p1);
  ld_act_ = static_cast<int>(act);
  lin_rows_ = static_cast<int>(R + hist);
  x_ = c.take<float>(R * ld_);
  stats_ = c.take<float>(R * 2);
  y_ = c.take<float>(R * ld_);
  p1_ = c.take<float>(R * p1);
  act_ = c.take<float>(R * act);
  u_ = c.take<float>(R * u);
  xp_ = c.take<float>(R * xp);
  dt_raw_ = c.take<float>(R * dtw);
  gate_raw_ = c.take<float>(R * gate);
  ld_aux_ = static_cast<int>(aux);
  ld_mix_ = static_cast<int>(mix);
  aux_ = c.take<float>(R * aux);
  mix_ = c.take<float>(R * mix);
  q_f32_ = c.take<float>(R * qf);
  q_abs_ = c.take<float>(rows_a_ * qabs);
  part_o_ = c.take<float>(std::max((rows_a_ + kLatentBlocks) * po, gpo));
  part_ml_ = c.take<float>(std::max((rows_a_ + kLatentBlocks) * ml * 2, gml));
  counters_ = c.take<uint32_t>(R);
  attn_counters_ = c.take<uint32_t>(cnt);
  if (loop_times_ > 0) {
    x0_ = c.take<float>(R * ld_);
    cat_ = c.take<float>(R * 2 * ld_);
  }
  if (!f32_) {
    xn_bf_ = c.take<__nv_bfloat16>(R * ld_);
    sel_bf_ = c.take<__nv_bfloat16>(R * ld_);
    if (loop_times_ > 0) cat_bf_ = c.take<__nv_bfloat16>(R * 2 * ld_);
    xz_bf_ = c.take<__nv_bfloat16>(R * xz);
    u_bf_ = c.take<__nv_bfloat16>(R * u);
    dtr_bf_ = c.take<__nv_bfloat16>(R * dtr);
    xp_planes_elems_ = xp * std::max<int64_t>(6 * R, 16 * std::min<int64_t>(R, 128));
    xp_planes_ = c.take<float>(xp_planes_elems_);
    act_bf_ = c.take<__nv_bfloat16>(R * act);
    gate_bf_ = c.take<__nv_bfloat16>(R * gate);
    // sequences of at least kChunkedRows rows: their chunks, the last one of each may be partial
    chunk_records_ = c.take<char>((R / kMatrixChunk + R / kChunkedRows + 1) * rec);
    q_pack_ = c.take<__nv_bfloat16>(R * qp);
    c_lin_ = c.take<__nv_bfloat16>(lin_rows_ * cl);
    kr_lin_ = c.take<__nv_bfloat16>(lin_rows_ * kr);
    kv_lin_ = c.take<__nv_bfloat16>(lin_rows_ * kv);
  }
  for (Layer& l : layers_)
    if (l.ring_pages && !(l.d.mixer == MTJ_MIXER_GROUPED_ATTENTION && l.d.kv_from >= 0))
      l.page_table = c.take<int32_t>(static_cast<int64_t>(max_batch_) * l.ring_pages);
  for (size_t i = 0; i < runs_.size(); ++i) {
    Run& r = runs_[i];
    const Layer& l = layers_[r.layer];
    if (l.d.mixer == MTJ_MIXER_GROUPED_ATTENTION) {
      if (r.kv_run != static_cast<int>(i)) {            // keys and values of an earlier run
        const Run& src = runs_[r.kv_run];
        r.k_pool = src.k_pool;
        r.v_pool = src.v_pool;
        r.page_table = src.page_table;
        continue;
      }
      const int64_t n = static_cast<int64_t>(max_batch_) * l.ring_pages * kPageTokens * l.d.kv_heads;
      auto pool = [&](int64_t elems) { return f32_ ? static_cast<void*>(c.take<float>(elems)) : static_cast<void*>(c.take<__nv_bfloat16>(elems)); };
      r.k_pool = pool(n * l.k_cols);
      r.v_pool = pool(n * l.v_cols);
      r.page_table = l.page_table;
    } else if (l.d.mixer == MTJ_MIXER_MATRIX_STATE_SSD || l.d.mixer == MTJ_MIXER_MATRIX_STATE_DELTA) {
      r.conv_state = c.take<float>(static_cast<int64_t>(max_batch_) * (l.d.conv - 1) * l.ld_u);
      r.ssm_state = c.take<float>(static_cast<int64_t>(max_batch_) * l.d.heads * l.d.dim * l.d.vdim);
    } else if (l.d.mixer == MTJ_MIXER_LATENT_ATTENTION) {
      const int64_t elems = static_cast<int64_t>(max_batch_) * l.ring_pages * kPageTokens * l.row_ld;
      r.cache = f32_ ? static_cast<void*>(c.take<float>(elems)) : static_cast<void*>(c.take<__nv_bfloat16>(elems));
    } else {
      r.conv_state = c.take<float>(static_cast<int64_t>(max_batch_) * (l.d.conv - 1) * l.ld_u);
      r.ssm_state = c.take<float>(static_cast<int64_t>(max_batch_) * l.d.inner * l.d.state);
    }
  }
  s_end_ = c.base ? c.base + c.off : nullptr;
}

int32_t LayerStack::add_leaf(const std::string& name, Leaf leaf) {
  leaf.id = leaf_count_++;
  leaf_map_[name] = leaf;
  return MTJ_OK;
}

int32_t LayerStack::bind(mtj_handle* h, cudaStream_t s) {
  // padding columns and rows are zero for good; caches start finite
  MTJ_CUDA(cudaMemsetAsync(w_begin_, 0, w_end_ - w_begin_, s));
  MTJ_CUDA(cudaMemsetAsync(s_begin_, 0, s_end_ - s_begin_, s));
  for (auto& t : tables_) {
    const int half = t.first.second / 2;
    std::vector<float2> tab(static_cast<size_t>(max_pos_) * half);
    for (int i = 0; i < half; ++i) {
      const double f = pow(t.first.first, -2.0 * i / t.first.second);
      for (int p = 0; p < max_pos_; ++p)
        tab[static_cast<size_t>(p) * half + i] = make_float2(static_cast<float>(sin(p * f)), static_cast<float>(cos(p * f)));
    }
    if (!tab.empty()) MTJ_CUDA(cudaMemcpyAsync(t.second, tab.data(), tab.size() * sizeof(float2), cudaMemcpyHostToDevice, s));
    MTJ_CUDA(cudaStreamSynchronize(s));            // `tab` goes out of scope
  }
  for (const Layer& l : layers_) {
    if (!l.page_table) continue;
    std::vector<int32_t> table(static_cast<size_t>(max_batch_) * l.ring_pages);
    for (size_t i = 0; i < table.size(); ++i) table[i] = static_cast<int32_t>(i);
    MTJ_CUDA(cudaMemcpyAsync(l.page_table, table.data(), table.size() * sizeof(int32_t), cudaMemcpyHostToDevice, s));
    MTJ_CUDA(cudaStreamSynchronize(s));
  }
  if (!f32_) {
    bool ok = true;
    auto wmap = [&](Linear& l) {
      if (l.w) ok = ok && make_tensor_map_bf16(&l.map, l.w, l.N, l.K, 128, l.ld) == cudaSuccess;
    };
    wmap(head_);
    wmap(loop_in_);
    for (Layer& l : layers_) {
      for (Linear* w : {&l.in, &l.out, &l.gate_up, &l.down, &l.x, &l.dt, &l.gate2, &l.up}) wmap(*w);
      if (l.d.mixer == MTJ_MIXER_GROUPED_ATTENTION && l.key_blocks)
        ok = ok && make_tensor_map_bf16(&l.map_q, q_pack_, R_, static_cast<int64_t>(l.d.heads) * l.q_cols, 128) == cudaSuccess;
      if (!l.up.w) continue;
      const int H = l.d.heads;
      ok = ok && make_tensor_map_bf16(&l.map_q, q_pack_, R_, static_cast<int64_t>(H) * 64 * l.key_blocks, 128) == cudaSuccess;
      ok = ok && make_tensor_map_bf16(&l.map_k, kv_lin_, lin_rows_, static_cast<int64_t>(H) * 64 * l.k_own, 64, l.up.N) == cudaSuccess;
      ok = ok && make_tensor_map_bf16(&l.map_v, kv_lin_ + static_cast<int64_t>(H) * 64 * l.k_own, lin_rows_,
                                      static_cast<int64_t>(H) * 64 * l.value_blocks, 64, l.up.N) == cudaSuccess;
      ok = ok && make_tensor_map_bf16(&l.map_kr, kr_lin_, lin_rows_, l.kr_ld, 64) == cudaSuccess;
    }
    for (Run& r : runs_) {
      const Layer& l = layers_[r.layer];
      if (l.d.mixer != MTJ_MIXER_GROUPED_ATTENTION || !l.key_blocks) continue;
      const int64_t n = static_cast<int64_t>(max_batch_) * l.ring_pages * kPageTokens;
      ok = ok && make_tensor_map_bf16(&r.map_k, r.k_pool, n, static_cast<int64_t>(l.d.kv_heads) * l.k_cols, kPageTokens) == cudaSuccess;
      ok = ok && make_tensor_map_bf16(&r.map_v, r.v_pool, n, static_cast<int64_t>(l.d.kv_heads) * l.v_cols, kPageTokens) == cudaSuccess;
    }
    if (!ok) return fail(MTJ_ERR_CUDA, "cuTensorMapEncodeTiled failed");
  }

  // the tensors this stack expects, by name
  leaf_map_.clear();
  leaf_count_ = 0;
  auto rows = [&](const std::string& n, int N, int K, __nv_bfloat16* dst, int ld, int r0 = 0, int gin = 1, int gout = 1,
                  int csplit = 1 << 30, int cshift = 0) {
    Leaf f = {};
    f.shape = {N, K};
    f.op = kRows;
    f.packs.push_back({0, N, dst, ld, r0, gin, gout, csplit, cshift});
    add_leaf(n, f);
  };
  auto vec = [&](const std::string& n, int N, float* dst) {
    Leaf f = {};
    f.shape = {N};
    f.op = kF32;
    f.dst = dst;
    add_leaf(n, f);
  };
  auto taps = [&](const std::string& n, int channels, int conv, float* dst, int ld) {
    Leaf f = {};
    f.shape = {channels, conv};
    f.op = kTransposeF32;
    f.dst = dst;
    f.ld = ld;
    add_leaf(n, f);
  };
  auto neg_exp = [&](const std::string& n, std::vector<int64_t> shape, float* dst) {
    Leaf f = {};
    f.shape = shape;
    f.op = kNegExp;
    f.dst = dst;
    add_leaf(n, f);
  };
  rows("embed", V_, d_, embed_, d_);
  vec("final.norm", d_, final_norm_);
  if (post_ln_) vec("final.norm.b", d_, final_norm_b_);
  rows("head", V_, d_, head_.w, head_.ld);
  if (loop_times_ > 0) rows("loop.in", d_, 2 * d_, loop_in_.w, loop_in_.ld, 0, 1, 1, d_, ld_ - d_);
  for (size_t i = 0; i < layers_.size(); ++i) {
    Layer& l = layers_[i];
    const mtj_layer_desc& m = l.d;
    const std::string p = "l" + std::to_string(i) + ".";
    vec(p + "norm1", d_, l.norm1);
    if (post_ln_) vec(p + "norm1.b", d_, l.norm1_b);
    else vec(p + "norm1b", d_, l.norm1b);
    rows(p + "mix.o", l.out.N, l.out.K, l.out.w, l.out.ld);
    if (m.mixer == MTJ_MIXER_LATENT_ATTENTION) {
      const int nq = m.heads * (m.dim + m.rot_dim);
      rows(p + "mix.q", nq, d_, l.in.w, l.in.ld);
      rows(p + "mix.dkv", m.kv_rank + m.rot_dim, d_, l.in.w, l.in.ld, nq);
      vec(p + "mix.dkv.norm", m.kv_rank, l.kv_norm);
      rows(p + "mix.uk", m.heads * m.dim, m.kv_rank, l.uk, l.kv_ld);
      rows(p + "mix.uv", m.heads * m.vdim, m.kv_rank, l.uv, l.kv_ld);
      if (l.up.w) {
        // once more in the expanded form
        leaf_map_[p + "mix.uk"].packs.push_back({0, m.heads * m.dim, l.up.w, l.up.ld, 0, m.dim, 64 * l.k_own, 1 << 30, 0});
        leaf_map_[p + "mix.uv"].packs.push_back({0, m.heads * m.vdim, l.up.w, l.up.ld, m.heads * 64 * l.k_own, m.vdim, 64 * l.value_blocks, 1 << 30, 0});
      }
    } else if (m.mixer == MTJ_MIXER_GROUPED_ATTENTION) {
      const int nq = m.heads * m.dim, nk = m.kv_heads * m.dim;
      rows(p + "mix.q", nq, d_, l.in.w, l.in.ld);
      vec(p + "mix.q.norm", nq, l.q_norm);
      if (m.kv_from < 0) {
        rows(p + "mix.k", nk, d_, l.in.w, l.in.ld, nq);
        rows(p + "mix.v", m.kv_heads * m.vdim, d_, l.in.w, l.in.ld, nq + nk);
        vec(p + "mix.k.norm", nk, l.k_norm);
      }
    } else if (m.mixer == MTJ_MIXER_MATRIX_STATE_SSD) {
      const int inner = m.heads * m.vdim;
      Leaf f = {};
      f.shape = {inner + l.channels + m.heads, d_};
      f.op = kRows;
      f.packs.push_back({0, inner, l.in.w, l.in.ld, 0, 1, 1, 1 << 30, 0});
      f.packs.push_back({inner, l.channels, l.in.w, l.in.ld, l.x0, 1, 1, 1 << 30, 0});
      f.packs.push_back({inner + l.channels, m.heads, l.in.w, l.in.ld, l.aux0, 1, 1, 1 << 30, 0});
      add_leaf(p + "mix.in", f);
      taps(p + "mix.conv", l.channels, m.conv, l.conv_w, l.ld_u);
      vec(p + "mix.conv.b", l.channels, l.conv_b);
      vec(p + "mix.dt_bias", m.heads, l.dt_b);
      vec(p + "mix.D", m.heads, l.D);
      vec(p + "mix.norm", inner, l.mix_norm);
      neg_exp(p + "mix.A_log", {m.heads}, l.A);
    } else if (m.mixer == MTJ_MIXER_MATRIX_STATE_DELTA) {
      const int inner = m.heads * m.vdim, keys = m.kv_heads * m.dim;
      int at = 0;
      for (const auto& part : {std::make_pair("q", keys), std::make_pair("k", keys), std::make_pair("v", inner)}) {
        rows(p + "mix." + part.first, part.second, d_, l.in.w, l.in.ld, at);
        taps(p + "mix." + part.first + ".conv", part.second, m.conv, l.conv_w + at, l.ld_u);
        at += part.second;
      }
      rows(p + "mix.a1", m.decay_rank, d_, l.in.w, l.in.ld, l.a0);
      rows(p + "mix.g1", m.gate_rank, d_, l.in.w, l.in.ld, l.g0);
      rows(p + "mix.b", m.heads, d_, l.in.w, l.in.ld, l.aux0);
      rows(p + "mix.a2", l.dt.N, l.dt.K, l.dt.w, l.dt.ld);
      rows(p + "mix.g2", l.gate2.N, l.gate2.K, l.gate2.w, l.gate2.ld);
      vec(p + "mix.dt_bias", m.heads * m.dim, l.dt_b);
      vec(p + "mix.norm", m.vdim, l.mix_norm);
      neg_exp(p + "mix.A_log", {m.heads}, l.A);
    } else {
      rows(p + "mix.in", 2 * m.inner, d_, l.in.w, l.in.ld, 0, m.inner, up8(m.inner));
      rows(p + "mix.x", l.x.N, l.x.K, l.x.w, l.x.ld);
      rows(p + "mix.dt", l.dt.N, l.dt.K, l.dt.w, l.dt.ld);
      vec(p + "mix.conv.b", m.inner, l.conv_b);
      vec(p + "mix.dt.b", m.inner, l.dt_b);
      vec(p + "mix.D", m.inner, l.D);
      taps(p + "mix.conv", m.inner, m.conv, l.conv_w, l.ld_u);
      neg_exp(p + "mix.A_log", {m.inner, m.state}, l.A);
    }
    if (m.ff > 0) {
      vec(p + "norm2", d_, l.norm2);
      if (post_ln_) vec(p + "norm2.b", d_, l.norm2_b);
      else vec(p + "norm2b", d_, l.norm2b);
      if (m.ff_kind == MTJ_FF_SWIGLU) {
        rows(p + "mlp.gate", m.ff, d_, l.gate_up.w, l.gate_up.ld, 0, 1, 2);
        rows(p + "mlp.up", m.ff, d_, l.gate_up.w, l.gate_up.ld, 1, 1, 2);
      } else {
        rows(p + "mlp.up", m.ff, d_, l.gate_up.w, l.gate_up.ld);
      }
      rows(p + "mlp.down", d_, m.ff, l.down.w, l.down.ld);
    }
  }
  h->expected = leaf_count_;
  return MTJ_OK;
}

int32_t LayerStack::load_param(mtj_handle* h, const std::string& name, const void* src, int32_t dtype, int32_t ndim,
                               const int64_t* shape, cudaStream_t s) {
  const auto it = leaf_map_.find(name);
  if (it == leaf_map_.end()) return fail(MTJ_ERR_INVALID, "unknown tensor: " + name);
  const Leaf& f = it->second;
  if (ndim != static_cast<int32_t>(f.shape.size()) || !std::equal(f.shape.begin(), f.shape.end(), shape))
    return fail(MTJ_ERR_INVALID, "shape mismatch for " + name);
  const int bf = dtype == MTJ_BF16;
  const int N = static_cast<int>(f.shape[0]), K = ndim > 1 ? static_cast<int>(f.shape[1]) : 1;
  switch (f.op) {
    case kRows:
      for (const Pack& k : f.packs) {
        const char* from = static_cast<const char*>(src) + static_cast<size_t>(k.src0) * K * (bf ? 2 : 4);
        MTJ_CUDA(launch_pack_rows(from, bf, k.n, K, k.dst, k.ld, k.r0, k.gin, k.gout, k.csplit, k.cshift, s));
      }
      break;
    case kF32: MTJ_CUDA(launch_to_f32(src, bf, N, static_cast<float*>(f.dst), s)); break;
    case kNegExp: MTJ_CUDA(launch_neg_exp(src, bf, static_cast<int64_t>(N) * K, static_cast<float*>(f.dst), s)); break;
    default: MTJ_CUDA(launch_transpose_f32(src, bf, N, K, static_cast<float*>(f.dst), f.ld, s)); break;
  }
  h->leaf_loaded[static_cast<size_t>(f.id)] = 1;
  return MTJ_OK;
}

// ------------------------------------------------------------------------------------------------- linear maps
bool LayerStack::use_tc(const mtj_handle* h, int M, bool decode) const {
  return !f32_ && M >= (decode ? h->tc_decode_min_b : tc_min_rows_);
}

const TensorMap* LayerStack::xmap(const __nv_bfloat16* buf, int K, int ld, int M) {
  const auto key = std::make_tuple(static_cast<const void*>(buf), K, ld);
  auto it = xmaps_.find(key);
  if (it == xmaps_.end()) {
    std::array<TensorMap, 3> maps;
    const int rows = buf == c_lin_ ? lin_rows_ : R_;
    for (int i = 0; i < 3; ++i)
      if (make_tensor_map_bf16(&maps[i], buf, rows, K, 32 << i, ld) != cudaSuccess) return nullptr;
    it = xmaps_.emplace(key, maps).first;
  }
  const int tile = M > 192 ? gemm_tc_wide_token_tile() : gemm_tc_token_tile_for(M);
  return &it->second[tile == 32 ? 0 : tile == 64 ? 1 : 2];
}

int32_t LayerStack::gemm(mtj_handle* h, GemvEpilogue epi, const Linear& l, const __nv_bfloat16* x, int M, float* out, int ld_out,
                         __nv_bfloat16* out_bf16, int ld_bf16, bool decode, cudaStream_t s, int x_row0, int x_ld, int f32_from) {
  const TensorMap* mx = xmap(x, l.K, x_ld > 0 ? x_ld : l.ld, M);
  if (!mx) return fail(MTJ_ERR_CUDA, "cuTensorMapEncodeTiled failed");
  GemmTcArgs a = {};
  a.M = M;
  a.N = l.N;
  a.K = l.K;
  a.x_row0 = x_row0;
  a.out = out;
  a.ld_out = ld_out;
  a.out_bf16 = out_bf16;
  a.ld_bf16 = ld_bf16;
  a.dev_err = h->dev_err;
  a.softcap = softcap_;
  a.f32_from = f32_from;
  a.pair = 1;
  a.cluster_k = h->tc_cluster_k ? gemm_tc_decode_cluster_k(l.N, M, l.K) : 1;
  if (M > 192) MTJ_CUDA(launch_gemm_tc_wide(epi, &l.map, mx, a, s));
  else MTJ_CUDA(launch_gemm_tc(epi, &l.map, mx, a, s, decode && h->use_pdl && h->tc_pdl));
  h->launches++;
  return MTJ_OK;
}

// A projection with few weight rows: K split over blocks, the partial sums [planes, M, N] left for the consumer to add.
int32_t LayerStack::gemm_planes(mtj_handle* h, const Linear& l, const __nv_bfloat16* x, int M, int* planes, bool decode,
                                cudaStream_t s) {
  const int bn = gemm_tc_token_tile_for(M);
  const auto key = xmap(x, l.K, l.ld, std::min(M, 128));
  if (!key) return fail(MTJ_ERR_CUDA, "cuTensorMapEncodeTiled failed");
  const int tiles = ((l.N + 127) / 128) * ((M + bn - 1) / bn);
  const int64_t fit = xp_planes_elems_ / (static_cast<int64_t>(M) * l.N);
  GemmTcArgs a = {};
  a.M = M;
  a.N = l.N;
  a.K = l.K;
  a.partial = xp_planes_;
  a.ksplit = static_cast<int>(std::max<int64_t>(1, std::min<int64_t>({fit, 296 / tiles, (l.K + 127) / 128, 16})));
  a.dev_err = h->dev_err;
  MTJ_CUDA(launch_gemm_tc(kEpiPlain, &l.map, key, a, s, decode && h->use_pdl && h->tc_pdl));
  h->launches++;
  *planes = a.ksplit;
  return MTJ_OK;
}

int32_t LayerStack::gemv(mtj_handle* h, GemvEpilogue epi, const Linear& l, const float* x, int ldx, int M, const float* norm,
                         float* out, int ld_out, const Post* post, bool pdl, cudaStream_t s, const int32_t* select,
                         const float* stats) {
  GemvArgs a = {};
  a.W = l.w;
  a.N = up4(l.N);
  a.n_valid = l.N;
  a.K = l.ld;
  a.M = M;
  a.x = x;
  a.ldx = ldx;
  a.ln_scale = norm;
  a.ln_offset = norm == final_norm_ && final_norm_b_ ? final_norm_b_ : zeros_;
  a.stats = stats ? stats : stats_;
  a.rows = {0, 1, 0, nullptr};
  a.row_select = select;
  a.dev_err = h->dev_err;
  a.ld_out = ld_out;
  if (epi == kEpiSwiGLU || epi == kEpiRelu2) a.act2 = out;
  else if (epi == kEpiLogits) { a.logits = out; a.ld_logits = ld_out; a.softcap = l.w == head_.w ? softcap_ : 0.f; }
  else a.out = out;
  if (post) {
    a.post_w = post->w;
    a.post_b = post->b;
    a.post_x = x_;
    a.post_ldx = ld_;
    a.post_mult = mult_;
    a.post_eps = eps_;
    a.stats_out = post->stats ? stats_ : nullptr;
    a.counters = counters_;
  }
  MTJ_CUDA(launch_gemv(epi, a, s, pdl));
  h->launches++;
  return MTJ_OK;
}

// --------------------------------------------------------------------------------------------------- mixers
#define MTJ_DO(expr)                       \
  do {                                     \
    const int32_t _rc = (expr);            \
    if (_rc) return _rc;                   \
  } while (0)

int32_t LayerStack::project_in(mtj_handle* h, const Linear& l, const float* norm, int M, float* out, int ld_out, bool pdl, cudaStream_t s) {
  return post_ln_ ? gemv(h, kEpiOut, l, x_, ld_, M, nullptr, out, ld_out, nullptr, pdl, s)
                  : gemv(h, kEpiLogits, l, x_, ld_, M, norm, out, ld_out, nullptr, pdl, s);
}

int32_t LayerStack::mamba(mtj_handle* h, const Run& r, int M, const RowMap& rows, bool tc, bool decode, const Post& post, cudaStream_t s) {
  Layer& l = layers_[r.layer];
  const mtj_layer_desc& m = l.d;
  const bool pdl = decode && h->use_pdl;
  SsmArgs a = {};
  a.M = M;
  a.inner = m.inner;
  a.state = m.state;
  a.taps = m.conv;
  a.dt_rank = m.dt_rank;
  a.rows = rows;
  a.nseq = M / rows.Tc;
  a.pad = h->pad;
  a.ld_xz = up8(l.in.N);
  a.z0 = l.ld_u;
  a.conv_w = l.conv_w;
  a.conv_b = l.conv_b;
  a.conv_state = r.conv_state;
  a.ld_u = l.ld_u;
  a.xp = xp_;
  a.ld_xp = l.ld_xp;
  a.w_dt = l.dt.w;
  a.ld_wdt = l.dt.ld;
  a.dt_b = l.dt_b;
  a.A = l.A;
  a.D = l.D;
  a.ssm_state = r.ssm_state;
  h->prof_begin(MTJ_FAMILY_INPROJ, s);
  if (tc) {
    a.xz = xz_bf_;
    a.xz_bf16 = 1;
    a.u_bf16 = u_bf_;
    a.out_bf16 = act_bf_;
    a.xp_planes = xp_planes_;
    a.xp_out = xp_;
    a.dtr_bf16 = dtr_bf_;
    a.ld_dtr = l.dt.ld;
    MTJ_DO(gemm(h, kEpiPlain, l.in, xn_bf_, M, nullptr, 0, xz_bf_, a.ld_xz, decode, s));
  } else {
    a.xz = p1_;
    a.u = u_;
    a.out = act_;
    MTJ_DO(project_in(h, l.in, l.norm1, M, p1_, a.ld_xz, pdl, s));
  }
  h->prof_end(s);
  h->prof_begin(MTJ_FAMILY_ATTN, s);
  MTJ_CUDA(launch_ssm_conv(a, s, pdl));
  h->launches += (rows.Tc == 1 || m.conv == 1) ? 1 : 2;
  if (tc) {
    MTJ_DO(gemm_planes(h, l.x, u_bf_, M, &a.planes, decode, s));
    MTJ_CUDA(launch_ssm_split(a, s, pdl));
    h->launches++;
    MTJ_DO(gemm(h, kEpiPlain, l.dt, dtr_bf_, M, dt_raw_, l.ld_u, nullptr, 0, decode, s));
    a.dt_raw = dt_raw_;
  } else {
    MTJ_DO(gemv(h, kEpiOut, l.x, u_, l.ld_u, M, nullptr, xp_, l.ld_xp, nullptr, pdl, s));
    if (rows.Tc > 1) {
      MTJ_DO(gemv(h, kEpiOut, l.dt, xp_, l.ld_xp, M, nullptr, dt_raw_, l.ld_u, nullptr, pdl, s));
      a.dt_raw = dt_raw_;
    }
  }
  if (rows.Tc == 1) MTJ_CUDA(launch_ssm_step(a, s, pdl));
  else MTJ_CUDA(launch_ssm_scan(a, s));
  h->launches++;
  h->prof_end(s);
  h->prof_begin(MTJ_FAMILY_OUTPROJ, s);
  if (tc) MTJ_DO(gemm(h, kEpiPlain, l.out, act_bf_, M, y_, ld_, nullptr, 0, decode, s));
  else MTJ_DO(gemv(h, kEpiOut, l.out, act_, l.out.ld, M, nullptr, y_, ld_, &post, pdl, s));
  h->prof_end(s);
  return MTJ_OK;
}

int32_t LayerStack::latent(mtj_handle* h, const Run& r, int M, const RowMap& rows, int hist, bool tc, bool decode, const Post& post,
                           cudaStream_t s) {
  Layer& l = layers_[r.layer];
  const mtj_layer_desc& m = l.d;
  const bool pdl = decode && h->use_pdl;
  LatentArgs a = {};
  a.M = M;
  a.heads = m.heads;
  a.dim = m.dim;
  a.rot = m.rot_dim;
  a.vdim = m.vdim;
  a.rank = m.kv_rank;
  a.window = m.window;
  a.scale = m.scale;
  a.eps = eps_;
  a.rows = rows;
  a.pad = h->pad;
  a.cache = {r.cache, f32_ ? 1 : 0, l.page_table, l.ring_pages, l.row_ld, l.kv_ld};
  a.sincos = l.sincos;
  a.p1 = p1_;
  a.ld_p1 = up8(l.in.N);
  a.kv_norm = l.kv_norm;
  a.w_uk = l.uk;
  a.w_uv = l.uv;
  a.q_abs = q_abs_;
  a.part_o = part_o_;
  a.part_ml = part_ml_;
  a.ld_out = l.out.ld;
  h->prof_begin(MTJ_FAMILY_INPROJ, s);
  if (tc) MTJ_DO(gemm(h, kEpiPlain, l.in, xn_bf_, M, p1_, a.ld_p1, nullptr, 0, decode, s));
  else MTJ_DO(project_in(h, l.in, l.norm1, M, p1_, a.ld_p1, pdl, s));
  h->prof_end(s);
  h->prof_begin(MTJ_FAMILY_ATTN, s);
  if (tc && !decode && l.up.w) {
    a.q_pack = q_pack_;
    a.key_blocks = l.key_blocks;
    a.k_own = l.k_own;
    a.c_lin = c_lin_;
    a.kr_lin = kr_lin_;
    a.kr_ld = l.kr_ld;
    a.nseq = M / rows.Tc;
    a.hist = std::min(hist, m.window - 1);
    a.key_rows = a.hist + rows.Tc;
    MTJ_CUDA(launch_latent_pack(a, s));
    MTJ_CUDA(launch_latent_history(a, s));
    MTJ_DO(gemm(h, kEpiPlain, l.up, c_lin_, a.nseq * a.key_rows, nullptr, 0, kv_lin_, l.up.N, decode, s));
    PrefillAttnTcArgs p = {};
    p.kv.pad = h->pad;
    p.rows = rows;
    p.M = M;
    p.heads = m.heads;
    p.out_bf16 = act_bf_;
    p.ld_out = l.out.ld;
    p.dev_err = h->dev_err;
    p.window = m.window;
    p.hist = a.hist;
    p.key_rows = a.key_rows;
    p.k_own = l.k_own;
    p.v_cols = m.vdim;
    p.scale_log2 = m.scale * 1.4426950408889634f;
    MTJ_CUDA(launch_prefill_attn_tc_linear(&l.map_q, &l.map_k, &l.map_kr, &l.map_v, l.key_blocks, l.value_blocks, p, s));
    h->launches += a.hist > 0 ? 3 : 2;
  } else {
    // blocks of rows of one sequence (or of one-row sequences)
    const int per = rows.Tc == 1 ? M : rows.Tc;
    for (int m0 = 0; m0 < M; m0 += per)
      for (int t0 = 0; t0 < per; t0 += rows_a_) {
        LatentArgs b = a;
        b.M = std::min(rows_a_, per - t0);
        b.tensor_cores = tc ? 1 : 0;
        b.rows = rows.Tc == 1 ? RowMap{rows.b0 + t0, 1, rows.pos0_host, rows.pos0_dev}
                              : RowMap{rows.b0 + m0 / per, b.M, rows.pos0_host + t0, rows.pos0_dev};
        b.p1 = p1_ + static_cast<size_t>(m0 + t0) * a.ld_p1;
        b.splits = latent_attn_splits(b.M, m.heads, l.row_ld, tc ? 1 : 0, std::min(m.window, max_pos_));
        if (tc) b.out_bf16 = act_bf_ + static_cast<size_t>(m0 + t0) * a.ld_out;
        else b.out = act_ + static_cast<size_t>(m0 + t0) * a.ld_out;
        MTJ_CUDA(launch_latent_absorb(b, s, pdl));
        MTJ_CUDA(launch_latent_attn(b, s, pdl));
        MTJ_CUDA(launch_latent_out(b, s, pdl));
        h->launches += 3;
      }
  }
  h->prof_end(s);
  h->prof_begin(MTJ_FAMILY_OUTPROJ, s);
  if (tc) MTJ_DO(gemm(h, kEpiPlain, l.out, act_bf_, M, y_, ld_, nullptr, 0, decode, s));
  else MTJ_DO(gemv(h, kEpiOut, l.out, act_, l.out.ld, M, nullptr, y_, ld_, &post, pdl, s));
  h->prof_end(s);
  return MTJ_OK;
}

int32_t LayerStack::grouped(mtj_handle* h, const Run& r, int M, const RowMap& rows, bool tc, bool decode, const Post& post, cudaStream_t s) {
  Layer& l = layers_[r.layer];
  const mtj_layer_desc& m = l.d;
  const bool pdl = decode && h->use_pdl;
  GroupedAttnArgs a = {};
  a.M = M;
  a.heads = m.heads;
  a.kv_heads = m.kv_heads;
  a.dim = m.dim;
  a.vdim = m.vdim;
  a.window = max_pos_;
  a.scale = m.scale;
  a.eps = eps_;
  a.q_temp_coef = m.q_temp_coef;
  a.q_temp_every = m.q_temp_every;
  a.rows = rows;
  a.pad = h->pad;
  a.cache = {r.k_pool, r.v_pool, f32_ ? 1 : 0, r.page_table, l.ring_pages, m.kv_heads * l.k_cols, m.kv_heads * l.v_cols};
  a.p1 = p1_;
  a.ld_p1 = up8(l.in.N);
  a.own_kv = m.kv_from < 0;
  a.q_norm = l.q_norm;
  a.k_norm = l.k_norm;
  a.q_bf16 = l.key_blocks ? q_pack_ : nullptr;
  a.q_f32 = l.key_blocks ? nullptr : q_f32_;
  a.q_cols = l.q_cols;
  a.part_o = part_o_;
  a.part_ml = part_ml_;
  a.counters = attn_counters_;
  a.ld_out = l.out.ld;
  h->prof_begin(MTJ_FAMILY_INPROJ, s);
  if (tc) MTJ_DO(gemm(h, kEpiPlain, l.in, xn_bf_, M, p1_, a.ld_p1, nullptr, 0, decode, s));
  else MTJ_DO(project_in(h, l.in, l.norm1, M, p1_, a.ld_p1, pdl, s));
  h->prof_end(s);
  h->prof_begin(MTJ_FAMILY_ATTN, s);
  MTJ_CUDA(launch_grouped_prep(a, s, pdl));
  h->launches++;
  if (tc && !decode && l.key_blocks) {
    PrefillAttnTcArgs p = {};
    p.kv.page_table = r.page_table;
    p.kv.ring_pages = l.ring_pages;
    p.kv.pad = h->pad;
    p.rows = rows;
    p.M = M;
    p.heads = m.heads;
    p.out_bf16 = act_bf_;
    p.ld_out = l.out.ld;
    p.dev_err = h->dev_err;
    p.window = a.window;
    p.kv_group = m.heads / m.kv_heads;
    p.k_cols = l.k_cols;
    p.v_ld = l.v_cols;
    p.v_cols = m.vdim;
    p.scale_log2 = m.scale * 1.4426950408889634f;
    MTJ_CUDA(launch_prefill_attn_tc_grouped(&l.map_q, &r.map_k, &r.map_v, l.key_blocks, l.value_blocks, p, s));
    h->launches++;
  } else {
    // blocks of rows of one sequence (or of one-row sequences)
    const int per = rows.Tc == 1 ? M : rows.Tc;
    for (int m0 = 0; m0 < M; m0 += per)
      for (int t0 = 0; t0 < per; t0 += rows_a_) {
        GroupedAttnArgs b = a;
        const size_t at = static_cast<size_t>(m0 + t0);
        b.M = std::min(rows_a_, per - t0);
        b.rows = rows.Tc == 1 ? RowMap{rows.b0 + t0, 1, rows.pos0_host, rows.pos0_dev}
                              : RowMap{rows.b0 + m0 / per, b.M, rows.pos0_host + t0, rows.pos0_dev};
        if (a.q_bf16) b.q_bf16 = a.q_bf16 + at * m.heads * l.q_cols;
        else b.q_f32 = a.q_f32 + at * m.heads * l.q_cols;
        b.splits = grouped_attn_splits(b.M, m.heads, m.kv_heads, max_pos_);
        if (tc) b.out_bf16 = act_bf_ + at * a.ld_out;
        else b.out = act_ + at * a.ld_out;
        MTJ_CUDA(launch_grouped_attn(b, s, pdl));
        h->launches++;
      }
  }
  h->prof_end(s);
  h->prof_begin(MTJ_FAMILY_OUTPROJ, s);
  if (tc) MTJ_DO(gemm(h, kEpiPlain, l.out, act_bf_, M, y_, ld_, nullptr, 0, decode, s));
  else MTJ_DO(gemv(h, kEpiOut, l.out, act_, l.out.ld, M, nullptr, y_, ld_, &post, pdl, s));
  h->prof_end(s);
  return MTJ_OK;
}

int32_t LayerStack::matrix(mtj_handle* h, const Run& r, int M, const RowMap& rows, bool tc, bool decode, const Post& post, cudaStream_t s) {
  Layer& l = layers_[r.layer];
  const mtj_layer_desc& m = l.d;
  const bool pdl = decode && h->use_pdl, ssd = m.mixer == MTJ_MIXER_MATRIX_STATE_SSD;
  const int ld_p = up8(l.in.N), inner = m.heads * m.vdim, keys = m.kv_heads * m.dim;
  // the input projection: convolution inputs, gates and low-rank parts in bf16, step sizes and update strengths in fp32
  const float* aux = tc ? aux_ : p1_ + l.aux0;
  const int ld_aux = tc ? ld_aux_ : ld_p;
  h->prof_begin(MTJ_FAMILY_INPROJ, s);
  if (tc) MTJ_DO(gemm(h, kEpiPlain, l.in, xn_bf_, M, aux_, ld_aux_, xz_bf_, ld_p, decode, s, 0, 0, l.aux0));
  else MTJ_DO(project_in(h, l.in, l.norm1, M, p1_, ld_p, pdl, s));
  h->prof_end(s);
  h->prof_begin(MTJ_FAMILY_ATTN, s);
  SsmArgs c = {};
  c.M = M;
  c.inner = l.channels;
  c.taps = m.conv;
  c.rows = rows;
  c.nseq = M / rows.Tc;
  c.pad = h->pad;
  if (tc) c.xz = xz_bf_ + l.x0;
  else c.xz = p1_ + l.x0;
  c.xz_bf16 = tc;
  c.ld_xz = ld_p;
  c.conv_w = l.conv_w;
  c.conv_b = l.conv_b;
  c.conv_state = r.conv_state;
  c.ld_u = l.ld_u;
  if (tc) c.u_bf16 = u_bf_;
  else c.u = u_;
  MTJ_CUDA(launch_ssm_conv(c, s, pdl));
  h->launches += (rows.Tc == 1 || m.conv == 1) ? 1 : 2;
  if (!ssd) {
    if (tc) {
      MTJ_DO(gemm(h, kEpiPlain, l.dt, xz_bf_ + l.a0, M, dt_raw_, up8(l.dt.N), nullptr, 0, decode, s, 0, ld_p));
      MTJ_DO(gemm(h, kEpiPlain, l.gate2, xz_bf_ + l.g0, M, nullptr, 0, gate_bf_, up8(inner), decode, s, 0, ld_p));
    } else {
      MTJ_DO(gemv(h, kEpiOut, l.dt, p1_ + l.a0, ld_p, M, nullptr, dt_raw_, up8(l.dt.N), nullptr, pdl, s));
      MTJ_DO(gemv(h, kEpiOut, l.gate2, p1_ + l.g0, ld_p, M, nullptr, gate_raw_, up8(inner), nullptr, pdl, s));
    }
  }
  MatrixStateArgs a = {};
  a.M = M;
  a.heads = m.heads;
  a.key_heads = m.kv_heads;
  a.dim = m.dim;
  a.vdim = m.vdim;
  a.delta = !ssd;
  a.rows = rows;
  a.nseq = M / rows.Tc;
  a.pad = h->pad;
  if (tc) a.u = u_bf_;
  else a.u = u_;
  a.u_bf16 = tc;
  a.ld_u = l.ld_u;
  a.v0 = ssd ? 0 : 2 * keys;
  a.k0 = ssd ? inner : keys;
  a.q0 = ssd ? inner + keys : 0;
  a.decay = ssd ? aux : dt_raw_;
  a.ld_decay = ssd ? ld_aux : up8(l.dt.N);
  a.decay_b = l.dt_b;
  a.A = l.A;
  a.beta = ssd ? nullptr : aux;
  a.ld_beta = ld_aux;
  a.D = l.D;
  a.q_scale = static_cast<float>(1.0 / sqrt(static_cast<double>(m.dim)));
  a.state = r.ssm_state;
  a.out = mix_;
  a.ld_out = ld_mix_;
  a.chunk_records = chunk_records_;
  a.dev_err = h->dev_err;
  GatedNormArgs g = {};
  g.M = M;
  g.parts = ssd ? m.norm_groups : m.heads;
  g.part_n = inner / g.parts;
  g.gate_first = ssd;
  g.eps = eps_;
  g.y = mix_;
  g.ld_y = ld_mix_;
  g.gate_bf16 = tc;
  if (ssd) g.gate = tc ? static_cast<const void*>(xz_bf_) : p1_;
  else g.gate = tc ? static_cast<const void*>(gate_bf_) : gate_raw_;
  g.ld_gate = ssd ? ld_p : up8(inner);
  g.w = l.mix_norm;
  if (tc) g.out_bf16 = act_bf_;
  else g.out = act_;
  g.ld_out = l.out.ld;
  const bool step = matrix_step_ok(a), normed = step && matrix_step_norms(a);
  if (step) MTJ_CUDA(launch_matrix_step(a, normed ? &g : nullptr, s, pdl));
  else if (tc && rows.Tc >= kChunkedRows) MTJ_CUDA(launch_matrix_chunks(a, s));
  else MTJ_CUDA(launch_matrix_scan(a, s, pdl));
  if (!normed) MTJ_CUDA(launch_gated_norm(g, s, pdl));
  h->launches += (normed ? 1 : 2) + (!step && tc && rows.Tc >= kChunkedRows ? 1 : 0);
  h->prof_end(s);
  h->prof_begin(MTJ_FAMILY_OUTPROJ, s);
  if (tc) MTJ_DO(gemm(h, kEpiPlain, l.out, act_bf_, M, y_, ld_, nullptr, 0, decode, s));
  else MTJ_DO(gemv(h, kEpiOut, l.out, act_, l.out.ld, M, nullptr, y_, ld_, &post, pdl, s));
  h->prof_end(s);
  return MTJ_OK;
}

// --------------------------------------------------------------------------------------------------- forward
int32_t LayerStack::forward(mtj_handle* h, const uint32_t* ids, int ids_ld, const RowMap& id_rows, int M, const RowMap& rows,
                            int hist, bool decode, cudaStream_t s) {
  if (M <= 0 || M > R_ || M % rows.Tc) return fail(MTJ_ERR_INVALID, "rows exceed max_rows");
  const bool tc = use_tc(h, M, decode), pdl = decode && h->use_pdl;
  last_tc_ = tc;
  EmbedArgs e = {};
  e.ids = ids;
  e.ids_ld = ids_ld;
  e.rows = id_rows;
  e.M = M;
  e.d = d_;
  e.vocab_local = V_;
  e.table = embed_;
  e.x = x_;
  e.ldx = ld_;
  e.scale = embed_scale_;
  if (post_ln_ && tc) e.x_bf16 = xn_bf_;               // what the first sublayer reads
  MTJ_CUDA(launch_embed(e, s, pdl));
  h->launches++;
  if (loop_times_ > 0) {
    MTJ_CUDA(launch_copy_rows(x_, x0_, static_cast<int64_t>(M) * ld_, s, pdl));
    h->launches++;
  }
  const int n_runs = stop_after > 0 ? std::min<int>(stop_after, runs()) : runs();
  // what follows a sublayer: the norm of the next one, the projection that opens a pass, or the final norm
  struct Next { const float* norm; bool pass; bool last = false; };
  auto next_run = [&](int i) -> Next {
    if (i >= n_runs) return {final_norm_, false, true};
    return {layers_[runs_[i].layer].norm1, runs_[i].first};
  };
  // residual add (y != null) and what the next sublayer reads; on the fp32 path the projections have done the add and
  // the statistics themselves
  auto settle = [&](const float* y, const Post& post, const Next& n) -> int32_t {
    if (post_ln_) {
      ResidualLayerNormArgs a = {};
      a.x = x_;
      a.M = M;
      a.d = d_;
      a.ld = ld_;
      a.y = y;
      a.w = post.w;
      a.b = post.b;
      a.alpha = mult_;
      a.eps = eps_;
      a.xn = xn_bf_;
      if (n.last) {
        a.w_next = final_norm_;
        a.b_next = final_norm_b_;
        a.stats = stats_;
      }
      MTJ_CUDA(launch_residual_layernorm(a, s, pdl));
      h->launches++;
      return MTJ_OK;
    }
    ResidualNormArgs a = {};
    a.x = x_;
    a.M = M;
    a.d = d_;
    a.ld = ld_;
    a.y = y;
    a.planes = 1;
    a.w_post = post.w;
    a.mult = mult_;
    a.eps = eps_;
    a.stats = stats_;
    if (n.pass) {
      a.x0 = x0_;
      if (tc) a.cat_bf16 = cat_bf_;
      else a.cat_f32 = cat_;
    } else if (tc) {
      a.w_next = n.norm;
      a.xn = xn_bf_;
    }
    MTJ_CUDA(launch_residual_norm(a, s, pdl));
    h->launches++;
    return MTJ_OK;
  };
  auto after = [&](const Post& post, const Next& n) -> int32_t {
    if (tc) return settle(y_, post, n);
    return n.pass ? settle(nullptr, Post{}, n) : MTJ_OK;
  };
  if (!post_ln_) MTJ_DO(settle(nullptr, Post{}, next_run(0)));
  for (int i = 0; i < n_runs; ++i) {
    const Run& r = runs_[i];
    const Layer& l = layers_[r.layer];
    if (r.first) {
      if (tc) MTJ_DO(gemm(h, kEpiPlain, loop_in_, cat_bf_, M, x_, ld_, nullptr, 0, decode, s));
      else MTJ_DO(gemv(h, kEpiOut, loop_in_, cat_, 2 * ld_, M, nullptr, x_, ld_, nullptr, pdl, s));
      MTJ_DO(settle(nullptr, Post{}, {l.norm1, false}));
    }
    const Next after_layer = next_run(i + 1), after_mixer = l.d.ff > 0 ? Next{l.norm2, false} : after_layer;
    // statistics of the new residual row: the next prologue's; behind a layer norm only the final norm has one
    const Post post1 = post_ln_ ? Post{l.norm1, l.norm1_b, after_mixer.last} : Post{l.norm1b, nullptr, true};
    const Post post2 = post_ln_ ? Post{l.norm2, l.norm2_b, after_layer.last} : Post{l.norm2b, nullptr, true};
    switch (l.d.mixer) {
      case MTJ_MIXER_LATENT_ATTENTION: MTJ_DO(latent(h, r, M, rows, hist, tc, decode, post1, s)); break;
      case MTJ_MIXER_GROUPED_ATTENTION: MTJ_DO(grouped(h, r, M, rows, tc, decode, post1, s)); break;
      case MTJ_MIXER_MAMBA1: MTJ_DO(mamba(h, r, M, rows, tc, decode, post1, s)); break;
      default: MTJ_DO(matrix(h, r, M, rows, tc, decode, post1, s)); break;
    }
    MTJ_DO(after(post1, after_mixer));
    if (l.d.ff > 0) {
      const GemvEpilogue act = l.d.ff_kind == MTJ_FF_SWIGLU ? kEpiSwiGLU : kEpiRelu2;
      h->prof_begin(MTJ_FAMILY_FFIN, s);
      if (tc) MTJ_DO(gemm(h, act, l.gate_up, xn_bf_, M, nullptr, 0, act_bf_, l.down.ld, decode, s));
      else MTJ_DO(gemv(h, act, l.gate_up, x_, ld_, M, post_ln_ ? nullptr : l.norm2, act_, l.down.ld, nullptr, pdl, s));
      h->prof_end(s);
      h->prof_begin(MTJ_FAMILY_OUTPROJ, s);
      if (tc) MTJ_DO(gemm(h, kEpiPlain, l.down, act_bf_, M, y_, ld_, nullptr, 0, decode, s));
      else MTJ_DO(gemv(h, kEpiOut, l.down, act_, l.down.ld, M, nullptr, y_, ld_, &post2, pdl, s));
      h->prof_end(s);
      MTJ_DO(after(post2, after_layer));
    }
  }
  return MTJ_OK;
}

int32_t LayerStack::logits(mtj_handle* h, int row0, int n, float* out, bool decode, cudaStream_t s) {
  h->prof_begin(MTJ_FAMILY_LOGITS, s);
  if (last_tc_) MTJ_DO(gemm(h, softcap_ > 0.f ? kEpiSoftcap : kEpiPlain, head_, xn_bf_, n, out, V_, nullptr, 0, decode, s, row0));
  else
    MTJ_DO(gemv(h, kEpiLogits, head_, x_ + static_cast<size_t>(row0) * ld_, ld_, n, final_norm_, out, V_, nullptr,
                decode && h->use_pdl, s, nullptr, stats_ + 2 * static_cast<size_t>(row0)));
  h->prof_end(s);
  return MTJ_OK;
}

int32_t LayerStack::logits_select(mtj_handle* h, const int32_t* rows_dev, int n, float* out, cudaStream_t s) {
  if (!last_tc_ || n <= kSelectGemvRows)
    return gemv(h, kEpiLogits, head_, x_, ld_, n, final_norm_, out, V_, nullptr, false, s, rows_dev);
  MTJ_CUDA(launch_gather_rows_bf16(xn_bf_, ld_, rows_dev, n, sel_bf_, s));
  h->launches++;
  return gemm(h, softcap_ > 0.f ? kEpiSoftcap : kEpiPlain, head_, sel_bf_, n, out, V_, nullptr, 0, false, s);
}

}  // namespace mtj
