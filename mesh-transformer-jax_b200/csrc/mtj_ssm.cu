// Selective state-space layers: causal convolution + silu, and the recurrence
//     S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c u_c B_n,   y_c = sum_n S[c, n] C_n + D_c u_c,   out = y * silu(z)
// with the convolution's last inputs and S (fp32) carried per sequence slot.  A sequence whose first row is in the call
// starts from zeros whatever its slot holds; rows before the start (left padding) change nothing.
#include <math.h>

#include <algorithm>

#include "mtj_common.cuh"
#include "mtj_stack_kernels.h"

namespace mtj {
namespace {

__device__ __forceinline__ float ld(const float* p, size_t i) { return p[i]; }
__device__ __forceinline__ float ld(const __nv_bfloat16* p, size_t i) { return __bfloat162float(p[i]); }
__device__ __forceinline__ float silu_exact(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float softplus_exact(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
// Elementwise functions of a run with T operands: the accurate ones for fp32 runs; serving runs, whose inputs carry bf16
// rounding, take the fast fp32 intrinsics (log(1 + e) by its series where 1 + e would round e away).
template <typename T>
struct Fn;
template <>
struct Fn<float> {
  __device__ static __forceinline__ float silu(float z) { return silu_exact(z); }
  __device__ static __forceinline__ float softplus(float z) { return softplus_exact(z); }
};
template <>
struct Fn<__nv_bfloat16> {
  __device__ static __forceinline__ float silu(float z) { return __fdividef(z, 1.0f + __expf(-z)); }
  __device__ static __forceinline__ float softplus(float z) {
    const float e = __expf(-fabsf(z));
    return fmaxf(z, 0.f) + (e < 0.01f ? e * (1.0f - e * (0.5f - e * 0.33333333f)) : __logf(1.0f + e));
  }
};

struct SeqSpan {
  int seq, start, n, row0;       // slot, own position of the first real row, real rows, its row index
};
// the real rows of sequence i of the call
__device__ __forceinline__ SeqSpan seq_span(const SsmArgs& a, int i) {
  SeqSpan s;
  s.seq = a.rows.b0 + i;
  const int p0 = (a.rows.pos0_dev ? *a.rows.pos0_dev : a.rows.pos0_host) - a.pad[s.seq];
  const int skip = min(max(-p0, 0), a.rows.Tc);
  s.start = p0 + skip;
  s.n = a.rows.Tc - skip;
  s.row0 = i * a.rows.Tc + skip;
  return s;
}

constexpr int kConvRows = 8;       // rows per block

template <typename T>
__global__ void __launch_bounds__(256) ssm_conv_kernel(const SsmArgs a) {
  pdl_wait();
  pdl_launch_dependents();
  const int c = blockIdx.x * 256 + threadIdx.x;
  if (c >= a.inner) return;
  const SeqSpan sp = seq_span(a, blockIdx.z);
  const T* x = static_cast<const T*>(a.xz);
  const float* old = a.conv_state + static_cast<size_t>(sp.seq) * (a.taps - 1) * a.ld_u + c;
  const float bias = a.conv_b[c];
  const int t0 = blockIdx.y * kConvRows, base = blockIdx.z * a.rows.Tc;
  for (int t = t0; t < min(t0 + kConvRows, a.rows.Tc); ++t) {
    const int row = base + t, rel = row - sp.row0;        // rel: index among the real rows
    float v = bias;
    if (rel >= 0) {
      for (int j = 0; j < a.taps; ++j) {
        const int back = a.taps - 1 - j;                  // rows back from the current one
        float xv;
        if (rel >= back) xv = ld(x, static_cast<size_t>(row - back) * a.ld_xz + c);
        else if (sp.start + rel >= back) xv = old[static_cast<size_t>(a.taps - 1 + rel - back) * a.ld_u];
        else continue;                                    // before the sequence: zero
        v = fmaf(a.conv_w[static_cast<size_t>(j) * a.ld_u + c], xv, v);
      }
    }
    v = rel >= 0 ? Fn<T>::silu(v) : 0.f;
    const size_t o = static_cast<size_t>(row) * a.ld_u + c;
    if (a.u) a.u[o] = v;
    if (a.u_bf16) a.u_bf16[o] = __float2bfloat16_rn(v);
  }
}

// The same for at most four taps, a thread owning eight neighbouring channels: it walks kVecRows rows with the last
// TAPS - 1 inputs in registers, one 16-byte load per row.  Columns between inner and the row stride hold zeros.
constexpr int kVecRows = 16;

__device__ __forceinline__ void ld8(const __nv_bfloat16* p, float* f) { unpack8(*reinterpret_cast<const uint4*>(p), f); }
__device__ __forceinline__ void ld8(const float* p, float* f) {
  const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
  f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}

template <typename T>
struct Raw8;                       // eight elements as loaded
template <>
struct Raw8<__nv_bfloat16> {
  using V = uint4;
  __device__ static __forceinline__ V load(const __nv_bfloat16* p) { return *reinterpret_cast<const uint4*>(p); }
  __device__ static __forceinline__ void get(const V& v, float* f) { unpack8(v, f); }
};
template <>
struct Raw8<float> {
  struct V { float4 a, b; };
  __device__ static __forceinline__ V load(const float* p) {
    return {reinterpret_cast<const float4*>(p)[0], reinterpret_cast<const float4*>(p)[1]};
  }
  __device__ static __forceinline__ void get(const V& v, float* f) {
    f[0] = v.a.x; f[1] = v.a.y; f[2] = v.a.z; f[3] = v.a.w; f[4] = v.b.x; f[5] = v.b.y; f[6] = v.b.z; f[7] = v.b.w;
  }
};

template <typename T, int TAPS>
__global__ void __launch_bounds__(128) ssm_conv_vec_kernel(const SsmArgs a) {
  pdl_wait();
  pdl_launch_dependents();
  const int c = (blockIdx.x * 128 + threadIdx.x) * 8;
  if (c >= a.ld_u) return;
  const SeqSpan sp = seq_span(a, blockIdx.z);
  const T* x = static_cast<const T*>(a.xz) + c;
  const float* old = a.conv_state + static_cast<size_t>(sp.seq) * (TAPS - 1) * a.ld_u + c;
  float w[TAPS][8], bias[8], hist[TAPS > 1 ? TAPS - 1 : 1][8];
#pragma unroll
  for (int j = 0; j < TAPS; ++j) ld8(a.conv_w + static_cast<size_t>(j) * a.ld_u + c, w[j]);
  ld8(a.conv_b + c, bias);
  const int t0 = blockIdx.y * kVecRows, base = blockIdx.z * a.rows.Tc, t1 = min(t0 + kVecRows, a.rows.Tc);
#pragma unroll
  for (int j = 0; j < TAPS - 1; ++j) {                   // the inputs in front of row t0
    const int rel = base + t0 - sp.row0 - (TAPS - 1) + j;
    if (rel >= 0) ld8(x + static_cast<size_t>(sp.row0 + rel) * a.ld_xz, hist[j]);
    else if (sp.start + rel >= 0 && rel >= -(TAPS - 1)) ld8(old + static_cast<size_t>(TAPS - 1 + rel) * a.ld_u, hist[j]);
    else
#pragma unroll
      for (int e = 0; e < 8; ++e) hist[j][e] = 0.f;
  }
  // two rows ahead in registers; the loop stays rolled, so its code is fetched once
  typename Raw8<T>::V raw0 = Raw8<T>::load(x + static_cast<size_t>(base + t0) * a.ld_xz);
  typename Raw8<T>::V raw1 = Raw8<T>::load(x + static_cast<size_t>(base + min(t0 + 1, t1 - 1)) * a.ld_xz);
#pragma unroll 1
  for (int t = t0; t < t1; ++t) {
    const typename Raw8<T>::V cur = raw0;
    raw0 = raw1;
    raw1 = Raw8<T>::load(x + static_cast<size_t>(base + min(t + 2, t1 - 1)) * a.ld_xz);
    const int row = base + t;
    const bool real = row >= sp.row0;
    float xv[8], v[8];
    Raw8<T>::get(cur, xv);
#pragma unroll
    for (int e = 0; e < 8; ++e) {
      float y = bias[e];
#pragma unroll
      for (int j = 0; j < TAPS - 1; ++j) y = fmaf(w[j][e], hist[j][e], y);
      y = fmaf(w[TAPS - 1][e], xv[e], y);
      v[e] = real ? Fn<T>::silu(y) : 0.f;
    }
    if (real) {
      if constexpr (TAPS > 1) {
#pragma unroll
        for (int j = 0; j < TAPS - 2; ++j)
#pragma unroll
          for (int e = 0; e < 8; ++e) hist[j][e] = hist[j + 1][e];
#pragma unroll
        for (int e = 0; e < 8; ++e) hist[TAPS - 2][e] = xv[e];
      }
    }
    const size_t o = static_cast<size_t>(row) * a.ld_u + c;
    if (a.u) {
      reinterpret_cast<float4*>(a.u + o)[0] = make_float4(v[0], v[1], v[2], v[3]);
      reinterpret_cast<float4*>(a.u + o)[1] = make_float4(v[4], v[5], v[6], v[7]);
    } else {
      *reinterpret_cast<uint4*>(a.u_bf16 + o) =
          make_uint4(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]), pack_bf16x2(v[4], v[5]), pack_bf16x2(v[6], v[7]));
    }
  }
}

// The last taps - 1 inputs of every sequence -> conv_state.  In place: entry j comes from a row of the call or from
// an entry at or behind j.
template <typename T>
__global__ void __launch_bounds__(256) ssm_conv_state_kernel(const SsmArgs a) {
  pdl_wait();
  pdl_launch_dependents();
  const int c = blockIdx.x * 256 + threadIdx.x;
  if (c >= a.inner) return;
  const SeqSpan sp = seq_span(a, blockIdx.y);
  if (sp.n <= 0) return;
  const T* x = static_cast<const T*>(a.xz);
  float* st = a.conv_state + static_cast<size_t>(sp.seq) * (a.taps - 1) * a.ld_u + c;
  for (int j = 0; j < a.taps - 1; ++j) {
    const int rel = sp.n - (a.taps - 1) + j;
    float v = 0.f;
    if (rel >= 0) v = ld(x, static_cast<size_t>(sp.row0 + rel) * a.ld_xz + c);
    else if (sp.start + rel >= 0) v = st[static_cast<size_t>(a.taps - 1 + rel) * a.ld_u];
    st[static_cast<size_t>(j) * a.ld_u] = v;
  }
}

// Decode (one row per sequence): convolution and state shift in one pass over the state.
template <typename T>
__global__ void __launch_bounds__(256) ssm_conv_step_kernel(const SsmArgs a) {
  pdl_wait();
  pdl_launch_dependents();
  const int c = blockIdx.x * 256 + threadIdx.x, m = blockIdx.y;
  if (c >= a.inner) return;
  const SeqSpan sp = seq_span(a, m);
  float* st = a.conv_state + static_cast<size_t>(sp.seq) * (a.taps - 1) * a.ld_u + c;
  const float x = ld(static_cast<const T*>(a.xz), static_cast<size_t>(m) * a.ld_xz + c);
  float v = fmaf(a.conv_w[static_cast<size_t>(a.taps - 1) * a.ld_u + c], x, a.conv_b[c]);
  for (int j = 0; j < a.taps - 1; ++j) {
    const float xv = sp.start >= a.taps - 1 - j ? st[static_cast<size_t>(j) * a.ld_u] : 0.f;
    v = fmaf(a.conv_w[static_cast<size_t>(j) * a.ld_u + c], xv, v);
    if (j > 0) st[static_cast<size_t>(j - 1) * a.ld_u] = xv;
  }
  if (a.taps > 1) st[static_cast<size_t>(a.taps - 2) * a.ld_u] = x;
  v = Fn<T>::silu(v);
  const size_t o = static_cast<size_t>(m) * a.ld_u + c;
  if (a.u) a.u[o] = v;
  if (a.u_bf16) a.u_bf16[o] = __float2bfloat16_rn(v);
}

// xp = sum of the split-K planes of the projection; its dt part once more in bf16, the operand of the next one.
__global__ void __launch_bounds__(64) ssm_split_kernel(const SsmArgs a) {
  pdl_wait();
  pdl_launch_dependents();
  const size_t m = blockIdx.x;
  const int n = a.dt_rank + 2 * a.state, i = blockIdx.y * 64 + threadIdx.x;
  if (i >= n) return;
  const float* src = a.xp_planes + m * n + i;
  const size_t plane = static_cast<size_t>(a.M) * n;
  float v = src[0];
#pragma unroll 16
  for (int p = 1; p < a.planes; ++p) v += src[p * plane];
  a.xp_out[m * a.ld_xp + i] = v;
  if (i < a.dt_rank) a.dtr_bf16[m * a.ld_dtr + i] = __float2bfloat16_rn(v);
}

// The recurrence over a sequence's rows.  G lanes share a channel, each holding NS of its states.  A block is three
// warps that work on CW = 32 / G channels: warp 0 runs the recurrence over a tile of rows, leaving per-lane partial
// outputs, while warp 1 fetches the tile after the next (cp.async: dt, u, z per channel, B and C shared) and finishes the
// step sizes of the next, and warp 2 adds up, gates and stores the outputs of the one behind; one block barrier a tile.  The bound is the exponentials: one per row, channel and state.

template <int BYTES>
__device__ __forceinline__ void cp_async(void* dst, const void* src) {
  if constexpr (BYTES == 16)
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
  else
    asm volatile("cp.async.ca.shared.global [%0], [%1], %2;" ::"r"(smem_u32(dst)), "l"(src), "n"(BYTES) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

// nt rows of CW neighbouring elements -> dst [nt][CW], by one warp
template <typename T, int CW>
__device__ __forceinline__ void tile_rows(T* dst, const T* src, size_t ld_src, int nt, int lane) {
  constexpr int kRow = CW * static_cast<int>(sizeof(T)), kPiece = kRow < 16 ? kRow : 16, kPer = kRow / kPiece, kElems = kPiece / static_cast<int>(sizeof(T));
  for (int i = lane; i < nt * kPer; i += 32) {
    const int t = i / kPer, q = i % kPer * kElems;
    if constexpr (kPiece >= 4) cp_async<kPiece>(dst + t * CW + q, src + t * ld_src + q);
    else dst[t * CW + q] = src[t * ld_src + q];
  }
}

template <int NS>
__device__ __forceinline__ void load_states(const float* p, float* v) {
#pragma unroll
  for (int i = 0; i < NS; i += 4) {
    const float4 f = *reinterpret_cast<const float4*>(p + i);
    v[i] = f.x; v[i + 1] = f.y; v[i + 2] = f.z; v[i + 3] = f.w;
  }
}

// fp32 runs take the accurate exponential, serving runs the hardware's base-2 one (A is scaled by log2 e for it)
template <typename T>
struct Decay;
template <>
struct Decay<float> {
  static constexpr float kScale = 1.0f;
  __device__ static __forceinline__ float f(float x) { return expf(x); }
};
template <>
struct Decay<__nv_bfloat16> {
  static constexpr float kScale = 1.4426950408889634f;
  __device__ static __forceinline__ float f(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
  }
};

template <typename T, int G, int NS>
struct ScanTile {
  static constexpr int CW = 32 / G, NSP = G * NS;
  static constexpr int kTT = NSP <= 64 ? 16 : 8;         // rows
  float B[kTT][NSP], C[kTT][NSP];
  float dt[kTT][CW];
  T u[kTT][CW], z[kTT][CW];
};
template <typename T, int G, int NS>
struct ScanSmem {
  static constexpr int kTT = ScanTile<T, G, NS>::kTT;
  ScanTile<T, G, NS> tile[4];      // behind, current, ahead, arriving
  float2 step[2][kTT][32 / G];     // (dt, dt u)
  float y[2][kTT][33];             // per lane; the padding spreads the last phase's reads over the banks
};

template <typename T, int G, int NS>
__global__ void __launch_bounds__(96) ssm_scan_kernel(const SsmArgs a) {
  using Tile = ScanTile<T, G, NS>;
  constexpr int CW = Tile::CW, NSP = Tile::NSP, kTT = Tile::kTT;
  extern __shared__ __align__(16) unsigned char sc_smem[];
  auto& sm = *reinterpret_cast<ScanSmem<T, G, NS>*>(sc_smem);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const SeqSpan sp = seq_span(a, blockIdx.y);
  const int c0 = blockIdx.x * CW;
  const int tiles = (sp.n + kTT - 1) / kTT;
  for (int i = threadIdx.x; i < static_cast<int>(sizeof(sm.tile) / 4); i += 96) reinterpret_cast<float*>(sm.tile)[i] = 0.f;   // padded states stay zero
  __syncthreads();
  if (warp == 0) {
    const int ch = lane / G, g = lane % G, c = c0 + ch;
    const bool c_ok = c < a.inner;
    float S[NS], A[NS];
    float* state = a.ssm_state + (static_cast<size_t>(sp.seq) * a.inner + (c_ok ? c : 0)) * a.state;
#pragma unroll
    for (int i = 0; i < NS; ++i) {
      const int n = g * NS + i;
      const bool ok = c_ok && n < a.state;
      A[i] = ok ? a.A[static_cast<size_t>(c) * a.state + n] * Decay<T>::kScale : 0.f;
      S[i] = (ok && sp.start > 0 && sp.n > 0) ? state[n] : 0.f;
    }
    __syncthreads();                                     // tile 0 and its steps are ready
    for (int k = 0; k < tiles; ++k) {
      const Tile& d = sm.tile[k & 3];
      const int nt = min(kTT, sp.n - k * kTT);
      // rows in groups: all shared-memory reads of a group come before its writes, which the compiler could not move
      // them over
      constexpr int kU = 4;
      static_assert(kTT % kU == 0 && NS % 4 == 0, "whole groups");
      auto group = [&](int t1, int rows_left) {
        float2 st[kU];
        float Bv[kU][NS], Cv[kU][NS], y[kU];
#pragma unroll
        for (int r = 0; r < kU; ++r) {
          st[r] = sm.step[k & 1][t1 + r][ch];
          load_states<NS>(&d.B[t1 + r][g * NS], Bv[r]);
          load_states<NS>(&d.C[t1 + r][g * NS], Cv[r]);
        }
#pragma unroll
        for (int r = 0; r < kU; ++r) {
          y[r] = 0.f;
          if (r < rows_left) {
#pragma unroll
            for (int i = 0; i < NS; ++i) {
              S[i] = fmaf(Decay<T>::f(st[r].x * A[i]), S[i], st[r].y * Bv[r][i]);
              y[r] = fmaf(S[i], Cv[r][i], y[r]);
            }
          }
        }
#pragma unroll
        for (int r = 0; r < kU; ++r) sm.y[k & 1][t1 + r][lane] = y[r];
      };
      if (nt == kTT) {
#pragma unroll
        for (int t = 0; t < kTT; t += kU) group(t, kU);
      } else {
        for (int t = 0; t < nt; t += kU) group(t, nt - t);
      }
      __syncthreads();
    }
    if (c_ok && sp.n > 0) {
#pragma unroll
      for (int i = 0; i < NS; ++i)
        if (g * NS + i < a.state) state[g * NS + i] = S[i];
    }
    return;
  }
  // warps 1 and 2
  const T* u = (a.u ? reinterpret_cast<const T*>(a.u) : reinterpret_cast<const T*>(a.u_bf16)) + static_cast<size_t>(sp.row0) * a.ld_u + c0;
  const T* z = static_cast<const T*>(a.xz) + static_cast<size_t>(sp.row0) * a.ld_xz + a.z0 + c0;
  const float* dtp = a.dt_raw + static_cast<size_t>(sp.row0) * a.ld_u + c0;
  const float* xp = a.xp + static_cast<size_t>(sp.row0) * a.ld_xp + a.dt_rank;
  const bool wide = ((a.state | a.dt_rank | a.ld_xp) & 3) == 0;
  // 16-byte pieces of a row's B and C, rows that a warp copies at once, this lane's place among them
  const int per = max(a.state >> 1, 1), half = a.state >> 2, rows_at_once = max(32 / per, 1);
  const int wt = per >= 32 ? 0 : lane < rows_at_once * per ? lane / per : kTT, wq = per >= 32 ? lane : lane % per;
  auto fetch = [&](int k) {                              // always commits a group, so that groups count tiles
    if (k < tiles) {
      Tile& d = sm.tile[k & 3];
      const int t0 = k * kTT, nt = min(kTT, sp.n - t0);
      tile_rows<float, CW>(&d.dt[0][0], dtp + static_cast<size_t>(t0) * a.ld_u, a.ld_u, nt, lane);
      tile_rows<T, CW>(&d.u[0][0], u + static_cast<size_t>(t0) * a.ld_u, a.ld_u, nt, lane);
      tile_rows<T, CW>(&d.z[0][0], z + static_cast<size_t>(t0) * a.ld_xz, a.ld_xz, nt, lane);
      if (wide) {                                        // B then C: neighbours in the row, 16 bytes at a time
        for (int t = wt; t < nt; t += rows_at_once) {
          for (int q = wq; q < per; q += 32) {
            float* dst = q < half ? &d.B[t][4 * q] : &d.C[t][4 * (q - half)];
            cp_async<16>(dst, xp + static_cast<size_t>(t0 + t) * a.ld_xp + 4 * q);
          }
        }
      } else {
        for (int n = lane; n < 2 * a.state; n += 32) {
          float* dst = n < a.state ? &d.B[0][n] : &d.C[0][n - a.state];
          const float* src = xp + static_cast<size_t>(t0) * a.ld_xp + n;
#pragma unroll 4
          for (int t = 0; t < nt; ++t) cp_async<4>(dst + t * NSP, src + static_cast<size_t>(t) * a.ld_xp);
        }
      }
    }
    cp_commit();
  };
  // lane -> channel fc, rows t = ft, ft + G, ...
  const int fc = lane % CW, ft = lane / CW;
  const bool f_ok = c0 + fc < a.inner;
  const float dt_b = f_ok ? a.dt_b[c0 + fc] : 0.f, D = f_ok ? a.D[c0 + fc] : 0.f;
  constexpr int kR = kTT / G > 0 ? kTT / G : 1;          // rows per lane
  auto steps = [&](int k) {
    const Tile& d = sm.tile[k & 3];
    float raw[kR], uu[kR];
#pragma unroll
    for (int i = 0; i < kR; ++i) {
      const int t = min(ft + i * G, kTT - 1);
      raw[i] = d.dt[t][fc];
      uu[i] = ld(&d.u[t][fc], 0);
    }
#pragma unroll
    for (int i = 0; i < kR; ++i) {
      const float dt = f_ok ? Fn<T>::softplus(raw[i] + dt_b) : 0.f;
      if (ft + i * G < kTT) sm.step[k & 1][ft + i * G][fc] = make_float2(dt, dt * uu[i]);
    }
  };
  const size_t o0 = static_cast<size_t>(sp.row0 + ft) * a.ld_u + c0 + fc, o_step = static_cast<size_t>(G) * a.ld_u;
  auto finish = [&](int k) {
    const Tile& d = sm.tile[k & 3];
    const int nt = min(kTT, sp.n - k * kTT);
    float yv[kR];
#pragma unroll
    for (int i = 0; i < kR; ++i) {
      const int t = min(ft + i * G, kTT - 1);
      float y = 0.f;
#pragma unroll
      for (int j = 0; j < G; ++j) y += sm.y[k & 1][t][fc * G + j];
      yv[i] = fmaf(D, ld(&d.u[t][fc], 0), y) * Fn<T>::silu(ld(&d.z[t][fc], 0));
    }
    const size_t o = o0 + static_cast<size_t>(k) * kTT * a.ld_u;
#pragma unroll
    for (int i = 0; i < kR; ++i) {
      if (!f_ok || ft + i * G >= nt) continue;
      if (a.out) a.out[o + i * o_step] = yv[i];
      if (a.out_bf16) a.out_bf16[o + i * o_step] = __float2bfloat16_rn(yv[i]);
    }
  };
  if (warp == 1) {
    fetch(0);
    fetch(1);
    cp_wait<1>();
    __syncwarp();                                        // every lane's copies of tile 0 are visible to the warp
    if (tiles > 0) steps(0);
    __syncthreads();
    for (int k = 0; k < tiles; ++k) {
      fetch(k + 2);                                      // over tile k - 2, which nobody reads any more
      cp_wait<1>();
      __syncwarp();
      if (k + 1 < tiles) steps(k + 1);
      __syncthreads();
    }
    return;
  }
  // rows in front of the sequence's start give zeros
  for (int t = ft; t < a.rows.Tc - sp.n; t += G) {
    const size_t o = (static_cast<size_t>(blockIdx.y) * a.rows.Tc + t) * a.ld_u + c0 + fc;
    if (f_ok && a.out) a.out[o] = 0.f;
    if (f_ok && a.out_bf16) a.out_bf16[o] = __float2bfloat16_rn(0.f);
  }
  __syncthreads();
  for (int k = 0; k < tiles; ++k) {
    if (k > 0) finish(k - 1);
    __syncthreads();
  }
  if (tiles > 0) finish(tiles - 1);
}

// Decode, one row per sequence: G lanes per channel do the step size (its projection too, unless dt_raw holds it),
// the state update and the output.  VEC: the state count is a multiple of four and every lane owns four
// neighbouring states (state <= 4 G), so a warp reads and writes whole lines of the state.
template <typename T, int G, bool VEC>
__global__ void __launch_bounds__(256) ssm_step_kernel(const SsmArgs a) {
  extern __shared__ float st_smem[];                     // dt | B | C of the row
  const int m = blockIdx.y, g = threadIdx.x % G, c = blockIdx.x * (256 / G) + threadIdx.x / G;
  const bool ok = c < a.inner;
  const int cc = ok ? c : 0;
  float4 A4 = make_float4(0.f, 0.f, 0.f, 0.f);
  if (VEC && 4 * g < a.state) A4 = *reinterpret_cast<const float4*>(a.A + static_cast<size_t>(cc) * a.state + 4 * g);
  if (!a.dt_raw)
    for (int k = g * 8; k < a.ld_wdt; k += G * 8) prefetch_l2(a.w_dt + static_cast<size_t>(cc) * a.ld_wdt + k);
  pdl_wait();
  pdl_launch_dependents();
  const SeqSpan sp = seq_span(a, m);
  float* state = a.ssm_state + (static_cast<size_t>(sp.seq) * a.inner + cc) * a.state;
  float4 s4 = make_float4(0.f, 0.f, 0.f, 0.f);
  if (VEC && 4 * g < a.state && sp.start > 0) s4 = *reinterpret_cast<const float4*>(state + 4 * g);
  float dt = a.dt_raw ? a.dt_raw[static_cast<size_t>(m) * a.ld_u + cc] : 0.f;
  const float u = a.u ? a.u[static_cast<size_t>(m) * a.ld_u + cc] : __bfloat162float(a.u_bf16[static_cast<size_t>(m) * a.ld_u + cc]);
  const float z = ld(static_cast<const T*>(a.xz), static_cast<size_t>(m) * a.ld_xz + a.z0 + cc);
  const float dt_b = a.dt_b[cc], D = a.D[cc];
  const int np = a.ld_wdt + 2 * a.state;                  // the dt part padded with zeros to the weight's row length
  for (int i = (a.dt_raw ? a.ld_wdt : 0) + threadIdx.x; i < np; i += 256) {
    const float* row = a.xp + static_cast<size_t>(m) * a.ld_xp;
    st_smem[i] = i < a.dt_rank ? row[i] : i < a.ld_wdt ? 0.f : row[a.dt_rank + i - a.ld_wdt];
  }
  __syncthreads();
  if (!a.dt_raw) {
#pragma unroll 4
    for (int k = g * 8; k < a.ld_wdt; k += G * 8) {
      float w8[8];
      unpack8(ld_stream16(a.w_dt + static_cast<size_t>(cc) * a.ld_wdt + k), w8);
#pragma unroll
      for (int e = 0; e < 8; ++e) dt = fmaf(w8[e], st_smem[k + e], dt);
    }
#pragma unroll
    for (int o = G / 2; o > 0; o >>= 1) dt += __shfl_xor_sync(0xffffffffu, dt, o);
  }
  dt = Fn<T>::softplus(dt + dt_b);
  const float du = dt * u;
  const float* B = st_smem + a.ld_wdt;
  const float* C = B + a.state;
  float y = 0.f;
  if (VEC) {
    if (4 * g < a.state) {
      const int n = 4 * g;
      s4.x = fmaf(expf(dt * A4.x), s4.x, du * B[n]);
      s4.y = fmaf(expf(dt * A4.y), s4.y, du * B[n + 1]);
      s4.z = fmaf(expf(dt * A4.z), s4.z, du * B[n + 2]);
      s4.w = fmaf(expf(dt * A4.w), s4.w, du * B[n + 3]);
      if (ok) *reinterpret_cast<float4*>(state + n) = s4;
      y = s4.x * C[n] + s4.y * C[n + 1] + s4.z * C[n + 2] + s4.w * C[n + 3];
    }
  } else {
    for (int n = g; n < a.state; n += G) {
      const float old = sp.start > 0 ? state[n] : 0.f;
      const float s = fmaf(expf(dt * a.A[static_cast<size_t>(cc) * a.state + n]), old, du * B[n]);
      if (ok) state[n] = s;
      y = fmaf(s, C[n], y);
    }
  }
#pragma unroll
  for (int o = G / 2; o > 0; o >>= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
  if (ok && g == 0) {
    y = fmaf(D, u, y) * Fn<T>::silu(z);
    const size_t o = static_cast<size_t>(m) * a.ld_u + c;
    if (a.out) a.out[o] = y;
    if (a.out_bf16) a.out_bf16[o] = __float2bfloat16_rn(y);
  }
}

bool conv_ok(const SsmArgs& a) {
  return a.M > 0 && a.inner > 0 && a.taps >= 1 && a.nseq > 0 && a.rows.Tc > 0 &&
         a.M == a.nseq * a.rows.Tc && a.ld_u >= a.inner && (a.ld_u & 7) == 0 && (a.ld_xz & 7) == 0 && (a.u != nullptr) != (a.u_bf16 != nullptr) &&
         (a.u != nullptr) == !a.xz_bf16;
}
bool ssm_ok(const SsmArgs& a) { return conv_ok(a) && a.state > 0 && a.state <= kSsmMaxState; }

template <typename T, int G, int NS>
cudaError_t scan(const SsmArgs& a, cudaStream_t s) {
  constexpr int smem = static_cast<int>(sizeof(ScanSmem<T, G, NS>)), CW = 32 / G;
  static_assert(smem <= 220 * 1024, "shared memory");
  static DeviceOnce once;
  cudaError_t e = once.run([&] {
    return cudaFuncSetAttribute(ssm_scan_kernel<T, G, NS>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  });
  if (e != cudaSuccess) return e;
  ssm_scan_kernel<T, G, NS><<<dim3((a.inner + CW - 1) / CW, a.nseq), 96, smem, s>>>(a);
  return cudaGetLastError();
}

template <typename T>
cudaError_t scan_states(const SsmArgs& a, cudaStream_t s) {
  if (a.state <= 16) return scan<T, 4, 4>(a, s);
  if (a.state <= 32) return scan<T, 8, 4>(a, s);
  if (a.state <= 64) return scan<T, 16, 4>(a, s);
  if (a.state <= 128) return scan<T, 32, 4>(a, s);
  return scan<T, 32, 8>(a, s);
}

template <typename T, int G, bool VEC>
cudaError_t step(const SsmArgs& a, size_t smem, cudaStream_t s, bool pdl) {
  constexpr int CH = 256 / G;
  return launch_pdl(ssm_step_kernel<T, G, VEC>, dim3((a.inner + CH - 1) / CH, a.M), dim3(256), smem, s, pdl, a);
}

template <typename T>
cudaError_t step_states(const SsmArgs& a, cudaStream_t s, bool pdl) {
  const size_t smem = sizeof(float) * (a.ld_wdt + 2 * static_cast<size_t>(a.state));
  if (smem > 48 * 1024) return cudaErrorInvalidValue;
  if ((a.state & 3) == 0 && a.state <= 128) {
    if (a.state <= 16) return step<T, 4, true>(a, smem, s, pdl);
    if (a.state <= 32) return step<T, 8, true>(a, smem, s, pdl);
    return step<T, 32, true>(a, smem, s, pdl);
  }
  return a.state <= 8 ? step<T, 8, false>(a, smem, s, pdl) : step<T, 32, false>(a, smem, s, pdl);
}

template <typename T>
cudaError_t conv_vec(const SsmArgs& a, cudaStream_t s, bool pdl) {
  const dim3 grid((a.ld_u / 8 + 127) / 128, (a.rows.Tc + kVecRows - 1) / kVecRows, a.nseq);
  switch (a.taps) {
    case 1: return launch_pdl(ssm_conv_vec_kernel<T, 1>, grid, dim3(128), 0, s, pdl, a);
    case 2: return launch_pdl(ssm_conv_vec_kernel<T, 2>, grid, dim3(128), 0, s, pdl, a);
    case 3: return launch_pdl(ssm_conv_vec_kernel<T, 3>, grid, dim3(128), 0, s, pdl, a);
    default: return launch_pdl(ssm_conv_vec_kernel<T, 4>, grid, dim3(128), 0, s, pdl, a);
  }
}

}  // namespace

cudaError_t launch_ssm_conv(const SsmArgs& a, cudaStream_t s, bool pdl) {
  if (!conv_ok(a)) return cudaErrorInvalidValue;
  const int cb = (a.inner + 255) / 256;
  if (a.rows.Tc == 1)
    return a.xz_bf16 ? launch_pdl(ssm_conv_step_kernel<__nv_bfloat16>, dim3(cb, a.M), dim3(256), 0, s, pdl, a)
                     : launch_pdl(ssm_conv_step_kernel<float>, dim3(cb, a.M), dim3(256), 0, s, pdl, a);
  const dim3 grid(cb, (a.rows.Tc + kConvRows - 1) / kConvRows, a.nseq);
  cudaError_t e = a.taps <= 4 ? (a.xz_bf16 ? conv_vec<__nv_bfloat16>(a, s, pdl) : conv_vec<float>(a, s, pdl))
                  : a.xz_bf16 ? launch_pdl(ssm_conv_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, pdl, a)
                              : launch_pdl(ssm_conv_kernel<float>, grid, dim3(256), 0, s, pdl, a);
  if (e != cudaSuccess || a.taps == 1) return e;
  return a.xz_bf16 ? launch_pdl(ssm_conv_state_kernel<__nv_bfloat16>, dim3(cb, a.nseq), dim3(256), 0, s, pdl, a)
                   : launch_pdl(ssm_conv_state_kernel<float>, dim3(cb, a.nseq), dim3(256), 0, s, pdl, a);
}

cudaError_t launch_ssm_split(const SsmArgs& a, cudaStream_t s, bool pdl) {
  if (!ssm_ok(a) || !a.dtr_bf16 || !a.xp_planes || !a.xp_out || a.planes < 1) return cudaErrorInvalidValue;
  return launch_pdl(ssm_split_kernel, dim3(a.M, (a.dt_rank + 2 * a.state + 63) / 64), dim3(64), 0, s, pdl, a);
}

cudaError_t launch_ssm_scan(const SsmArgs& a, cudaStream_t s) {
  if (!ssm_ok(a) || !a.dt_raw || (a.ld_u & 7) || (a.ld_xz & 7) || (a.z0 & 7)) return cudaErrorInvalidValue;
  return a.xz_bf16 ? scan_states<__nv_bfloat16>(a, s) : scan_states<float>(a, s);
}

cudaError_t launch_ssm_step(const SsmArgs& a, cudaStream_t s, bool pdl) {
  if (!ssm_ok(a) || a.rows.Tc != 1) return cudaErrorInvalidValue;
  return a.xz_bf16 ? step_states<__nv_bfloat16>(a, s, pdl) : step_states<float>(a, s, pdl);
}

}  // namespace mtj
