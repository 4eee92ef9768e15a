// Recurrences whose state is a matrix S [keys, values] per head, fp32, carried per sequence slot:
//     SSD    S <- exp(A dt) S + dt k v^T,  o = S^T q + D v
//     delta  S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q     (g per key channel)
// and the norm and gate of their outputs.  The columns of S (one per value channel) are independent of each other, so
// blocks own column groups of a head and nothing is exchanged between them.  A sequence whose first row is in the call
// starts from zeros whatever its slot holds; rows before the start (left padding) change nothing and give zeros.
//
// This file walks the rows one by one: matrix_scan_kernel (short portions, 32-bit runs) and matrix_step_kernel (one row
// per sequence: the state passes through registers once, 16 bytes a load); mtj_matrix_chunk.cu takes long prompts in
// chunks on the tensor cores.
#include <math.h>

#include <algorithm>

#include "mtj_common.cuh"
#include "mtj_matrix_state.cuh"

namespace mtj {
namespace {

constexpr int kMsThreads = 128;
constexpr int kMsKL = 8;             // lanes that share a column, each holding every 8th group of four keys
constexpr int kMsCols = 32;          // columns per block: a warp has 4 column lanes of 2 columns
constexpr int kMsRows = 16;          // rows staged at a time

template <int NK>
struct MsSmem {
  static constexpr int DP = kMsKL * NK;
  float k[kMsRows][DP], q[kMsRows][DP], g[kMsRows][DP];
  float v[kMsRows][kMsCols];
  float2 c[kMsRows];                 // SSD: (decay, dt); delta: (beta, -)
};

template <typename T, bool DELTA, int NK>
__global__ void __launch_bounds__(kMsThreads) matrix_scan_kernel(const MatrixStateArgs a) {
  using Smem = MsSmem<NK>;
  constexpr int DP = Smem::DP, NQ = NK / 4;
  extern __shared__ __align__(16) unsigned char ms_smem[];
  Smem& sm = *reinterpret_cast<Smem*>(ms_smem);
  const int head = blockIdx.x, c0 = blockIdx.y * kMsCols;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int kl = lane & (kMsKL - 1), cl = lane / kMsKL;
  const int col = warp * 8 + cl * 2;                     // first of this lane's two columns within the block
  const bool ok0 = c0 + col < a.vdim, ok1 = c0 + col + 1 < a.vdim;
  const int kh = head / (a.heads / a.key_heads);
  const float A = a.A[head], D = DELTA ? 0.f : a.D[head], bias = DELTA ? 0.f : a.decay_b[head];
  pdl_wait();
  pdl_launch_dependents();
  const MsSpan sp = ms_span(a, blockIdx.z);
  const T* u = static_cast<const T*>(a.u);
  float S[2][NK];                                        // S[c][4 j + e]: key (8 j + kl) * 4 + e
  float* state = a.state + (static_cast<size_t>(sp.seq) * a.heads + head) * a.dim * a.vdim + c0 + col;
#pragma unroll
  for (int j = 0; j < NQ; ++j)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int n = (j * kMsKL + kl) * 4 + e;
      const bool have = n < a.dim && sp.start > 0 && sp.n > 0;
      S[0][4 * j + e] = have && ok0 ? state[static_cast<size_t>(n) * a.vdim] : 0.f;
      S[1][4 * j + e] = have && ok1 ? state[static_cast<size_t>(n) * a.vdim + 1] : 0.f;
    }
  for (int t = threadIdx.x; t < (a.rows.Tc - sp.n) * kMsCols; t += kMsThreads) {     // rows in front of the start
    const int c = c0 + t % kMsCols;
    if (c < a.vdim) a.out[static_cast<size_t>(blockIdx.z * a.rows.Tc + t / kMsCols) * a.ld_out + head * a.vdim + c] = 0.f;
  }
  for (int t0 = 0; t0 < sp.n; t0 += kMsRows) {
    const int nt = min(kMsRows, sp.n - t0);
    __syncthreads();                                     // the last tile has been read
    for (int t = warp; t < nt; t += kMsThreads / 32) {
      const size_t m = static_cast<size_t>(sp.row0 + t0 + t);
      const T* row = u + m * a.ld_u;
      float kv[DP / 32 > 0 ? DP / 32 : 1], qv[DP / 32 > 0 ? DP / 32 : 1], ks = 0.f, qs = 0.f;
#pragma unroll
      for (int i = 0; i < DP / 32; ++i) {
        const int n = i * 32 + lane;
        kv[i] = n < a.dim ? ms_ld(row, a.k0 + kh * a.dim + n) : 0.f;
        qv[i] = n < a.dim ? ms_ld(row, a.q0 + kh * a.dim + n) : 0.f;
        ks = fmaf(kv[i], kv[i], ks);
        qs = fmaf(qv[i], qv[i], qs);
      }
      float kr = 1.f, qr = 1.f;
      if (DELTA) {
        kr = 1.0f / sqrtf(warp_sum(ks) + kUnitEps);
        qr = a.q_scale / sqrtf(warp_sum(qs) + kUnitEps);
      }
#pragma unroll
      for (int i = 0; i < DP / 32; ++i) {
        const int n = i * 32 + lane;
        sm.k[t][n] = kv[i] * kr;
        sm.q[t][n] = qv[i] * qr;
        if (DELTA)
          sm.g[t][n] = n < a.dim ? MsFn<T>::exp(A * MsFn<T>::softplus(a.decay[m * a.ld_decay + head * a.dim + n] + a.decay_b[head * a.dim + n])) : 0.f;
      }
      sm.v[t][lane] = c0 + lane < a.vdim ? ms_ld(row, a.v0 + head * a.vdim + c0 + lane) : 0.f;
      if (lane == 0) {
        if (DELTA) {
          sm.c[t] = make_float2(MsFn<T>::sigmoid(a.beta[m * a.ld_beta + head]), 0.f);
        } else {
          const float dt = MsFn<T>::softplus(a.decay[m * a.ld_decay + head] + bias);
          sm.c[t] = make_float2(MsFn<T>::exp(A * dt), dt);
        }
      }
    }
    __syncthreads();
    for (int t = 0; t < nt; ++t) {
      const float2 c = sm.c[t];
      const float2 v = *reinterpret_cast<const float2*>(&sm.v[t][col]);
      float kf[NK];
#pragma unroll
      for (int j = 0; j < NQ; ++j) {
        const float4 f = *reinterpret_cast<const float4*>(&sm.k[t][(j * kMsKL + kl) * 4]);
        kf[4 * j] = f.x; kf[4 * j + 1] = f.y; kf[4 * j + 2] = f.z; kf[4 * j + 3] = f.w;
      }
      float u0, u1;
      if (DELTA) {
        float r0 = 0.f, r1 = 0.f;
#pragma unroll
        for (int j = 0; j < NQ; ++j) {
          const float4 f = *reinterpret_cast<const float4*>(&sm.g[t][(j * kMsKL + kl) * 4]);
          const float gf[4] = {f.x, f.y, f.z, f.w};
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            S[0][4 * j + e] *= gf[e];
            S[1][4 * j + e] *= gf[e];
            r0 = fmaf(S[0][4 * j + e], kf[4 * j + e], r0);
            r1 = fmaf(S[1][4 * j + e], kf[4 * j + e], r1);
          }
        }
#pragma unroll
        for (int o = 1; o < kMsKL; o <<= 1) {
          r0 += __shfl_xor_sync(0xffffffffu, r0, o);
          r1 += __shfl_xor_sync(0xffffffffu, r1, o);
        }
        u0 = c.x * (v.x - r0);
        u1 = c.x * (v.y - r1);
      } else {
        u0 = c.y * v.x;
        u1 = c.y * v.y;
      }
      float y0 = 0.f, y1 = 0.f;
#pragma unroll
      for (int j = 0; j < NQ; ++j) {
        const float4 f = *reinterpret_cast<const float4*>(&sm.q[t][(j * kMsKL + kl) * 4]);
        const float qf[4] = {f.x, f.y, f.z, f.w};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          float s0 = S[0][4 * j + e], s1 = S[1][4 * j + e];
          if (!DELTA) {
            s0 *= c.x;
            s1 *= c.x;
          }
          s0 = fmaf(kf[4 * j + e], u0, s0);
          s1 = fmaf(kf[4 * j + e], u1, s1);
          y0 = fmaf(s0, qf[e], y0);
          y1 = fmaf(s1, qf[e], y1);
          S[0][4 * j + e] = s0;
          S[1][4 * j + e] = s1;
        }
      }
#pragma unroll
      for (int o = 1; o < kMsKL; o <<= 1) {
        y0 += __shfl_xor_sync(0xffffffffu, y0, o);
        y1 += __shfl_xor_sync(0xffffffffu, y1, o);
      }
      if (kl == 0) {
        float* o = a.out + static_cast<size_t>(sp.row0 + t0 + t) * a.ld_out + head * a.vdim + c0 + col;
        if (ok0) o[0] = fmaf(D, v.x, y0);
        if (ok1) o[1] = fmaf(D, v.y, y1);
      }
    }
  }
  if (sp.n > 0) {
#pragma unroll
    for (int j = 0; j < NQ; ++j)
#pragma unroll
      for (int e = 0; e < 4; ++e) {
        const int n = (j * kMsKL + kl) * 4 + e;
        if (n < a.dim && ok0) state[static_cast<size_t>(n) * a.vdim] = S[0][4 * j + e];
        if (n < a.dim && ok1) state[static_cast<size_t>(n) * a.vdim + 1] = S[1][4 * j + e];
      }
  }
}

template <typename T, bool DELTA, int NK>
cudaError_t scan(const MatrixStateArgs& a, cudaStream_t s, bool pdl) {
  constexpr int smem = static_cast<int>(sizeof(MsSmem<NK>));
  static_assert(smem <= 220 * 1024, "shared memory");
  static DeviceOnce once;
  cudaError_t e = once.run([&] {
    return cudaFuncSetAttribute(matrix_scan_kernel<T, DELTA, NK>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
  });
  if (e != cudaSuccess) return e;
  return launch_pdl(matrix_scan_kernel<T, DELTA, NK>, dim3(a.heads, (a.vdim + kMsCols - 1) / kMsCols, a.nseq), dim3(kMsThreads), smem, s, pdl, a);
}

template <typename T, bool DELTA>
cudaError_t scan_keys(const MatrixStateArgs& a, cudaStream_t s, bool pdl) {
  if (a.dim <= 32) return scan<T, DELTA, 4>(a, s, pdl);
  if (a.dim <= 64) return scan<T, DELTA, 8>(a, s, pdl);
  if (a.dim <= 128) return scan<T, DELTA, 16>(a, s, pdl);
  return scan<T, DELTA, 32>(a, s, pdl);
}

// ---- one row per sequence.  A block owns up to 128 columns of a head; a thread holds four neighbouring columns of
// every RPP-th key, so a row of the state is read and written in whole lines.
constexpr int kStepThreads = 256, kStepCols = 128;

template <typename T, bool DELTA, int NI>
__global__ void __launch_bounds__(kStepThreads) matrix_step_kernel(const MatrixStateArgs a, const GatedNormArgs nm, int norm) {
  __shared__ float sk[kMatrixMaxDim], sq[kMatrixMaxDim], sg[DELTA ? kMatrixMaxDim : 1], su[kStepCols], sv[kStepCols];
  __shared__ __align__(16) float part[4 * kStepThreads];
  __shared__ float red[3][kStepThreads / 32];
  const int head = blockIdx.x, c0 = blockIdx.y * kStepCols, cols = min(kStepCols, a.vdim - c0), m = blockIdx.z;
  const int lpr = cols >> 2, rpp = kStepThreads / lpr, r = threadIdx.x / lpr, c4 = threadIdx.x % lpr * 4;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, t = threadIdx.x;
  const int kh = head / (a.heads / a.key_heads);
  const float A = a.A[head];
  float bias = 0.f;
  if (DELTA) bias = t < a.dim ? a.decay_b[head * a.dim + t] : 0.f;
  else bias = a.decay_b[head];
  // the state was written kernels ago: it does not wait for the predecessor
  const MsSpan sp = ms_span(a, m);
  float4* state = reinterpret_cast<float4*>(a.state + (static_cast<size_t>(sp.seq) * a.heads + head) * a.dim * a.vdim + c0 + c4);
  const int ld4 = a.vdim >> 2;
  float4 S[NI];
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int n = r + i * rpp;
    S[i] = r < rpp && n < a.dim && sp.start > 0 ? state[static_cast<size_t>(n) * ld4] : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  pdl_wait();
  pdl_launch_dependents();
  const T* row = static_cast<const T*>(a.u) + static_cast<size_t>(m) * a.ld_u;
  const float k = t < a.dim ? ms_ld(row, a.k0 + kh * a.dim + t) : 0.f, q = t < a.dim ? ms_ld(row, a.q0 + kh * a.dim + t) : 0.f;
  if (t < cols) sv[t] = ms_ld(row, a.v0 + head * a.vdim + c0 + t);
  float c_decay = 0.f, c_in = 0.f;                       // SSD: decay and step size; delta: update strength in c_in
  if (DELTA) {
    const float d = t < a.dim ? a.decay[static_cast<size_t>(m) * a.ld_decay + head * a.dim + t] + bias : 0.f;
    c_in = MsFn<T>::sigmoid(a.beta[static_cast<size_t>(m) * a.ld_beta + head]);
    const float ks = warp_sum(k * k), qs = warp_sum(q * q);
    if (lane == 0) {
      red[0][warp] = ks;
      red[1][warp] = qs;
    }
    if (t < a.dim) sg[t] = MsFn<T>::exp(A * MsFn<T>::softplus(d));
    __syncthreads();
    float kt = 0.f, qt = 0.f;
#pragma unroll
    for (int i = 0; i < kStepThreads / 32; ++i) {
      kt += red[0][i];
      qt += red[1][i];
    }
    if (t < a.dim) {
      sk[t] = k / sqrtf(kt + kUnitEps);
      sq[t] = q * a.q_scale / sqrtf(qt + kUnitEps);
    }
  } else {
    c_in = MsFn<T>::softplus(a.decay[static_cast<size_t>(m) * a.ld_decay + head] + bias);
    c_decay = MsFn<T>::exp(A * c_in);
    if (t < a.dim) {
      sk[t] = k;
      sq[t] = q;
    }
  }
  __syncthreads();
  auto column = [&](int c) {                             // sum of the threads' partial results for column c
    float v = 0.f;
#pragma unroll 8
    for (int i = 0; i < rpp; ++i) v += part[i * cols + c];
    return v;
  };
  float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
  if (DELTA) {
#pragma unroll
    for (int i = 0; i < NI; ++i) {
      const int n = r + i * rpp;
      const float g = n < a.dim ? sg[n] : 0.f, kn = n < a.dim ? sk[n] : 0.f;
      S[i].x *= g; S[i].y *= g; S[i].z *= g; S[i].w *= g;
      acc.x = fmaf(S[i].x, kn, acc.x); acc.y = fmaf(S[i].y, kn, acc.y); acc.z = fmaf(S[i].z, kn, acc.z); acc.w = fmaf(S[i].w, kn, acc.w);
    }
    if (r < rpp) *reinterpret_cast<float4*>(&part[r * cols + c4]) = acc;
    __syncthreads();
    if (t < cols) su[t] = c_in * (sv[t] - column(t));
  } else if (t < cols) {
    su[t] = c_in * sv[t];
  }
  __syncthreads();
  const float4 u = r < rpp ? *reinterpret_cast<const float4*>(&su[c4]) : make_float4(0.f, 0.f, 0.f, 0.f);
  acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
  for (int i = 0; i < NI; ++i) {
    const int n = r + i * rpp;
    const float kn = n < a.dim ? sk[n] : 0.f, qn = n < a.dim ? sq[n] : 0.f;
    float4 s = S[i];
    if (!DELTA) { s.x *= c_decay; s.y *= c_decay; s.z *= c_decay; s.w *= c_decay; }
    s.x = fmaf(kn, u.x, s.x); s.y = fmaf(kn, u.y, s.y); s.z = fmaf(kn, u.z, s.z); s.w = fmaf(kn, u.w, s.w);
    acc.x = fmaf(s.x, qn, acc.x); acc.y = fmaf(s.y, qn, acc.y); acc.z = fmaf(s.z, qn, acc.z); acc.w = fmaf(s.w, qn, acc.w);
    if (r < rpp && n < a.dim && sp.n > 0) state[static_cast<size_t>(n) * ld4] = s;
  }
  if (r < rpp) *reinterpret_cast<float4*>(&part[r * cols + c4]) = acc;
  __syncthreads();
  float y = 0.f;
  if (t < cols) {
    y = column(t);
    if (!DELTA) y = fmaf(a.D[head], sv[t], y);
    if (sp.n <= 0) y = 0.f;
  }
  if (DELTA && norm) {                                   // the block holds the whole head
    const float s = warp_sum(y * y);
    if (lane == 0) red[2][warp] = s;
    __syncthreads();
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < kStepThreads / 32; ++i) ss += red[2][i];
    if (t < cols) {
      const int c = head * a.vdim + t;
      y *= nm.w[t] / sqrtf(ss / static_cast<float>(a.vdim) + nm.eps);
      y *= MsFn<T>::sigmoid(ms_ld(static_cast<const T*>(nm.gate), static_cast<size_t>(m) * nm.ld_gate + c));
      const size_t o = static_cast<size_t>(m) * nm.ld_out + c;
      if (nm.out) nm.out[o] = y;
      if (nm.out_bf16) nm.out_bf16[o] = __float2bfloat16_rn(y);
    }
  } else if (t < cols) {
    a.out[static_cast<size_t>(m) * a.ld_out + head * a.vdim + c0 + t] = y;
  }
}

template <typename T, bool DELTA>
cudaError_t step(const MatrixStateArgs& a, const GatedNormArgs* norm, cudaStream_t s, bool pdl) {
  const dim3 grid(a.heads, (a.vdim + kStepCols - 1) / kStepCols, a.M);
  const int rpp = kStepThreads / (std::min(a.vdim, kStepCols) / 4), ni = (a.dim + rpp - 1) / rpp;
  const GatedNormArgs nm = norm ? *norm : GatedNormArgs{};
  auto go = [&](auto kernel) { return launch_pdl(kernel, grid, dim3(kStepThreads), 0, s, pdl, a, nm, norm ? 1 : 0); };
  if (ni <= 4) return go(matrix_step_kernel<T, DELTA, 4>);
  if (ni <= 8) return go(matrix_step_kernel<T, DELTA, 8>);
  if (ni <= 16) return go(matrix_step_kernel<T, DELTA, 16>);
  return go(matrix_step_kernel<T, DELTA, 32>);
}

// ---- norm and gate of the outputs: one group of TH threads per (row, part)
__device__ __forceinline__ float4 ms_ld4(const float* p, size_t i) { return *reinterpret_cast<const float4*>(p + i); }
__device__ __forceinline__ float4 ms_ld4(const __nv_bfloat16* p, size_t i) {
  const uint2 w = *reinterpret_cast<const uint2*>(p + i);
  return make_float4(bf16_lo(w.x), bf16_hi(w.x), bf16_lo(w.y), bf16_hi(w.y));
}
__device__ __forceinline__ float4 mul4(const float4& x, const float4& y) { return make_float4(x.x * y.x, x.y * y.y, x.z * y.z, x.w * y.w); }
template <typename F>
__device__ __forceinline__ float4 map4(const float4& x, F&& f) { return make_float4(f(x.x), f(x.y), f(x.z), f(x.w)); }

// part_n and the row strides multiples of four, part_n up to 4 TH HOLD: four neighbouring columns a thread, loads first
template <typename T, int TH, int HOLD>
__global__ void __launch_bounds__(256) gated_norm_vec_kernel(const GatedNormArgs a) {
  __shared__ float red[8];
  pdl_wait();
  pdl_launch_dependents();
  constexpr int kGroups = 256 / TH, kHold = HOLD;
  const int grp = threadIdx.x / TH, t = threadIdx.x % TH;
  const int64_t id = static_cast<int64_t>(blockIdx.x) * kGroups + grp;
  if (id >= static_cast<int64_t>(a.M) * a.parts) return;   // whole groups leave; with TH = 256 the grid is exact
  const size_t m = static_cast<size_t>(id / a.parts);
  const int c0 = static_cast<int>(id % a.parts) * a.part_n;
  const float* y = a.y + m * a.ld_y + c0;
  const T* gate = static_cast<const T*>(a.gate) + m * a.ld_gate + c0;
  float4 v[kHold], g[kHold];
#pragma unroll
  for (int j = 0; j < kHold; ++j) {
    const int i = 4 * (j * TH + t);
    v[j] = i < a.part_n ? ms_ld4(y, i) : make_float4(0.f, 0.f, 0.f, 0.f);
    g[j] = i < a.part_n ? ms_ld4(gate, i) : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  float ss = 0.f;
#pragma unroll
  for (int j = 0; j < kHold; ++j) {
    if (a.gate_first) v[j] = mul4(v[j], map4(g[j], [](float z) { return MsFn<T>::silu(z); }));
    ss += (v[j].x * v[j].x + v[j].y * v[j].y) + (v[j].z * v[j].z + v[j].w * v[j].w);
  }
  ss = warp_sum(ss);
  if (TH > 32) {
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
    __syncthreads();
    ss = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) ss += red[i];
  }
  const float rs = 1.0f / sqrtf(ss / static_cast<float>(a.part_n) + a.eps);
#pragma unroll
  for (int j = 0; j < kHold; ++j) {
    const int i = 4 * (j * TH + t);
    if (i >= a.part_n) continue;
    float4 o = mul4(map4(v[j], [&](float z) { return z * rs; }), ms_ld4(a.w, a.gate_first ? c0 + i : i));
    if (!a.gate_first) o = mul4(o, map4(g[j], [](float z) { return MsFn<T>::sigmoid(z); }));
    const size_t at = m * a.ld_out + c0 + i;
    if (a.out) *reinterpret_cast<float4*>(a.out + at) = o;
    if (a.out_bf16) *reinterpret_cast<uint2*>(a.out_bf16 + at) = make_uint2(pack_bf16x2(o.x, o.y), pack_bf16x2(o.z, o.w));
  }
}

template <typename T, int TH>
__global__ void __launch_bounds__(256) gated_norm_kernel(const GatedNormArgs a) {
  __shared__ float red[8];
  pdl_wait();
  pdl_launch_dependents();
  constexpr int kGroups = 256 / TH;
  const int grp = threadIdx.x / TH, t = threadIdx.x % TH;
  const int64_t id = static_cast<int64_t>(blockIdx.x) * kGroups + grp;
  if (id >= static_cast<int64_t>(a.M) * a.parts) return;   // whole groups leave; with TH = 256 the grid is exact
  const size_t m = static_cast<size_t>(id / a.parts);
  const int part = static_cast<int>(id % a.parts), c0 = part * a.part_n;
  const float* y = a.y + m * a.ld_y + c0;
  const T* gate = static_cast<const T*>(a.gate) + m * a.ld_gate + c0;
  constexpr int kHold = 8;                               // values a thread keeps; longer parts are read twice
  float held[kHold], ss = 0.f;
  auto value = [&](int i) {
    const float v = y[i];
    return a.gate_first ? v * MsFn<T>::silu(ms_ld(gate, i)) : v;
  };
#pragma unroll
  for (int j = 0; j < kHold; ++j) {
    const int i = j * TH + t;
    held[j] = i < a.part_n ? value(i) : 0.f;
    ss = fmaf(held[j], held[j], ss);
  }
  for (int i = kHold * TH + t; i < a.part_n; i += TH) {
    const float v = value(i);
    ss = fmaf(v, v, ss);
  }
  ss = warp_sum(ss);
  if (TH > 32) {
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
    __syncthreads();
    ss = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) ss += red[i];
  }
  const float rs = 1.0f / sqrtf(ss / static_cast<float>(a.part_n) + a.eps);
  auto store = [&](int i, float v) {
    v *= rs * a.w[a.gate_first ? c0 + i : i];
    if (!a.gate_first) v *= MsFn<T>::sigmoid(ms_ld(gate, i));
    const size_t o = m * a.ld_out + c0 + i;
    if (a.out) a.out[o] = v;
    if (a.out_bf16) a.out_bf16[o] = __float2bfloat16_rn(v);
  };
#pragma unroll
  for (int j = 0; j < kHold; ++j)
    if (j * TH + t < a.part_n) store(j * TH + t, held[j]);
  for (int i = kHold * TH + t; i < a.part_n; i += TH) store(i, value(i));
}

template <typename T>
cudaError_t gated_norm(const GatedNormArgs& a, cudaStream_t s, bool pdl) {
  const int64_t n = static_cast<int64_t>(a.M) * a.parts;
  if (((a.part_n | a.ld_y | a.ld_gate | a.ld_out) & 3) == 0 && a.part_n <= 16 * 256)
  {
    const dim3 eight(static_cast<unsigned>((n + 7) / 8)), one(static_cast<unsigned>(n)), block(256);
    if (a.part_n <= 128) return launch_pdl(gated_norm_vec_kernel<T, 32, 1>, eight, block, 0, s, pdl, a);
    if (a.part_n <= 512) return launch_pdl(gated_norm_vec_kernel<T, 32, 4>, eight, block, 0, s, pdl, a);
    return a.part_n <= 1024 ? launch_pdl(gated_norm_vec_kernel<T, 256, 1>, one, block, 0, s, pdl, a) : launch_pdl(gated_norm_vec_kernel<T, 256, 4>, one, block, 0, s, pdl, a);
  }
  if (a.part_n <= 256) return launch_pdl(gated_norm_kernel<T, 32>, dim3(static_cast<unsigned>((n + 7) / 8)), dim3(256), 0, s, pdl, a);
  return launch_pdl(gated_norm_kernel<T, 256>, dim3(static_cast<unsigned>(n)), dim3(256), 0, s, pdl, a);
}

}  // namespace

cudaError_t launch_matrix_scan(const MatrixStateArgs& a, cudaStream_t s, bool pdl) {
  if (!matrix_state_ok(a)) return cudaErrorInvalidValue;
  if (a.u_bf16) return a.delta ? scan_keys<__nv_bfloat16, true>(a, s, pdl) : scan_keys<__nv_bfloat16, false>(a, s, pdl);
  return a.delta ? scan_keys<float, true>(a, s, pdl) : scan_keys<float, false>(a, s, pdl);
}

bool matrix_step_ok(const MatrixStateArgs& a) { return a.rows.Tc == 1 && (a.vdim & 3) == 0 && a.M <= 65535; }
bool matrix_step_norms(const MatrixStateArgs& a) { return matrix_step_ok(a) && a.delta && a.vdim <= kStepCols; }

cudaError_t launch_matrix_step(const MatrixStateArgs& a, const GatedNormArgs* norm, cudaStream_t s, bool pdl) {
  if (!matrix_state_ok(a) || !matrix_step_ok(a) || (norm && !matrix_step_norms(a))) return cudaErrorInvalidValue;
  if (norm && (norm->gate_bf16 != 0) != (a.u_bf16 != 0)) return cudaErrorInvalidValue;
  if (a.u_bf16) return a.delta ? step<__nv_bfloat16, true>(a, norm, s, pdl) : step<__nv_bfloat16, false>(a, norm, s, pdl);
  return a.delta ? step<float, true>(a, norm, s, pdl) : step<float, false>(a, norm, s, pdl);
}

cudaError_t launch_gated_norm(const GatedNormArgs& a, cudaStream_t s, bool pdl) {
  if (a.M <= 0 || a.parts <= 0 || a.part_n <= 0 || !a.y || !a.gate || !a.w) return cudaErrorInvalidValue;
  return a.gate_bf16 ? gated_norm<__nv_bfloat16>(a, s, pdl) : gated_norm<float>(a, s, pdl);
}

}  // namespace mtj
