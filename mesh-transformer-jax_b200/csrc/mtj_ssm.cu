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
__device__ __forceinline__ float silu(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }

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
  const float* old = a.conv_state + static_cast<size_t>(sp.seq) * (a.taps - 1) * a.inner + c;
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
        else if (sp.start + rel >= back) xv = old[static_cast<size_t>(a.taps - 1 + rel - back) * a.inner];
        else continue;                                    // before the sequence: zero
        v = fmaf(a.conv_w[static_cast<size_t>(j) * a.ld_u + c], xv, v);
      }
    }
    v = rel >= 0 ? silu(v) : 0.f;
    const size_t o = static_cast<size_t>(row) * a.ld_u + c;
    if (a.u) a.u[o] = v;
    if (a.u_bf16) a.u_bf16[o] = __float2bfloat16_rn(v);
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
  float* st = a.conv_state + static_cast<size_t>(sp.seq) * (a.taps - 1) * a.inner + c;
  for (int j = 0; j < a.taps - 1; ++j) {
    const int rel = sp.n - (a.taps - 1) + j;
    float v = 0.f;
    if (rel >= 0) v = ld(x, static_cast<size_t>(sp.row0 + rel) * a.ld_xz + c);
    else if (sp.start + rel >= 0) v = st[static_cast<size_t>(a.taps - 1 + rel) * a.inner];
    st[static_cast<size_t>(j) * a.inner] = v;
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
  float* st = a.conv_state + static_cast<size_t>(sp.seq) * (a.taps - 1) * a.inner + c;
  const float x = ld(static_cast<const T*>(a.xz), static_cast<size_t>(m) * a.ld_xz + c);
  float v = fmaf(a.conv_w[static_cast<size_t>(a.taps - 1) * a.ld_u + c], x, a.conv_b[c]);
  for (int j = 0; j < a.taps - 1; ++j) {
    const float xv = sp.start >= a.taps - 1 - j ? st[static_cast<size_t>(j) * a.inner] : 0.f;
    v = fmaf(a.conv_w[static_cast<size_t>(j) * a.ld_u + c], xv, v);
    if (j > 0) st[static_cast<size_t>(j - 1) * a.inner] = xv;
  }
  if (a.taps > 1) st[static_cast<size_t>(a.taps - 2) * a.inner] = x;
  v = silu(v);
  const size_t o = static_cast<size_t>(m) * a.ld_u + c;
  if (a.u) a.u[o] = v;
  if (a.u_bf16) a.u_bf16[o] = __float2bfloat16_rn(v);
}

__global__ void ssm_split_kernel(const SsmArgs a) {
  const size_t m = blockIdx.x;
  for (int i = threadIdx.x; i < a.dt_rank; i += blockDim.x)
    a.dtr_bf16[m * a.ld_dtr + i] = __float2bfloat16_rn(a.xp[m * a.ld_xp + i]);
}

// The recurrence over a sequence's rows.  G lanes share a channel, each holding NS of its states; a block covers
// 128 / G channels and stages kTT rows of dt, u, z (per channel) and B, C (shared) in shared memory.
constexpr int kScanThreads = 128;
constexpr int kTT = 32;

template <typename T, int G, int NS>
__global__ void __launch_bounds__(kScanThreads) ssm_scan_kernel(const SsmArgs a) {
  constexpr int CH = kScanThreads / G;
  extern __shared__ float sc_smem[];
  const int nsp = G * NS;                                // states, padded
  float* sB = sc_smem;                                   // [kTT][nsp]
  float* sC = sB + kTT * nsp;
  float* sDt = sC + kTT * nsp;                           // [kTT][CH]
  float* sU = sDt + kTT * CH;
  float* sY = sU + kTT * CH;
  const SeqSpan sp = seq_span(a, blockIdx.y);
  const int ch = threadIdx.x / G, g = threadIdx.x % G;
  const int c0 = blockIdx.x * CH, c = c0 + ch;
  const bool c_ok = c < a.inner;
  const T* u = a.u ? reinterpret_cast<const T*>(a.u) : reinterpret_cast<const T*>(a.u_bf16);
  const T* xz = static_cast<const T*>(a.xz);
  float S[NS], A[NS];
  float* state = a.ssm_state + (static_cast<size_t>(sp.seq) * a.inner + (c_ok ? c : 0)) * a.state;
#pragma unroll
  for (int i = 0; i < NS; ++i) {
    const int n = g * NS + i;
    const bool ok = c_ok && n < a.state;
    A[i] = ok ? a.A[static_cast<size_t>(c) * a.state + n] : 0.f;
    S[i] = (ok && sp.start > 0 && sp.n > 0) ? state[n] : 0.f;
  }
  // rows in front of the sequence's start give zeros
  for (int i = threadIdx.x; i < (a.rows.Tc - sp.n) * CH; i += kScanThreads) {
    const int t = i / CH, cc = c0 + i % CH;
    if (cc < a.inner) {
      const size_t o = (static_cast<size_t>(blockIdx.y) * a.rows.Tc + t) * a.ld_u + cc;
      if (a.out) a.out[o] = 0.f;
      if (a.out_bf16) a.out_bf16[o] = __float2bfloat16_rn(0.f);
    }
  }
  for (int t0 = 0; t0 < sp.n; t0 += kTT) {
    const int nt = min(kTT, sp.n - t0);
    __syncthreads();
    for (int i = threadIdx.x; i < nt * nsp; i += kScanThreads) {
      const int t = i / nsp, n = i % nsp;
      const float* row = a.xp + static_cast<size_t>(sp.row0 + t0 + t) * a.ld_xp + a.dt_rank;
      sB[i] = n < a.state ? row[n] : 0.f;
      sC[i] = n < a.state ? row[a.state + n] : 0.f;
    }
    for (int i = threadIdx.x; i < nt * CH; i += kScanThreads) {
      const int t = i / CH, cc = c0 + i % CH;
      const size_t o = static_cast<size_t>(sp.row0 + t0 + t) * a.ld_u + cc;
      const bool ok = cc < a.inner;
      sDt[i] = ok ? softplus(a.dt_raw[o] + a.dt_b[cc]) : 0.f;
      sU[i] = ok ? ld(u, o) : 0.f;
    }
    __syncthreads();
#pragma unroll 4
    for (int t = 0; t < nt; ++t) {
      const float dt = sDt[t * CH + ch], du = dt * sU[t * CH + ch];
      float y = 0.f;
#pragma unroll
      for (int i = 0; i < NS; ++i) {
        S[i] = fmaf(expf(dt * A[i]), S[i], du * sB[t * nsp + g * NS + i]);
        y = fmaf(S[i], sC[t * nsp + g * NS + i], y);
      }
#pragma unroll
      for (int o = G / 2; o > 0; o >>= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
      if (g == 0) sY[t * CH + ch] = y;
    }
    __syncthreads();
    for (int i = threadIdx.x; i < nt * CH; i += kScanThreads) {
      const int t = i / CH, cc = c0 + i % CH;
      if (cc >= a.inner) continue;
      const size_t m = static_cast<size_t>(sp.row0 + t0 + t), o = m * a.ld_u + cc;
      const float y = fmaf(a.D[cc], sU[i], sY[i]) * silu(ld(xz, m * a.ld_xz + a.z0 + cc));
      if (a.out) a.out[o] = y;
      if (a.out_bf16) a.out_bf16[o] = __float2bfloat16_rn(y);
    }
  }
  if (c_ok && sp.n > 0) {
#pragma unroll
    for (int i = 0; i < NS; ++i)
      if (g * NS + i < a.state) state[g * NS + i] = S[i];
  }
}

// Decode: G lanes per channel do the step-size projection, the state update and the output of one row.
template <typename T, int G>
__global__ void __launch_bounds__(256) ssm_step_kernel(const SsmArgs a) {
  extern __shared__ float st_smem[];                     // dt | B | C of the row
  pdl_wait();
  pdl_launch_dependents();
  const int m = blockIdx.y, g = threadIdx.x % G, c = blockIdx.x * (256 / G) + threadIdx.x / G;
  const SeqSpan sp = seq_span(a, m);
  const int np = a.ld_wdt + 2 * a.state;                  // the dt part padded with zeros to the weight's row length
  for (int i = threadIdx.x; i < np; i += 256) {
    const float* row = a.xp + static_cast<size_t>(m) * a.ld_xp;
    st_smem[i] = i < a.dt_rank ? row[i] : i < a.ld_wdt ? 0.f : row[a.dt_rank + i - a.ld_wdt];
  }
  __syncthreads();
  const bool ok = c < a.inner;
  const int cc = ok ? c : 0;
  float dt = 0.f;
  for (int k = g * 8; k < a.ld_wdt; k += G * 8) {
    float w8[8];
    unpack8(ld_stream16(a.w_dt + static_cast<size_t>(cc) * a.ld_wdt + k), w8);
#pragma unroll
    for (int e = 0; e < 8; ++e) dt = fmaf(w8[e], st_smem[k + e], dt);
  }
#pragma unroll
  for (int o = G / 2; o > 0; o >>= 1) dt += __shfl_xor_sync(0xffffffffu, dt, o);
  dt = softplus(dt + a.dt_b[cc]);
  const float u = a.u ? a.u[static_cast<size_t>(m) * a.ld_u + cc] : __bfloat162float(a.u_bf16[static_cast<size_t>(m) * a.ld_u + cc]);
  const float du = dt * u;
  const float* B = st_smem + a.ld_wdt;
  float* state = a.ssm_state + (static_cast<size_t>(sp.seq) * a.inner + cc) * a.state;
  float y = 0.f;
  for (int n = g; n < a.state; n += G) {
    const float old = sp.start > 0 ? state[n] : 0.f;
    const float s = fmaf(expf(dt * a.A[static_cast<size_t>(cc) * a.state + n]), old, du * B[n]);
    if (ok) state[n] = s;
    y = fmaf(s, B[a.state + n], y);
  }
#pragma unroll
  for (int o = G / 2; o > 0; o >>= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
  if (ok && g == 0) {
    const float z = ld(static_cast<const T*>(a.xz), static_cast<size_t>(m) * a.ld_xz + a.z0 + c);
    y = fmaf(a.D[c], u, y) * silu(z);
    const size_t o = static_cast<size_t>(m) * a.ld_u + c;
    if (a.out) a.out[o] = y;
    if (a.out_bf16) a.out_bf16[o] = __float2bfloat16_rn(y);
  }
}

bool ssm_ok(const SsmArgs& a) {
  return a.M > 0 && a.inner > 0 && a.state > 0 && a.state <= kSsmMaxState && a.taps >= 1 && a.nseq > 0 && a.rows.Tc > 0 &&
         a.M == a.nseq * a.rows.Tc && a.ld_u >= a.inner && (a.u != nullptr) != (a.u_bf16 != nullptr) &&
         (a.u != nullptr) == !a.xz_bf16;
}

template <typename T, int G, int NS>
cudaError_t scan(const SsmArgs& a, cudaStream_t s) {
  constexpr int CH = kScanThreads / G;
  const size_t smem = sizeof(float) * kTT * (2 * G * NS + 3 * CH);
  static DeviceOnce once;
  cudaError_t e = once.run([&] {
    return cudaFuncSetAttribute(ssm_scan_kernel<T, G, NS>, cudaFuncAttributeMaxDynamicSharedMemorySize, static_cast<int>(smem));
  });
  if (e != cudaSuccess) return e;
  ssm_scan_kernel<T, G, NS><<<dim3((a.inner + CH - 1) / CH, a.nseq), kScanThreads, smem, s>>>(a);
  return cudaGetLastError();
}

template <typename T>
cudaError_t scan_states(const SsmArgs& a, cudaStream_t s) {
  if (a.state <= 8) return scan<T, 4, 2>(a, s);
  if (a.state <= 16) return scan<T, 4, 4>(a, s);
  if (a.state <= 32) return scan<T, 8, 4>(a, s);
  if (a.state <= 64) return scan<T, 16, 4>(a, s);
  if (a.state <= 128) return scan<T, 32, 4>(a, s);
  return scan<T, 32, 8>(a, s);
}

template <typename T>
cudaError_t step_states(const SsmArgs& a, cudaStream_t s, bool pdl) {
  const size_t smem = sizeof(float) * (a.ld_wdt + 2 * static_cast<size_t>(a.state));
  if (smem > 48 * 1024) return cudaErrorInvalidValue;
  if (a.state <= 8) return launch_pdl(ssm_step_kernel<T, 8>, dim3((a.inner + 31) / 32, a.M), dim3(256), smem, s, pdl, a);
  if (a.state <= 16) return launch_pdl(ssm_step_kernel<T, 16>, dim3((a.inner + 15) / 16, a.M), dim3(256), smem, s, pdl, a);
  return launch_pdl(ssm_step_kernel<T, 32>, dim3((a.inner + 7) / 8, a.M), dim3(256), smem, s, pdl, a);
}

}  // namespace

cudaError_t launch_ssm_conv(const SsmArgs& a, cudaStream_t s, bool pdl) {
  if (!ssm_ok(a)) return cudaErrorInvalidValue;
  const int cb = (a.inner + 255) / 256;
  if (a.rows.Tc == 1)
    return a.xz_bf16 ? launch_pdl(ssm_conv_step_kernel<__nv_bfloat16>, dim3(cb, a.M), dim3(256), 0, s, pdl, a)
                     : launch_pdl(ssm_conv_step_kernel<float>, dim3(cb, a.M), dim3(256), 0, s, pdl, a);
  const dim3 grid(cb, (a.rows.Tc + kConvRows - 1) / kConvRows, a.nseq);
  cudaError_t e = a.xz_bf16 ? launch_pdl(ssm_conv_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, pdl, a)
                            : launch_pdl(ssm_conv_kernel<float>, grid, dim3(256), 0, s, pdl, a);
  if (e != cudaSuccess || a.taps == 1) return e;
  return a.xz_bf16 ? launch_pdl(ssm_conv_state_kernel<__nv_bfloat16>, dim3(cb, a.nseq), dim3(256), 0, s, pdl, a)
                   : launch_pdl(ssm_conv_state_kernel<float>, dim3(cb, a.nseq), dim3(256), 0, s, pdl, a);
}

cudaError_t launch_ssm_split(const SsmArgs& a, cudaStream_t s) {
  if (!ssm_ok(a) || !a.dtr_bf16) return cudaErrorInvalidValue;
  ssm_split_kernel<<<a.M, 64, 0, s>>>(a);
  return cudaGetLastError();
}

cudaError_t launch_ssm_scan(const SsmArgs& a, cudaStream_t s) {
  if (!ssm_ok(a) || !a.dt_raw) return cudaErrorInvalidValue;
  return a.xz_bf16 ? scan_states<__nv_bfloat16>(a, s) : scan_states<float>(a, s);
}

cudaError_t launch_ssm_step(const SsmArgs& a, cudaStream_t s, bool pdl) {
  if (!ssm_ok(a) || a.rows.Tc != 1) return cudaErrorInvalidValue;
  return a.xz_bf16 ? step_states<__nv_bfloat16>(a, s, pdl) : step_states<float>(a, s, pdl);
}

}  // namespace mtj
