// Device helpers shared by the matrix-state kernels.
#pragma once
#include <math.h>

#include "mtj_common.cuh"
#include "mtj_stack_kernels.h"

namespace mtj {

constexpr float kUnitEps = 1e-6f;    // under the root of the unit norms

__device__ __forceinline__ float ms_ld(const float* p, size_t i) { return p[i]; }
__device__ __forceinline__ float ms_ld(const __nv_bfloat16* p, size_t i) { return __bfloat162float(p[i]); }

// Elementwise functions of a run with T operands: the accurate ones for fp32 runs; serving runs, whose inputs carry bf16
// rounding, take the fast fp32 intrinsics (log(1 + e) by its series where 1 + e would round e away).
template <typename T>
struct MsFn;
template <>
struct MsFn<float> {
  __device__ static __forceinline__ float exp(float x) { return expf(x); }
  __device__ static __forceinline__ float sigmoid(float z) { return 1.0f / (1.0f + expf(-z)); }
  __device__ static __forceinline__ float silu(float z) { return z / (1.0f + expf(-z)); }
  __device__ static __forceinline__ float softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
};
template <>
struct MsFn<__nv_bfloat16> {
  __device__ static __forceinline__ float exp(float x) { return __expf(x); }
  __device__ static __forceinline__ float sigmoid(float z) { return __fdividef(1.0f, 1.0f + __expf(-z)); }
  __device__ static __forceinline__ float silu(float z) { return __fdividef(z, 1.0f + __expf(-z)); }
  __device__ static __forceinline__ float softplus(float z) {
    const float e = __expf(-fabsf(z));
    return fmaxf(z, 0.f) + (e < 0.01f ? e * (1.0f - e * (0.5f - e * 0.33333333f)) : __logf(1.0f + e));
  }
};

struct MsSpan {
  int seq, start, n, row0;           // slot, own position of the first real row, real rows, its row index
};
// the real rows of sequence i of the call
__device__ __forceinline__ MsSpan ms_span(const MatrixStateArgs& a, int i) {
  MsSpan s;
  s.seq = a.rows.b0 + i;
  const int p0 = (a.rows.pos0_dev ? *a.rows.pos0_dev : a.rows.pos0_host) - a.pad[s.seq];
  const int skip = min(max(-p0, 0), a.rows.Tc);
  s.start = p0 + skip;
  s.n = a.rows.Tc - skip;
  s.row0 = i * a.rows.Tc + skip;
  return s;
}

inline bool matrix_state_ok(const MatrixStateArgs& a) {
  return a.M > 0 && a.heads > 0 && a.key_heads > 0 && a.heads % a.key_heads == 0 && a.dim > 0 && a.dim <= kMatrixMaxDim &&
         a.vdim > 0 && a.nseq > 0 && a.rows.Tc > 0 && a.M == a.nseq * a.rows.Tc && a.u && a.decay && a.decay_b && a.A && a.state &&
         a.out && (a.delta ? a.beta != nullptr : a.D != nullptr);
}

}  // namespace mtj
