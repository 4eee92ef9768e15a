// Row kernels of layer-stack models (residual + norms) and the repacking of their weights.
#include <math.h>

#include <algorithm>

#include "mtj_common.cuh"
#include "mtj_stack_kernels.h"

namespace mtj {
namespace {

constexpr int kRnThreads = 256;

__device__ __forceinline__ float rn_block_sum(float v, float* red) {
  v = warp_sum(v);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  if (lane == 0) red[warp] = v;
  __syncthreads();
  float t = 0.f;
#pragma unroll
  for (int i = 0; i < kRnThreads / 32; ++i) t += red[i];
  __syncthreads();
  return t;
}

__device__ __forceinline__ float dot4(const float4& a) { return a.x * a.x + a.y * a.y + a.z * a.z + a.w * a.w; }
__device__ __forceinline__ uint2 pack4(const float4& v) {
  return make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
}

// Norm after the sublayer, residual add and the norm before the next sublayer, one pass over the row.  Every thread
// touches only the columns it owns, so the row lives in shared memory without barriers between the passes.
__global__ void __launch_bounds__(kRnThreads) residual_norm_kernel(const ResidualNormArgs a) {
  extern __shared__ float4 rn_row[];                   // x, then (with y) y
  __shared__ float red[kRnThreads / 32];
  pdl_wait();
  pdl_launch_dependents();
  const int n4 = a.ld >> 2;
  const size_t m = blockIdx.x;
  float4* xrow = reinterpret_cast<float4*>(a.x + m * a.ld);
  float ss = 0.f;
  if (a.y) {
    float4* yrow = rn_row + n4;
    float ys = 0.f;
    for (int i = threadIdx.x; i < n4; i += kRnThreads) {
      float4 v = reinterpret_cast<const float4*>(a.y + m * a.ld)[i];
      for (int p = 1; p < a.planes; ++p) {
        const float4 w = reinterpret_cast<const float4*>(a.y + (static_cast<size_t>(p) * a.M + m) * a.ld)[i];
        v.x += w.x; v.y += w.y; v.z += w.z; v.w += w.w;
      }
      yrow[i] = v;
      rn_row[i] = xrow[i];
      ys += dot4(v);
    }
    const float rs = a.mult / sqrtf(rn_block_sum(ys, red) / static_cast<float>(a.d) + a.eps);
    for (int i = threadIdx.x; i < n4; i += kRnThreads) {
      const float4 y = yrow[i], w = reinterpret_cast<const float4*>(a.w_post)[i];
      float4 x = rn_row[i];
      x.x = fmaf(y.x * rs, w.x, x.x);
      x.y = fmaf(y.y * rs, w.y, x.y);
      x.z = fmaf(y.z * rs, w.z, x.z);
      x.w = fmaf(y.w * rs, w.w, x.w);
      rn_row[i] = x;
      xrow[i] = x;
      ss += dot4(x);
    }
  } else {
    for (int i = threadIdx.x; i < n4; i += kRnThreads) {
      const float4 x = xrow[i];
      rn_row[i] = x;
      ss += dot4(x);
    }
  }
  const float rs = 1.0f / sqrtf(rn_block_sum(ss, red) / static_cast<float>(a.d) + a.eps);
  if (a.stats && threadIdx.x == 0) {
    a.stats[2 * m] = 0.f;
    a.stats[2 * m + 1] = rs;
  }
  if (a.xn) {
    uint2* o = reinterpret_cast<uint2*>(a.xn + m * a.ld);
    for (int i = threadIdx.x; i < n4; i += kRnThreads) {
      const float4 x = rn_row[i], w = reinterpret_cast<const float4*>(a.w_next)[i];
      o[i] = pack4(make_float4(x.x * rs * w.x, x.y * rs * w.y, x.z * rs * w.z, x.w * rs * w.w));
    }
  }
  if (a.cat_f32 || a.cat_bf16) {
    const float4* x0 = reinterpret_cast<const float4*>(a.x0 + m * a.ld);
    for (int i = threadIdx.x; i < n4; i += kRnThreads) {
      const float4 x = rn_row[i], e = x0[i];
      if (a.cat_f32) {
        float4* o = reinterpret_cast<float4*>(a.cat_f32 + m * 2 * a.ld);
        o[i] = x;
        o[n4 + i] = e;
      }
      if (a.cat_bf16) {
        uint2* o = reinterpret_cast<uint2*>(a.cat_bf16 + m * 2 * a.ld);
        o[i] = pack4(x);
        o[n4 + i] = pack4(e);
      }
    }
  }
}

// The same for layers with a layer norm behind the residual sum.
__global__ void __launch_bounds__(kRnThreads) residual_layernorm_kernel(const ResidualLayerNormArgs a) {
  extern __shared__ float4 rn_row[];
  __shared__ float red[kRnThreads / 32];
  pdl_wait();
  pdl_launch_dependents();
  const int n4 = a.ld >> 2;
  const size_t m = blockIdx.x;
  float4* xrow = reinterpret_cast<float4*>(a.x + m * a.ld);
  const float inv_n = 1.0f / static_cast<float>(a.d);
  auto norm = [&](float sum, float* mu, float* rs) {
    *mu = rn_block_sum(sum, red) * inv_n;
    float v = 0.f;
    for (int i = threadIdx.x; i < n4; i += kRnThreads) {
      const float4 z = rn_row[i];
      const int left = a.d - 4 * i;                       // columns that exist
      v += dot4(make_float4(left > 0 ? z.x - *mu : 0.f, left > 1 ? z.y - *mu : 0.f, left > 2 ? z.z - *mu : 0.f, left > 3 ? z.w - *mu : 0.f));
    }
    *rs = 1.0f / sqrtf(rn_block_sum(v, red) * inv_n + a.eps);
  };
  auto scaled = [&](int i, float mu, float rs, const float* w, const float* b) {
    const float4 z = rn_row[i], w4 = reinterpret_cast<const float4*>(w)[i], b4 = reinterpret_cast<const float4*>(b)[i];
    return make_float4(fmaf((z.x - mu) * rs, w4.x, b4.x), fmaf((z.y - mu) * rs, w4.y, b4.y), fmaf((z.z - mu) * rs, w4.z, b4.z),
                       fmaf((z.w - mu) * rs, w4.w, b4.w));
  };
  float sum = 0.f, mu, rs;
  for (int i = threadIdx.x; i < n4; i += kRnThreads) {
    float4 x = xrow[i];
    if (a.y) {
      const float4 y = reinterpret_cast<const float4*>(a.y + m * a.ld)[i];
      x = make_float4(fmaf(a.alpha, x.x, y.x), fmaf(a.alpha, x.y, y.y), fmaf(a.alpha, x.z, y.z), fmaf(a.alpha, x.w, y.w));
    }
    rn_row[i] = x;
    sum += (x.x + x.y) + (x.z + x.w);
  }
  if (a.y) {
    norm(sum, &mu, &rs);
    sum = 0.f;
    for (int i = threadIdx.x; i < n4; i += kRnThreads) {
      const float4 x = scaled(i, mu, rs, a.w, a.b);       // w and b are zero in the padding
      rn_row[i] = x;
      xrow[i] = x;
      sum += (x.x + x.y) + (x.z + x.w);
      if (a.xn && !a.w_next) reinterpret_cast<uint2*>(a.xn + m * a.ld)[i] = pack4(x);
    }
  } else if (a.xn && !a.w_next) {
    for (int i = threadIdx.x; i < n4; i += kRnThreads) reinterpret_cast<uint2*>(a.xn + m * a.ld)[i] = pack4(rn_row[i]);
  }
  if (!a.w_next && !a.stats) return;
  norm(sum, &mu, &rs);
  if (a.stats && threadIdx.x == 0) {
    a.stats[2 * m] = mu;
    a.stats[2 * m + 1] = rs;
  }
  if (a.xn && a.w_next)
    for (int i = threadIdx.x; i < n4; i += kRnThreads)
      reinterpret_cast<uint2*>(a.xn + m * a.ld)[i] = pack4(scaled(i, mu, rs, a.w_next, a.b_next));
}

__global__ void gather_rows_bf16_kernel(const __nv_bfloat16* __restrict__ src, int ld, const int32_t* __restrict__ rows,
                                        __nv_bfloat16* __restrict__ dst) {
  const uint4* s = reinterpret_cast<const uint4*>(src + static_cast<size_t>(rows[blockIdx.x]) * ld);
  uint4* d = reinterpret_cast<uint4*>(dst + static_cast<size_t>(blockIdx.x) * ld);
  for (int i = threadIdx.x; i < ld / 8; i += blockDim.x) d[i] = s[i];
}

__global__ void copy_rows_kernel(const float4* __restrict__ src, float4* __restrict__ dst, int64_t n4) {
  pdl_wait();
  pdl_launch_dependents();
  const int64_t step = static_cast<int64_t>(gridDim.x) * blockDim.x;
  for (int64_t i = static_cast<int64_t>(blockIdx.x) * blockDim.x + threadIdx.x; i < n4; i += step) dst[i] = src[i];
}

__device__ __forceinline__ float load_any(const void* p, int is_bf16, int64_t i) {
  return is_bf16 ? __bfloat162float(static_cast<const __nv_bfloat16*>(p)[i]) : static_cast<const float*>(p)[i];
}

__global__ void pack_rows_kernel(const void* src, int src_is_bf16, int N, int K, __nv_bfloat16* dst, int ld, int r0,
                                 int gin, int gout, int csplit, int cshift) {
  const int64_t total = static_cast<int64_t>(N) * K, step = static_cast<int64_t>(gridDim.x) * blockDim.x;
  for (int64_t i = static_cast<int64_t>(blockIdx.x) * blockDim.x + threadIdx.x; i < total; i += step) {
    const int n = static_cast<int>(i / K), k = static_cast<int>(i % K);
    const size_t row = static_cast<size_t>(r0) + static_cast<size_t>(n / gin) * gout + n % gin;
    dst[row * ld + (k < csplit ? k : k + cshift)] = __float2bfloat16_rn(load_any(src, src_is_bf16, i));
  }
}

__global__ void neg_exp_kernel(const void* src, int src_is_bf16, int64_t n, float* dst) {
  const int64_t step = static_cast<int64_t>(gridDim.x) * blockDim.x;
  for (int64_t i = static_cast<int64_t>(blockIdx.x) * blockDim.x + threadIdx.x; i < n; i += step)
    dst[i] = -expf(load_any(src, src_is_bf16, i));
}

__global__ void transpose_f32_kernel(const void* src, int src_is_bf16, int N, int K, float* dst, int ld) {
  const int64_t total = static_cast<int64_t>(N) * K, step = static_cast<int64_t>(gridDim.x) * blockDim.x;
  for (int64_t i = static_cast<int64_t>(blockIdx.x) * blockDim.x + threadIdx.x; i < total; i += step)
    dst[static_cast<size_t>(i % K) * ld + i / K] = load_any(src, src_is_bf16, i);
}

int load_grid(int64_t n) { return static_cast<int>(std::min<int64_t>((n + 255) / 256, 4096)); }

}  // namespace

cudaError_t launch_residual_norm(const ResidualNormArgs& a, cudaStream_t s, bool pdl) {
  if (a.M <= 0 || a.d <= 0 || a.ld < a.d || (a.ld & 3)) return cudaErrorInvalidValue;
  const size_t smem = static_cast<size_t>(a.ld) * sizeof(float) * (a.y ? 2 : 1);
  if (smem > 200 * 1024) return cudaErrorInvalidValue;
  static DeviceOnce once;
  cudaError_t e = once.run([&] {
    return cudaFuncSetAttribute(residual_norm_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
  });
  if (e != cudaSuccess) return e;
  return launch_pdl(residual_norm_kernel, dim3(a.M), dim3(kRnThreads), smem, s, pdl, a);
}

cudaError_t launch_residual_layernorm(const ResidualLayerNormArgs& a, cudaStream_t s, bool pdl) {
  if (a.M <= 0 || a.d <= 0 || a.ld < a.d || (a.ld & 3) || (a.y && (!a.w || !a.b)) || (a.w_next && !a.b_next)) return cudaErrorInvalidValue;
  const size_t smem = static_cast<size_t>(a.ld) * sizeof(float);
  if (smem > 200 * 1024) return cudaErrorInvalidValue;
  static DeviceOnce once;
  cudaError_t e = once.run([&] {
    return cudaFuncSetAttribute(residual_layernorm_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024);
  });
  if (e != cudaSuccess) return e;
  return launch_pdl(residual_layernorm_kernel, dim3(a.M), dim3(kRnThreads), smem, s, pdl, a);
}

cudaError_t launch_gather_rows_bf16(const __nv_bfloat16* src, int ld, const int32_t* rows, int n, __nv_bfloat16* dst,
                                    cudaStream_t s) {
  if (n <= 0 || (ld & 7)) return cudaErrorInvalidValue;
  gather_rows_bf16_kernel<<<n, 128, 0, s>>>(src, ld, rows, dst);
  return cudaGetLastError();
}

cudaError_t launch_copy_rows(const float* src, float* dst, int64_t n, cudaStream_t s, bool pdl) {
  if (n <= 0 || (n & 3)) return cudaErrorInvalidValue;
  return launch_pdl(copy_rows_kernel, dim3(static_cast<int>(std::min<int64_t>((n / 4 + 255) / 256, 1184))), dim3(256), 0, s, pdl,
                    reinterpret_cast<const float4*>(src), reinterpret_cast<float4*>(dst), n / 4);
}

cudaError_t launch_pack_rows(const void* src, int src_is_bf16, int N, int K, __nv_bfloat16* dst, int ld, int r0, int gin,
                             int gout, int csplit, int cshift, cudaStream_t s) {
  pack_rows_kernel<<<load_grid(static_cast<int64_t>(N) * K), 256, 0, s>>>(src, src_is_bf16, N, K, dst, ld, r0, gin, gout,
                                                                          csplit, cshift);
  return cudaGetLastError();
}

cudaError_t launch_neg_exp(const void* src, int src_is_bf16, int64_t n, float* dst, cudaStream_t s) {
  neg_exp_kernel<<<load_grid(n), 256, 0, s>>>(src, src_is_bf16, n, dst);
  return cudaGetLastError();
}

cudaError_t launch_transpose_f32(const void* src, int src_is_bf16, int N, int K, float* dst, int ld, cudaStream_t s) {
  transpose_f32_kernel<<<load_grid(static_cast<int64_t>(N) * K), 256, 0, s>>>(src, src_is_bf16, N, K, dst, ld);
  return cudaGetLastError();
}

}  // namespace mtj
