// Tensor-core GEMM: host side (tensor maps, launch selection) and the two small kernels around it.  The GEMM kernels
// are in mtj_gemm_tc.cuh, their instances in mtj_gemm_tc_gptj.cu and mtj_gemm_tc_stack.cu.
#include "mtj_gemm_tc.cuh"

namespace mtj {
namespace {

// LayerNorm of fp32 rows into bf16 (the GEMM's activation operand), layers.py:17-36.
__global__ void __launch_bounds__(256) ln_rows_kernel(const float* __restrict__ x, const float* __restrict__ scale,
                                                      const float* __restrict__ offset,
                                                      __nv_bfloat16* __restrict__ out, __nv_bfloat16* out_lo, int d) {
  __shared__ float red[8];
  pdl_wait();
  pdl_launch_dependents();
  const float* xr = x + static_cast<size_t>(blockIdx.x) * d;
  __nv_bfloat16* o = out + static_cast<size_t>(blockIdx.x) * d;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  auto block_sum = [&](float v) {
    v = warp_sum(v);
    if (lane == 0) red[warp] = v;
    __syncthreads();
    float t = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) t += red[i];
    __syncthreads();
    return t;
  };
  float s = 0.f;
  for (int i = threadIdx.x; i < d; i += 256) s += xr[i];
  const float mu = block_sum(s) / static_cast<float>(d);
  float v = 0.f;
  for (int i = threadIdx.x; i < d; i += 256) {
    const float t = xr[i] - mu;
    v = fmaf(t, t, v);
  }
  const float rstd = 1.0f / sqrtf(block_sum(v) / static_cast<float>(d) + 1e-5f);
  for (int i = threadIdx.x; i < d; i += 256) {
    const float y = fmaf(scale[i] * rstd, xr[i] - mu, offset[i]);
    const __nv_bfloat16 hi = __float2bfloat16_rn(y);
    o[i] = hi;
    if (out_lo) out_lo[static_cast<size_t>(blockIdx.x) * d + i] = __float2bfloat16_rn(y - __bfloat162float(hi));
  }
}

PFN_cuTensorMapEncodeTiled_v12000 encode_fn() {
  static PFN_cuTensorMapEncodeTiled_v12000 fn = nullptr;
  if (fn) return fn;
  void* p = nullptr;
  cudaDriverEntryPointQueryResult q;
  if (cudaGetDriverEntryPoint("cuTensorMapEncodeTiled", &p, cudaEnableDefault, &q) != cudaSuccess ||
      q != cudaDriverEntryPointSuccess)
    return nullptr;
  fn = reinterpret_cast<PFN_cuTensorMapEncodeTiled_v12000>(p);
  return fn;
}

}  // namespace

int gemm_tc_token_tile() { return 128; }
// Batched decode streams each weight tile once, and a block keeps only its TMA ring in flight: with fewer tiles
// than the GPU holds blocks (two per SM), K is split over a cluster of 2 or 4 blocks per tile so that the
// bytes in flight -- and with them the HBM rate -- do not fall with the tile count (tensor-parallel slices).
int gemm_tc_decode_cluster_k(int weight_rows, int M, int K) {
  if (M > 64) return 1;
  const int tiles = (weight_rows + kBM - 1) / kBM;      // one token tile
  int ck = 1;
  while (ck < 4 && tiles * ck * 2 <= 296 && K / kBK >= ck * 2 * 2) ck *= 2;
  return ck;
}

int gemm_tc_token_tile_for(int M) { return M <= 32 ? 32 : (M <= 64 ? 64 : 128); }
int gemm_tc_wide_token_tile() { return kPBN / 2; }     // rows of the activation box: a tile takes two of them

cudaError_t launch_gemm_tc_wide(GemvEpilogue epi, const void* map_w, const void* map_x, const GemmTcArgs& a,
                                cudaStream_t s) {
  if (a.M <= 0 || a.N <= 0 || a.K <= 0 || a.partial) return cudaErrorInvalidValue;
  const CUtensorMap& mw = *static_cast<const CUtensorMap*>(map_w);
  const CUtensorMap& mx = *static_cast<const CUtensorMap*>(map_x);
  if (epi == kEpiPlain || epi == kEpiSwiGLU) return launch_gemm_tc_stack(epi, true, mw, mx, a, s, false);
  if (epi == kEpiRelu2 || epi == kEpiSoftcap) return launch_gemm_tc_stack_post(epi, true, mw, mx, a, s, false);
  return launch_gemm_tc_gptj(epi, true, mw, mx, nullptr, a, s, false);
}

cudaError_t make_tensor_map_bf16(void* map_out, const void* base, int64_t rows, int64_t K, int box_rows, int64_t ld) {
  if (ld <= 0) ld = K;
  PFN_cuTensorMapEncodeTiled_v12000 fn = encode_fn();
  if (!fn) return cudaErrorNotSupported;
  if ((reinterpret_cast<uintptr_t>(base) & 15) || (ld * 2) % 16 || ld < K || box_rows > 256) return cudaErrorInvalidValue;
  cuuint64_t dims[2] = {static_cast<cuuint64_t>(K), static_cast<cuuint64_t>(rows)};
  cuuint64_t strides[1] = {static_cast<cuuint64_t>(ld) * 2};
  cuuint32_t box[2] = {static_cast<cuuint32_t>(kBK), static_cast<cuuint32_t>(box_rows)};
  cuuint32_t estr[2] = {1, 1};
  CUresult r = fn(static_cast<CUtensorMap*>(map_out), CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(base),
                  dims, strides, box, estr, CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B,
                  CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
  return r == CUDA_SUCCESS ? cudaSuccess : cudaErrorInvalidValue;
}

cudaError_t launch_gemm_tc(GemvEpilogue epi, const void* map_w, const void* map_x, const GemmTcArgs& a,
                           cudaStream_t s, bool pdl, const void* map_x_lo) {
  if (a.M <= 0 || a.N <= 0 || a.K <= 0) return cudaErrorInvalidValue;
  const CUtensorMap& mw = *static_cast<const CUtensorMap*>(map_w);
  const CUtensorMap& mx = *static_cast<const CUtensorMap*>(map_x);
  if (epi == kEpiPlain || epi == kEpiSwiGLU)
    return map_x_lo ? cudaErrorInvalidValue : launch_gemm_tc_stack(epi, false, mw, mx, a, s, pdl);
  if (epi == kEpiRelu2 || epi == kEpiSoftcap)
    return map_x_lo ? cudaErrorInvalidValue : launch_gemm_tc_stack_post(epi, false, mw, mx, a, s, pdl);
  return launch_gemm_tc_gptj(epi, false, mw, mx, static_cast<const CUtensorMap*>(map_x_lo), a, s, pdl);
}

namespace {
// out[m, n] = sum_z partial[z, m, n] + bias[n] (+ residual[m, n]); fixed summation order
__global__ void splitk_reduce_kernel(const float* __restrict__ partial, int ksplit, int M, int N,
                                     const float* __restrict__ bias, const float* residual, float* out, int ld_out,
                                     const uint32_t* slot_sel, size_t slot_stride) {
  const size_t total = static_cast<size_t>(M) * N;
  pdl_wait();                      // the partial sums come from the predecessor kernel
  pdl_launch_dependents();
  if (slot_sel) out += static_cast<size_t>(*slot_sel & 1u) * slot_stride;
  for (size_t i = static_cast<size_t>(blockIdx.x) * blockDim.x + threadIdx.x; i < total;
       i += static_cast<size_t>(gridDim.x) * blockDim.x) {
    const int n = static_cast<int>(i % N);
    const size_t m = i / N;
    float acc = 0.f;
    for (int z = 0; z < ksplit; ++z) acc += partial[static_cast<size_t>(z) * total + i];
    if (bias) acc += bias[n];
    if (residual) acc += residual[i];
    out[m * ld_out + n] = acc;
  }
}
}  // namespace

cudaError_t launch_splitk_reduce(const float* partial, int ksplit, int M, int N, const float* bias,
                                 const float* residual, float* out, int ld_out, const uint32_t* slot_sel,
                                 size_t slot_stride, cudaStream_t s, bool pdl) {
  const size_t total = static_cast<size_t>(M) * N;
  const int grid = static_cast<int>(std::min<size_t>((total + 255) / 256, 148 * 8));
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(grid);
  cfg.blockDim = dim3(256);
  cfg.stream = s;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = pdl ? 1 : 0;
  return cudaLaunchKernelEx(&cfg, splitk_reduce_kernel, partial, ksplit, M, N, bias, residual, out, ld_out, slot_sel,
                            slot_stride);
}

cudaError_t launch_ln_rows(const float* x, const float* scale, const float* offset, __nv_bfloat16* out, int rows,
                           int d, cudaStream_t s, bool pdl, __nv_bfloat16* out_lo) {
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(rows);
  cfg.blockDim = dim3(256);
  cfg.stream = s;
  cudaLaunchAttribute attr[1];
  attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
  attr[0].val.programmaticStreamSerializationAllowed = 1;
  cfg.attrs = attr;
  cfg.numAttrs = pdl ? 1 : 0;
  return cudaLaunchKernelEx(&cfg, ln_rows_kernel, x, scale, offset, out, out_lo, d);
}

}  // namespace mtj
