// Latent attention: the keys and values of all heads are linear maps of one normalised latent per token, plus one
// rotated key part shared by the heads; the cache holds the latent and that part, paged and ring-addressed by the
// position inside the sequence (window layers: pages fall out of the window and are used again).
//
//   absorbed form (decode, short portions, 32-bit runs), CUDA cores:
//     latent_absorb_kernel  latent norm + key rotation + cache write; q' = W_uk^T q per head, rotated query part
//     latent_attn_kernel    one block = (row, 8 heads, key range): 32-key tiles of the cache in shared memory, one warp
//                           per head for the scores and the online softmax, then every thread accumulates its latent
//                           columns for all 8 heads -- a cached byte is read once per 8 heads
//     latent_out_kernel     merges the key ranges, W_uv per head
//   expanded form (prefill): latent_pack_kernel / latent_history_kernel lay out queries and latents for the
//     up-projection GEMM and the tensor-core attention (mtj_attn_tc_latent.cu).
// Scores, softmax and norms are fp32 throughout.
#include <math.h>

#include <algorithm>

#include "mtj_common.cuh"
#include "mtj_stack_kernels.h"

namespace mtj {
namespace {

constexpr int kThreads = 256;
constexpr int kHG = 8;            // heads per block (= warps)
constexpr int kTK = 32;           // keys per tile (= lanes)

__device__ __forceinline__ float la_block_sum(float v, float* red) {
  v = warp_sum(v);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  if (lane == 0) red[warp] = v;
  __syncthreads();
  float t = 0.f;
#pragma unroll
  for (int i = 0; i < kThreads / 32; ++i) t += red[i];
  __syncthreads();
  return t;
}

__device__ __forceinline__ void st(float* p, float v) { *p = v; }
__device__ __forceinline__ void st(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }

// position of row m inside its sequence (negative: left padding)
__device__ __forceinline__ int own_pos(const RowMap& r, const int32_t* pad, int m, int* seq) {
  *seq = r.b0 + m / r.Tc;
  return (r.pos0_dev ? *r.pos0_dev : r.pos0_host) + m % r.Tc - pad[*seq];
}
__device__ __forceinline__ size_t cache_row(const LatentCache& c, int seq, int p) {
  const int page = c.page_table[static_cast<size_t>(seq) * c.ring_pages + (p / kPageTokens) % c.ring_pages];
  return (static_cast<size_t>(page) * kPageTokens + p % kPageTokens) * c.row_ld;
}
// element j of a rotated vector: (u, v) pairs are neighbours
__device__ __forceinline__ float rotated(const float* x, int j, const float2* sc) {
  const float2 t = sc[j >> 1];
  return (j & 1) ? x[j] * t.y + x[j - 1] * t.x : x[j] * t.y - x[j + 1] * t.x;
}

template <typename T, int RT>
__global__ void __launch_bounds__(kThreads) latent_absorb_kernel(const LatentArgs a) {
  extern __shared__ float ab_smem[];
  __shared__ float red[kThreads / 32];
  pdl_wait();
  pdl_launch_dependents();
  const int m0 = blockIdx.x * RT, nr = min(RT, a.M - m0);
  if (blockIdx.y == a.heads) {
    for (int r = 0; r < nr; ++r) {
      int seq;
      const int p = own_pos(a.rows, a.pad, m0 + r, &seq);
      const float* c = a.p1 + static_cast<size_t>(m0 + r) * a.ld_p1 + a.heads * (a.dim + a.rot);
      float ss = 0.f;
      for (int i = threadIdx.x; i < a.rank; i += kThreads) ss = fmaf(c[i], c[i], ss);
      const float rs = 1.0f / sqrtf(la_block_sum(ss, red) / static_cast<float>(a.rank) + a.eps);
      if (p < 0) continue;
      T* row = static_cast<T*>(a.cache.pool) + cache_row(a.cache, seq, p);
      for (int i = threadIdx.x; i < a.rank; i += kThreads) st(row + i, c[i] * rs * a.kv_norm[i]);
      const float2* sc = a.sincos + static_cast<size_t>(p) * (a.rot >> 1);
      for (int j = threadIdx.x; j < a.rot; j += kThreads) st(row + a.cache.kv_ld + j, rotated(c + a.rank, j, sc));
    }
    return;
  }
  const int h = blockIdx.y, hd = a.dim + a.rot;
  float* qs = ab_smem;                                  // [RT][dim]
  float* part = ab_smem + RT * a.dim;                   // [dsplit][RT][kv_ld]
  for (int r = 0; r < RT; ++r) {
    const int m = m0 + min(r, nr - 1);
    const float* q = a.p1 + static_cast<size_t>(m) * a.ld_p1 + h * hd;
    for (int j = threadIdx.x; j < a.dim; j += kThreads) qs[r * a.dim + j] = q[j] * a.scale;
    if (r < nr) {
      int seq;
      const int p = max(own_pos(a.rows, a.pad, m, &seq), 0);
      const float2* sc = a.sincos + static_cast<size_t>(p) * (a.rot >> 1);
      float* o = a.q_abs + (static_cast<size_t>(m) * a.heads + h) * a.cache.row_ld + a.cache.kv_ld;
      for (int j = threadIdx.x; j < a.cache.row_ld - a.cache.kv_ld; j += kThreads)
        o[j] = j < a.rot ? rotated(q + a.dim, j, sc) * a.scale : 0.f;
    }
  }
  __syncthreads();
  // a thread owns 8 latent columns and every dsplit-th query dimension
  const int groups = a.cache.kv_ld >> 3, dsplit = kThreads / groups;
  const int g = threadIdx.x % groups, ds = threadIdx.x / groups;
  if (ds < dsplit) {
    float acc[RT][8] = {};
    const __nv_bfloat16* w = a.w_uk + static_cast<size_t>(h) * a.dim * a.cache.kv_ld + g * 8;
#pragma unroll 4
    for (int j = ds; j < a.dim; j += dsplit) {
      float w8[8];
      unpack8(ld_stream16(w + static_cast<size_t>(j) * a.cache.kv_ld), w8);
#pragma unroll
      for (int r = 0; r < RT; ++r) {
        const float q = qs[r * a.dim + j];
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[r][e] = fmaf(w8[e], q, acc[r][e]);
      }
    }
#pragma unroll
    for (int r = 0; r < RT; ++r)
#pragma unroll
      for (int e = 0; e < 8; ++e) part[(ds * RT + r) * a.cache.kv_ld + g * 8 + e] = acc[r][e];
  }
  __syncthreads();
  for (int i = threadIdx.x; i < nr * a.cache.kv_ld; i += kThreads) {
    const int r = i / a.cache.kv_ld, k = i % a.cache.kv_ld;
    float v = 0.f;
    for (int d = 0; d < dsplit; ++d) v += part[(d * RT + r) * a.cache.kv_ld + k];
    a.q_abs[(static_cast<size_t>(m0 + r) * a.heads + h) * a.cache.row_ld + k] = v;
  }
}

template <typename T>
struct Vec8;                       // eight cached elements
template <>
struct Vec8<__nv_bfloat16> {
  static constexpr int kPad = 8;   // row padding of the tile in shared memory: 16-byte reads without bank conflicts
  __device__ static __forceinline__ void get(const __nv_bfloat16* p, float* f) { unpack8(*reinterpret_cast<const uint4*>(p), f); }
  __device__ static __forceinline__ float2 pair(const __nv_bfloat16* p) {
    const uint32_t w = *reinterpret_cast<const uint32_t*>(p);
    return make_float2(bf16_lo(w), bf16_hi(w));
  }
};
template <>
struct Vec8<float> {
  static constexpr int kPad = 4;
  __device__ static __forceinline__ void get(const float* p, float* f) {
    const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
  }
  __device__ static __forceinline__ float2 pair(const float* p) { return *reinterpret_cast<const float2*>(p); }
};

template <typename T, int NC>
__global__ void __launch_bounds__(kThreads) latent_attn_kernel(const LatentArgs a) {
  extern __shared__ __align__(16) unsigned char la_smem[];
  __shared__ float s_corr[kHG];
  __shared__ __align__(16) float s_p[kTK][kHG];
  pdl_wait();
  pdl_launch_dependents();
  const int m = blockIdx.z, h0 = blockIdx.y * kHG, split = blockIdx.x;
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int ld = a.cache.row_ld, kv_ld = a.cache.kv_ld, tld = ld + Vec8<T>::kPad;
  float* qs = reinterpret_cast<float*>(la_smem);                    // [kHG][ld]
  T* cs = reinterpret_cast<T*>(la_smem + sizeof(float) * kHG * ld);  // [kTK][tld]
  int seq;
  const int p = own_pos(a.rows, a.pad, m, &seq);
  const int lo = max(0, p - a.window + 1), n = p - lo + 1;            // n <= 0: a padding row
  const int per = (((max(n, 0) + a.splits - 1) / a.splits) + kTK - 1) / kTK * kTK;
  const int k0 = lo + split * per, k1 = min(k0 + per, p + 1);

  for (int i = threadIdx.x; i < kHG * (ld >> 2); i += kThreads) {
    const int h = i / (ld >> 2), c = i % (ld >> 2);
    reinterpret_cast<float4*>(qs)[i] =
        h0 + h < a.heads ? reinterpret_cast<const float4*>(a.q_abs + (static_cast<size_t>(m) * a.heads + h0 + h) * ld)[c]
                         : make_float4(0.f, 0.f, 0.f, 0.f);
  }
  float acc[NC][kHG][2] = {};
  float mx = -INFINITY, l = 0.f;                                    // of head h0 + warp, the same in every lane
  constexpr int kVec = 16 / static_cast<int>(sizeof(T));
  const int nv = ld / kVec;
  for (int kt = k0; kt < k1; kt += kTK) {
    __syncthreads();                                                // the tile and the weights of the last round are read
    for (int i = threadIdx.x; i < kTK * nv; i += kThreads) {
      const int key = i / nv, c = i % nv;
      uint4 v = make_uint4(0u, 0u, 0u, 0u);
      if (kt + key < k1)
        v = *reinterpret_cast<const uint4*>(static_cast<const T*>(a.cache.pool) + cache_row(a.cache, seq, kt + key) + c * kVec);
      *reinterpret_cast<uint4*>(cs + key * tld + c * kVec) = v;
    }
    __syncthreads();
    float s = 0.f, s2 = 0.f;
    {
      const float* q = qs + warp * ld;
      const T* c = cs + lane * tld;
      for (int i = 0; i < ld; i += 8) {
        float f[8];
        Vec8<T>::get(c + i, f);
        const float4 qa = *reinterpret_cast<const float4*>(q + i), qb = *reinterpret_cast<const float4*>(q + i + 4);
        s = fmaf(f[0], qa.x, s); s2 = fmaf(f[1], qa.y, s2); s = fmaf(f[2], qa.z, s); s2 = fmaf(f[3], qa.w, s2);
        s = fmaf(f[4], qb.x, s); s2 = fmaf(f[5], qb.y, s2); s = fmaf(f[6], qb.z, s); s2 = fmaf(f[7], qb.w, s2);
      }
    }
    s = kt + lane < k1 ? s + s2 : -INFINITY;
    const float m_new = fmaxf(mx, warp_max(s));                     // the tile holds at least one key
    const float corr = expf(mx - m_new), w = expf(s - m_new);
    l = l * corr + warp_sum(w);
    mx = m_new;
    s_p[lane][warp] = w;
    if (lane == 0) s_corr[warp] = corr;
    __syncthreads();
#pragma unroll
    for (int c = 0; c < NC; ++c) {
      const int col = c * 2 * kThreads + 2 * threadIdx.x;
      if (col < kv_ld) {
#pragma unroll
        for (int h = 0; h < kHG; ++h) {
          acc[c][h][0] *= s_corr[h];
          acc[c][h][1] *= s_corr[h];
        }
#pragma unroll 4
        for (int key = 0; key < kTK; ++key) {
          const float2 v = Vec8<T>::pair(cs + key * tld + col);
          const float4 pa = *reinterpret_cast<const float4*>(&s_p[key][0]), pb = *reinterpret_cast<const float4*>(&s_p[key][4]);
          const float pw[kHG] = {pa.x, pa.y, pa.z, pa.w, pb.x, pb.y, pb.z, pb.w};
#pragma unroll
          for (int h = 0; h < kHG; ++h) {
            acc[c][h][0] = fmaf(pw[h], v.x, acc[c][h][0]);
            acc[c][h][1] = fmaf(pw[h], v.y, acc[c][h][1]);
          }
        }
      }
    }
  }
  const size_t base = (static_cast<size_t>(m) * a.heads + h0) * a.splits + split;
#pragma unroll
  for (int c = 0; c < NC; ++c) {
    const int col = c * 2 * kThreads + 2 * threadIdx.x;
    if (col < kv_ld) {
#pragma unroll
      for (int h = 0; h < kHG; ++h)
        if (h0 + h < a.heads)
          *reinterpret_cast<float2*>(a.part_o + (base + static_cast<size_t>(h) * a.splits) * kv_ld + col) =
              make_float2(acc[c][h][0], acc[c][h][1]);
    }
  }
  if (lane == 0 && h0 + warp < a.heads) {
    float* ml = a.part_ml + 2 * (base + static_cast<size_t>(warp) * a.splits);
    ml[0] = mx;
    ml[1] = l;
  }
}

constexpr int kMaxSplits = 64;
constexpr int kVC = 32;           // value rows per block

template <int RT>
__global__ void __launch_bounds__(kThreads) latent_out_kernel(const LatentArgs a) {
  extern __shared__ float lo_smem[];                     // [RT][kv_ld]
  __shared__ float ws[RT][kMaxSplits];
  pdl_wait();
  pdl_launch_dependents();
  const int h = blockIdx.x, v0 = blockIdx.y * kVC, m0 = blockIdx.z * RT, nr = min(RT, a.M - m0);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, kv_ld = a.cache.kv_ld;
  if (warp < nr) {
    const float* ml = a.part_ml + 2 * (static_cast<size_t>(m0 + warp) * a.heads + h) * a.splits;
    float mx = -INFINITY;
    for (int s = lane; s < a.splits; s += 32) mx = fmaxf(mx, ml[2 * s]);
    mx = warp_max(mx);
    float l = 0.f;
    for (int s = lane; s < a.splits; s += 32) {
      const float w = ml[2 * s] == -INFINITY ? 0.f : expf(ml[2 * s] - mx);
      ws[warp][s] = w;
      l = fmaf(w, ml[2 * s + 1], l);
    }
    l = warp_sum(l);
    const float inv = l > 0.f ? 1.0f / l : 0.f;
    for (int s = lane; s < a.splits; s += 32) ws[warp][s] *= inv;
  }
  __syncthreads();
  for (int r = 0; r < RT; ++r) {
    const float* po = a.part_o + (static_cast<size_t>(m0 + min(r, nr - 1)) * a.heads + h) * a.splits * kv_ld;
    for (int k = threadIdx.x; k < kv_ld; k += kThreads) {
      float v = 0.f;
      for (int s = 0; s < a.splits; ++s) v = fmaf(ws[min(r, nr - 1)][s], po[static_cast<size_t>(s) * kv_ld + k], v);
      lo_smem[r * kv_ld + k] = v;
    }
  }
  __syncthreads();
  for (int v = v0 + warp; v < min(v0 + kVC, a.vdim); v += kThreads / 32) {
    const __nv_bfloat16* w = a.w_uv + (static_cast<size_t>(h) * a.vdim + v) * kv_ld;
    float acc[RT] = {};
    for (int k = lane * 8; k < kv_ld; k += 256) {
      float w8[8];
      unpack8(ld_stream16(w + k), w8);
#pragma unroll
      for (int r = 0; r < RT; ++r) {
        const float* o = lo_smem + r * kv_ld + k;
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[r] = fmaf(w8[e], o[e], acc[r]);
      }
    }
#pragma unroll
    for (int r = 0; r < RT; ++r) {
      const float y = warp_sum(acc[r]);
      if (lane == 0 && r < nr) {
        const size_t o = static_cast<size_t>(m0 + r) * a.ld_out + h * a.vdim + v;
        if (a.out) a.out[o] = y;
        if (a.out_bf16) a.out_bf16[o] = __float2bfloat16_rn(y);
      }
    }
  }
}

// One block per row: latent norm, cache and c_lin / kr_lin rows, rotated queries packed per head into
// [own columns, padded | rotated columns, padded].
template <typename T>
__global__ void __launch_bounds__(kThreads) latent_pack_kernel(const LatentArgs a) {
  __shared__ float red[kThreads / 32];
  const int m = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5, hd = a.dim + a.rot;
  int seq;
  const int p = own_pos(a.rows, a.pad, m, &seq), pc = max(p, 0);
  const float2* sc = a.sincos + static_cast<size_t>(pc) * (a.rot >> 1);
  const float* row = a.p1 + static_cast<size_t>(m) * a.ld_p1;
  const float* c = row + a.heads * hd;
  float ss = 0.f;
  for (int i = threadIdx.x; i < a.rank; i += kThreads) ss = fmaf(c[i], c[i], ss);
  const float rs = 1.0f / sqrtf(la_block_sum(ss, red) / static_cast<float>(a.rank) + a.eps);
  const size_t lin = static_cast<size_t>(m / a.rows.Tc) * a.key_rows + a.hist + m % a.rows.Tc;
  T* cache = static_cast<T*>(a.cache.pool) + cache_row(a.cache, seq, pc);
  for (int i = threadIdx.x; i < a.rank; i += kThreads) {
    const float v = c[i] * rs * a.kv_norm[i];
    if (p >= 0) st(cache + i, v);
    a.c_lin[lin * a.cache.kv_ld + i] = __float2bfloat16_rn(v);
  }
  for (int j = threadIdx.x; j < a.kr_ld; j += kThreads) {
    const float v = j < a.rot ? rotated(c + a.rank, j, sc) : 0.f;
    if (p >= 0 && j < a.rot) st(cache + a.cache.kv_ld + j, v);
    a.kr_lin[lin * a.kr_ld + j] = __float2bfloat16_rn(v);
  }
  for (int h = warp; h < a.heads; h += kThreads / 32) {
    const float* q = row + h * hd;
    __nv_bfloat16* o = a.q_pack + (static_cast<size_t>(m) * a.heads + h) * (64 * a.key_blocks);
    for (int j = lane; j < a.dim; j += 32) o[j] = __float2bfloat16_rn(q[j]);
    for (int j = lane; j < a.rot; j += 32) o[64 * a.k_own + j] = __float2bfloat16_rn(rotated(q + a.dim, j, sc));
  }
}

template <typename T>
__global__ void __launch_bounds__(128) latent_history_kernel(const LatentArgs a) {
  const int i = blockIdx.x, b = blockIdx.y, seq = a.rows.b0 + b;
  const int p = a.rows.pos0_host - a.hist + i - a.pad[seq];
  const size_t lin = static_cast<size_t>(b) * a.key_rows + i;
  const T* cache = static_cast<const T*>(a.cache.pool) + cache_row(a.cache, seq, max(p, 0));
  auto get = [&](int j) { return p >= 0 ? static_cast<float>(cache[j]) : 0.f; };
  for (int j = threadIdx.x; j < a.rank; j += 128) a.c_lin[lin * a.cache.kv_ld + j] = __float2bfloat16_rn(get(j));
  for (int j = threadIdx.x; j < a.kr_ld; j += 128)
    a.kr_lin[lin * a.kr_ld + j] = __float2bfloat16_rn(j < a.rot ? get(a.cache.kv_ld + j) : 0.f);
}

bool latent_ok(const LatentArgs& a) {
  return a.M > 0 && a.heads > 0 && a.rank > 0 && a.cache.kv_ld >= a.rank && (a.cache.kv_ld & 7) == 0 &&
         (a.cache.row_ld & 7) == 0 && a.cache.row_ld - a.cache.kv_ld >= a.rot && a.cache.kv_ld <= kLatentMaxRank &&
         (a.rot & 1) == 0 && a.window > 0 && a.rows.Tc > 0;
}

template <typename K>
cudaError_t allow_smem(DeviceOnce& once, K kernel, int bytes) {
  return once.run([&] { return cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes); });
}

template <typename T, int RT>
cudaError_t absorb(const LatentArgs& a, cudaStream_t s, bool pdl) {
  static DeviceOnce once;
  const size_t smem = sizeof(float) * (static_cast<size_t>(RT) * a.dim + static_cast<size_t>(kThreads) * 8 * RT);
  cudaError_t e = allow_smem(once, latent_absorb_kernel<T, RT>, 160 * 1024);
  if (e != cudaSuccess) return e;
  if (smem > 160 * 1024) return cudaErrorInvalidValue;
  return launch_pdl(latent_absorb_kernel<T, RT>, dim3((a.M + RT - 1) / RT, a.heads + 1), dim3(kThreads), smem, s, pdl, a);
}

template <typename T, int NC>
cudaError_t attend(const LatentArgs& a, cudaStream_t s, bool pdl) {
  static DeviceOnce once;
  const size_t smem = sizeof(float) * kHG * a.cache.row_ld + sizeof(T) * kTK * (a.cache.row_ld + Vec8<T>::kPad);
  cudaError_t e = allow_smem(once, latent_attn_kernel<T, NC>, 220 * 1024);
  if (e != cudaSuccess) return e;
  if (smem > 220 * 1024) return cudaErrorInvalidValue;
  return launch_pdl(latent_attn_kernel<T, NC>, dim3(a.splits, (a.heads + kHG - 1) / kHG, a.M), dim3(kThreads), smem, s, pdl, a);
}

}  // namespace

int latent_attn_splits(int window) { return std::max(1, std::min(kMaxSplits, (window + 63) / 64)); }

cudaError_t launch_latent_absorb(const LatentArgs& a, cudaStream_t s, bool pdl) {
  if (!latent_ok(a)) return cudaErrorInvalidValue;
  if (a.cache.f32) return a.M == 1 ? absorb<float, 1>(a, s, pdl) : absorb<float, 4>(a, s, pdl);
  return a.M == 1 ? absorb<__nv_bfloat16, 1>(a, s, pdl) : absorb<__nv_bfloat16, 4>(a, s, pdl);
}

cudaError_t launch_latent_attn(const LatentArgs& a, cudaStream_t s, bool pdl) {
  if (!latent_ok(a) || a.splits < 1 || a.splits > kMaxSplits) return cudaErrorInvalidValue;
  const bool two = a.cache.kv_ld > 2 * kThreads;
  if (a.cache.f32) return two ? attend<float, 2>(a, s, pdl) : attend<float, 1>(a, s, pdl);
  return two ? attend<__nv_bfloat16, 2>(a, s, pdl) : attend<__nv_bfloat16, 1>(a, s, pdl);
}

cudaError_t launch_latent_out(const LatentArgs& a, cudaStream_t s, bool pdl) {
  if (!latent_ok(a) || a.splits < 1 || a.splits > kMaxSplits) return cudaErrorInvalidValue;
  const int chunks = (a.vdim + kVC - 1) / kVC;
  if (a.M == 1)
    return launch_pdl(latent_out_kernel<1>, dim3(a.heads, chunks, 1), dim3(kThreads), sizeof(float) * a.cache.kv_ld, s, pdl, a);
  return launch_pdl(latent_out_kernel<4>, dim3(a.heads, chunks, (a.M + 3) / 4), dim3(kThreads),
                    sizeof(float) * 4 * a.cache.kv_ld, s, pdl, a);
}

cudaError_t launch_latent_pack(const LatentArgs& a, cudaStream_t s) {
  if (!latent_ok(a) || a.kr_ld < a.rot || a.key_rows < a.hist + a.rows.Tc) return cudaErrorInvalidValue;
  if (a.cache.f32) latent_pack_kernel<float><<<a.M, kThreads, 0, s>>>(a);
  else latent_pack_kernel<__nv_bfloat16><<<a.M, kThreads, 0, s>>>(a);
  return cudaGetLastError();
}

cudaError_t launch_latent_history(const LatentArgs& a, cudaStream_t s) {
  if (a.hist <= 0) return cudaSuccess;
  if (!latent_ok(a) || a.nseq <= 0 || a.rows.pos0_dev) return cudaErrorInvalidValue;
  if (a.cache.f32) latent_history_kernel<float><<<dim3(a.hist, a.nseq), 128, 0, s>>>(a);
  else latent_history_kernel<__nv_bfloat16><<<dim3(a.hist, a.nseq), 128, 0, s>>>(a);
  return cudaGetLastError();
}

}  // namespace mtj
