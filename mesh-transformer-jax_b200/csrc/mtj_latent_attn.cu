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
constexpr int kAbsorbCols = 128;  // latent columns per block of the absorb kernel

__device__ __forceinline__ void cp16(uint32_t dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

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
  // a thread owns 8 latent columns of the block's chunk and every dsplit-th query dimension
  const int k0 = blockIdx.z * kAbsorbCols, cols = min(kAbsorbCols, a.cache.kv_ld - k0);
  const int groups = cols >> 3, dsplit = kThreads / groups;
  const int g = threadIdx.x % groups, ds = threadIdx.x / groups;
  const __nv_bfloat16* w =
      a.w_uk + static_cast<size_t>(blockIdx.y < a.heads ? blockIdx.y : 0) * a.dim * a.cache.kv_ld + k0 + g * 8;
  if (blockIdx.y < a.heads && ds < dsplit)
    for (int j = ds; j < a.dim; j += dsplit) prefetch_l2(w + static_cast<size_t>(j) * a.cache.kv_ld);
  pdl_wait();
  pdl_launch_dependents();
  const int m0 = blockIdx.x * RT, nr = min(RT, a.M - m0);
  if (blockIdx.y == a.heads) {
    if (blockIdx.z) return;
    // one row: the whole block; several: a warp per row
    constexpr int kW = RT == 1 ? kThreads : 32;
    const int lane = threadIdx.x % kW;
    for (int r = threadIdx.x / kW; r < nr; r += kThreads / kW) {
      int seq;
      const int p = own_pos(a.rows, a.pad, m0 + r, &seq);
      const float* c = a.p1 + static_cast<size_t>(m0 + r) * a.ld_p1 + a.heads * (a.dim + a.rot);
      constexpr int kC = kLatentMaxRank / kW;
      float cv[kC], ss = 0.f;
#pragma unroll
      for (int i = 0; i < kC; ++i) cv[i] = i * kW + lane < a.rank ? c[i * kW + lane] : 0.f;
#pragma unroll
      for (int i = 0; i < kC; ++i) ss = fmaf(cv[i], cv[i], ss);
      ss = RT == 1 ? la_block_sum(ss, red) : warp_sum(ss);
      const float rs = 1.0f / sqrtf(ss / static_cast<float>(a.rank) + a.eps);
      if (p < 0) continue;
      T* row = static_cast<T*>(a.cache.pool) + cache_row(a.cache, seq, p);
      const float2* sc = a.sincos + static_cast<size_t>(p) * (a.rot >> 1);
      for (int j = lane; j < a.rot; j += kW) st(row + a.cache.kv_ld + j, rotated(c + a.rank, j, sc));
#pragma unroll
      for (int i = 0; i < kC; ++i)
        if (i * kW + lane < a.rank) st(row + i * kW + lane, cv[i] * rs * a.kv_norm[i * kW + lane]);
    }
    return;
  }
  const int h = blockIdx.y, hd = a.dim + a.rot;
  float* qs = ab_smem;                                  // [RT][dim]
  float* part = ab_smem + RT * a.dim;                   // [dsplit][RT][cols]
  {
    const float* q = a.p1 + static_cast<size_t>(m0) * a.ld_p1 + h * hd;
#pragma unroll 4
    for (int i = threadIdx.x; i < nr * a.dim; i += kThreads)
      qs[i] = q[static_cast<size_t>(i / a.dim) * a.ld_p1 + i % a.dim] * a.scale;
    for (int i = nr * a.dim + threadIdx.x; i < RT * a.dim; i += kThreads) qs[i] = 0.f;
    const int rot_ld = a.cache.row_ld - a.cache.kv_ld;
    if (blockIdx.z == 0)
#pragma unroll 2
      for (int i = threadIdx.x; i < nr * rot_ld; i += kThreads) {
        const int r = i / rot_ld, j = i % rot_ld;
        int seq;
        const int p = max(own_pos(a.rows, a.pad, m0 + r, &seq), 0);
        const float2* sc = a.sincos + static_cast<size_t>(p) * (a.rot >> 1);
        a.q_abs[(static_cast<size_t>(m0 + r) * a.heads + h) * a.cache.row_ld + a.cache.kv_ld + j] =
            j < a.rot ? rotated(q + static_cast<size_t>(r) * a.ld_p1 + a.dim, j, sc) * a.scale : 0.f;
      }
  }
  __syncthreads();
  if (ds < dsplit) {
    float acc[RT][8] = {};
#pragma unroll 8
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
      for (int e = 0; e < 8; ++e) part[(ds * RT + r) * cols + g * 8 + e] = acc[r][e];
  }
  __syncthreads();
  for (int i = threadIdx.x; i < nr * cols; i += kThreads) {
    const int r = i / cols, k = i % cols;
    float v = 0.f;
    for (int d = 0; d < dsplit; ++d) v += part[(d * RT + r) * cols + k];
    a.q_abs[(static_cast<size_t>(m0 + r) * a.heads + h) * a.cache.row_ld + k0 + k] = v;
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
    for (int key = warp; key < kTK; key += kThreads / 32) {           // a warp per row, all copies in flight at once
      T* dst = cs + key * tld;
      if (kt + key < k1) {
        const T* src = static_cast<const T*>(a.cache.pool) + cache_row(a.cache, seq, kt + key);
        for (int c = lane; c < nv; c += 32) cp16(smem_u32(dst + c * kVec), src + c * kVec);
      } else {
        for (int c = lane; c < nv; c += 32) *reinterpret_cast<uint4*>(dst + c * kVec) = make_uint4(0u, 0u, 0u, 0u);
      }
    }
    cp_commit();
    cp_wait<0>();
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

// The same for several rows at a time with bf16 caches, on the tensor cores: one block = (row, 16 MT heads, key range).
// The heads are the M dimension of mma.m16n8k16: S[heads, 32 keys] = Q' . C^T, fp32 online softmax, O[heads, latent] +=
// P . C from the same tile, so a cached byte is read once per 16 MT heads.  A warp owns NT 8-column blocks of O.  Tiles
// come by cp.async, one ahead.  (M is the number of heads, far below the 128 rows of a tcgen05 tile, and the bound is
// the cache traffic.)
__device__ __forceinline__ void ldsm4(uint32_t* r, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm2(uint32_t* r, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];" : "=r"(r[0]), "=r"(r[1]) : "r"(addr));
}
__device__ __forceinline__ void ldsm4t(uint32_t* r, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mma16816(float* d, const uint32_t* a, const uint32_t* b) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b[0]), "r"(b[1]));
}

template <int MT>
constexpr size_t mma_smem_bytes(int row_ld) {
  const size_t row = (row_ld + 15) / 16 * 16 + 8;       // an odd number of 16-byte units: conflict-free ldmatrix
  return 2 * row * (16 * MT + 2 * kTK) + 2 * 16 * MT * 40 + 4 * (3 - MT) * 16 * MT * (kTK + 1) + 4 * 16 * MT;
}

template <int MT, int NT>
__global__ void __launch_bounds__(kThreads) latent_attn_mma_kernel(const LatentArgs a) {
  constexpr int HM = 16 * MT, KH = 3 - MT;               // MT == 1: two warps share a score tile, half of K each
  constexpr int kPld = 40, kSld = kTK + 1;
  extern __shared__ __align__(16) unsigned char lm_smem[];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int ld = a.cache.row_ld, kv_ld = a.cache.kv_ld, kd = (ld + 15) & ~15, sld = kd + 8;
  __nv_bfloat16* qs = reinterpret_cast<__nv_bfloat16*>(lm_smem);            // [HM][sld]
  __nv_bfloat16* cs = qs + HM * sld;                                        // [2][kTK][sld]
  __nv_bfloat16* ps = cs + 2 * kTK * sld;                                   // [HM][kPld]
  float* ss = reinterpret_cast<float*>(ps + HM * kPld);                     // [KH][HM][kSld]
  float* corr_s = ss + KH * HM * kSld;                                      // [HM]
  const int m = blockIdx.z, h0 = blockIdx.y * HM, split = blockIdx.x;
  pdl_wait();
  pdl_launch_dependents();
  int seq;
  const int p = own_pos(a.rows, a.pad, m, &seq);
  const int lo = max(0, p - a.window + 1), n = p - lo + 1;
  const int per = (((max(n, 0) + a.splits - 1) / a.splits) + kTK - 1) / kTK * kTK;
  const int k0 = lo + split * per, k1 = min(k0 + per, p + 1);
  const int nv = ld >> 3;
  auto fetch = [&](int kt, int b) {
    for (int key = warp; key < kTK; key += kThreads / 32) {
      __nv_bfloat16* dst = cs + (b * kTK + key) * sld;
      if (kt + key < k1) {
        const __nv_bfloat16* src = static_cast<const __nv_bfloat16*>(a.cache.pool) + cache_row(a.cache, seq, kt + key);
        for (int c = lane; c < nv; c += 32) cp16(smem_u32(dst + c * 8), src + c * 8);
      } else {
        for (int c = lane; c < nv; c += 32) *reinterpret_cast<uint4*>(dst + c * 8) = make_uint4(0u, 0u, 0u, 0u);
      }
    }
    cp_commit();
  };
  if (k0 < k1) fetch(k0, 0);
  for (int i = threadIdx.x; i < HM * (kd >> 3); i += kThreads) {
    const int h = i / (kd >> 3), c = i % (kd >> 3) * 8;
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (h0 + h < a.heads && c < ld) {
      const float4* q = reinterpret_cast<const float4*>(a.q_abs + (static_cast<size_t>(m) * a.heads + h0 + h) * ld + c);
      const float4 x = q[0], y = q[1];
      v = make_uint4(pack_bf16x2(x.x, x.y), pack_bf16x2(x.z, x.w), pack_bf16x2(y.x, y.y), pack_bf16x2(y.z, y.w));
    }
    *reinterpret_cast<uint4*>(qs + h * sld + c) = v;
  }
  if (kd > ld)                                           // the last half block of K in the key tiles
    for (int i = threadIdx.x; i < 2 * kTK; i += kThreads) *reinterpret_cast<uint4*>(cs + i * sld + ld) = make_uint4(0u, 0u, 0u, 0u);

  float acc[MT][NT][4] = {};
  float mx[2 * MT], l[2 * MT];                           // of rows warp, warp + 8, ...
#pragma unroll
  for (int i = 0; i < 2 * MT; ++i) {
    mx[i] = -INFINITY;
    l[i] = 0.f;
  }
  const uint32_t q_base = smem_u32(qs), p_base = smem_u32(ps);
  for (int kt = k0, it = 0; kt < k1; kt += kTK, ++it) {
    const int b = it & 1;
    const uint32_t c_base = smem_u32(cs + b * kTK * sld);
    if (kt + kTK < k1) {
      fetch(kt + kTK, b ^ 1);
      cp_wait<1>();
    } else {
      cp_wait<0>();
    }
    __syncthreads();
    {
      const int mt = MT == 2 ? warp >> 2 : 0, kh = MT == 2 ? 0 : warp >> 2, nt = warp & 3;
      const int ks = kd >> 4, s0 = KH == 2 ? kh * (ks >> 1) : 0, s1 = KH == 2 && kh == 0 ? ks >> 1 : ks;
      float s4[2][4] = {};
      const uint32_t qa = q_base + 2u * ((mt * 16 + (lane & 15)) * sld + (lane >> 4) * 8);
      const uint32_t ca = c_base + 2u * ((nt * 8 + (lane & 7)) * sld + ((lane >> 3) & 1) * 8);
#pragma unroll 2
      for (int k = s0; k < s1; k += 2) {                   // two chains
        uint32_t af[4], bf[2];
        ldsm4(af, qa + 32u * k);
        ldsm2(bf, ca + 32u * k);
        mma16816(s4[0], af, bf);
        if (k + 1 < s1) {
          ldsm4(af, qa + 32u * k + 32u);
          ldsm2(bf, ca + 32u * k + 32u);
          mma16816(s4[1], af, bf);
        }
      }
      float* sp = ss + (kh * HM + mt * 16 + (lane >> 2)) * kSld + nt * 8 + (lane & 3) * 2;
      sp[0] = s4[0][0] + s4[1][0];
      sp[1] = s4[0][1] + s4[1][1];
      sp[8 * kSld] = s4[0][2] + s4[1][2];
      sp[8 * kSld + 1] = s4[0][3] + s4[1][3];
    }
    __syncthreads();
#pragma unroll
    for (int i = 0; i < 2 * MT; ++i) {
      const int r = warp + 8 * i;
      float s = ss[r * kSld + lane];
      if (KH == 2) s += ss[(HM + r) * kSld + lane];
      if (kt + lane >= k1) s = -INFINITY;
      const float m_new = fmaxf(mx[i], warp_max(s));
      const float corr = __expf(mx[i] - m_new), w = __expf(s - m_new);
      l[i] = l[i] * corr + warp_sum(w);
      mx[i] = m_new;
      ps[r * kPld + lane] = __float2bfloat16_rn(w);
      if (lane == 0) corr_s[r] = corr;
    }
    __syncthreads();
    uint32_t pf[MT][2][4];
#pragma unroll
    for (int mt = 0; mt < MT; ++mt) {
      const float c0 = corr_s[mt * 16 + (lane >> 2)], c1 = corr_s[mt * 16 + (lane >> 2) + 8];
#pragma unroll
      for (int j = 0; j < NT; ++j) {
        acc[mt][j][0] *= c0;
        acc[mt][j][1] *= c0;
        acc[mt][j][2] *= c1;
        acc[mt][j][3] *= c1;
      }
#pragma unroll
      for (int k = 0; k < 2; ++k) ldsm4(pf[mt][k], p_base + 2u * ((mt * 16 + (lane & 15)) * kPld + k * 16 + (lane >> 4) * 8));
    }
#pragma unroll
    for (int j = 0; j < NT; j += 2) {
      const int col = (warp * NT + j) * 8;
      if (col < kv_ld) {
#pragma unroll
        for (int k = 0; k < 2; ++k) {
          uint32_t bf[4];
          ldsm4t(bf, c_base + 2u * ((k * 16 + (lane & 15)) * sld + col + (lane >> 4) * 8));
#pragma unroll
          for (int mt = 0; mt < MT; ++mt) {
            mma16816(acc[mt][j], pf[mt][k], bf);
            mma16816(acc[mt][j + 1], pf[mt][k], bf + 2);
          }
        }
      }
    }
    __syncthreads();                                     // the tile may be fetched over
  }
  const size_t base = (static_cast<size_t>(m) * a.heads + h0) * a.splits + split;
#pragma unroll
  for (int mt = 0; mt < MT; ++mt)
#pragma unroll
    for (int j = 0; j < NT; ++j) {
      const int col = (warp * NT + j) * 8 + (lane & 3) * 2, h = mt * 16 + (lane >> 2);
      if (col < kv_ld) {
        if (h0 + h < a.heads)
          *reinterpret_cast<float2*>(a.part_o + (base + static_cast<size_t>(h) * a.splits) * kv_ld + col) = make_float2(acc[mt][j][0], acc[mt][j][1]);
        if (h0 + h + 8 < a.heads)
          *reinterpret_cast<float2*>(a.part_o + (base + static_cast<size_t>(h + 8) * a.splits) * kv_ld + col) = make_float2(acc[mt][j][2], acc[mt][j][3]);
      }
    }
#pragma unroll
  for (int i = 0; i < 2 * MT; ++i) {
    const int r = warp + 8 * i;
    if (lane == 0 && h0 + r < a.heads) {
      float* ml = a.part_ml + 2 * (base + static_cast<size_t>(r) * a.splits);
      ml[0] = mx[i];
      ml[1] = l[i];
    }
  }
}

constexpr int kMaxSplits = 64;
constexpr int kMmaRows = 5;       // rows from which the tensor-core form is used
constexpr int kVC = 32;           // value rows per block

// KC = 256-column chunks of a latent row; a warp owns four value rows, whose weights it has loaded before the
// predecessor kernel is done.
template <int RT, int KC>
__global__ void __launch_bounds__(kThreads) latent_out_kernel(const LatentArgs a) {
  extern __shared__ float lo_smem[];                     // [RT][kv_ld]
  __shared__ float ws[RT][kMaxSplits];
  constexpr int kVW = kVC / (kThreads / 32);             // value rows per warp
  const int h = blockIdx.x, v0 = blockIdx.y * kVC, m0 = blockIdx.z * RT, nr = min(RT, a.M - m0);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, kv_ld = a.cache.kv_ld;
  uint4 w[kVW][KC];
#pragma unroll
  for (int i = 0; i < kVW; ++i)
#pragma unroll
    for (int c = 0; c < KC; ++c) {
      const int v = v0 + warp * kVW + i, k = c * 256 + lane * 8;
      w[i][c] = v < a.vdim && k < kv_ld ? ld_stream16(a.w_uv + (static_cast<size_t>(h) * a.vdim + v) * kv_ld + k) : make_uint4(0u, 0u, 0u, 0u);
    }
  pdl_wait();
  pdl_launch_dependents();
  for (int r = warp; r < nr; r += kThreads / 32) {
    const float* ml = a.part_ml + 2 * (static_cast<size_t>(m0 + r) * a.heads + h) * a.splits;
    float mx = -INFINITY;
    for (int s = lane; s < a.splits; s += 32) mx = fmaxf(mx, ml[2 * s]);
    mx = warp_max(mx);
    float l = 0.f;
    for (int s = lane; s < a.splits; s += 32) {
      const float e = ml[2 * s] == -INFINITY ? 0.f : expf(ml[2 * s] - mx);
      ws[r][s] = e;
      l = fmaf(e, ml[2 * s + 1], l);
    }
    l = warp_sum(l);
    const float inv = l > 0.f ? 1.0f / l : 0.f;
    for (int s = lane; s < a.splits; s += 32) ws[r][s] *= inv;
  }
  __syncthreads();
  // RT == 1: two threads share a column group, each adding half of the ranges
  constexpr int kParts = RT == 1 ? 2 : 1;
  const int k4 = kv_ld >> 2;
#pragma unroll 2
  for (int i = threadIdx.x; i < kParts * nr * k4; i += kThreads) {
    const int part = i / (nr * k4), j = i % (nr * k4), r = j / k4, k = j % k4;
    const float4* po = reinterpret_cast<const float4*>(a.part_o + (static_cast<size_t>(m0 + r) * a.heads + h) * a.splits * kv_ld) + k;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    constexpr int kIn = RT == 1 ? 16 : 4;                // loads in flight
    for (int s0 = part; s0 < a.splits; s0 += kIn * kParts) {
      float4 p[kIn];
#pragma unroll
      for (int i = 0; i < kIn; ++i) p[i] = po[static_cast<size_t>(min(s0 + i * kParts, a.splits - 1)) * k4];
#pragma unroll
      for (int i = 0; i < kIn; ++i) {
        const int s = s0 + i * kParts;
        const float e = s < a.splits ? ws[r][s] : 0.f;
        v.x = fmaf(e, p[i].x, v.x); v.y = fmaf(e, p[i].y, v.y); v.z = fmaf(e, p[i].z, v.z); v.w = fmaf(e, p[i].w, v.w);
      }
    }
    reinterpret_cast<float4*>(lo_smem)[i] = v;
  }
  __syncthreads();
  if (kParts == 2) {
    for (int i = threadIdx.x; i < kv_ld; i += kThreads) lo_smem[i] += lo_smem[kv_ld + i];
    __syncthreads();
  }
  for (int r = 0; r < nr; ++r) {
    float acc[kVW] = {};
#pragma unroll
    for (int c = 0; c < KC; ++c) {
      const int k = c * 256 + lane * 8;
      if (k < kv_ld) {
        const float4 o0 = *reinterpret_cast<const float4*>(lo_smem + r * kv_ld + k), o1 = *reinterpret_cast<const float4*>(lo_smem + r * kv_ld + k + 4);
        const float o[8] = {o0.x, o0.y, o0.z, o0.w, o1.x, o1.y, o1.z, o1.w};
#pragma unroll
        for (int i = 0; i < kVW; ++i) {
          float w8[8];
          unpack8(w[i][c], w8);
#pragma unroll
          for (int e = 0; e < 8; ++e) acc[i] = fmaf(w8[e], o[e], acc[i]);
        }
      }
    }
    float y = 0.f;
#pragma unroll
    for (int i = 0; i < kVW; ++i) {
      const float t = warp_sum(acc[i]);
      if (lane == i) y = t;
    }
    const int v = v0 + warp * kVW + lane;
    if (lane < kVW && v < a.vdim) {
      const size_t o = static_cast<size_t>(m0 + r) * a.ld_out + h * a.vdim + v;
      if (a.out) a.out[o] = y;
      if (a.out_bf16) a.out_bf16[o] = __float2bfloat16_rn(y);
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
    if (((a.dim | a.rot | a.ld_p1) & 3) == 0) {
      for (int j = 4 * lane; j < a.dim; j += 128) {
        const float4 v = *reinterpret_cast<const float4*>(q + j);
        *reinterpret_cast<uint2*>(o + j) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
      }
      for (int j = 4 * lane; j < a.rot; j += 128) {
        const float4 v = *reinterpret_cast<const float4*>(q + a.dim + j);
        const float2 s0 = sc[j >> 1], s1 = sc[(j >> 1) + 1];
        *reinterpret_cast<uint2*>(o + 64 * a.k_own + j) =
            make_uint2(pack_bf16x2(v.x * s0.y - v.y * s0.x, v.y * s0.y + v.x * s0.x),
                       pack_bf16x2(v.z * s1.y - v.w * s1.x, v.w * s1.y + v.z * s1.x));
      }
    } else {
      for (int j = lane; j < a.dim; j += 32) o[j] = __float2bfloat16_rn(q[j]);
      for (int j = lane; j < a.rot; j += 32) o[64 * a.k_own + j] = __float2bfloat16_rn(rotated(q + a.dim, j, sc));
    }
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
  return launch_pdl(latent_absorb_kernel<T, RT>, dim3((a.M + RT - 1) / RT, a.heads + 1, (a.cache.kv_ld + kAbsorbCols - 1) / kAbsorbCols), dim3(kThreads), smem, s, pdl, a);
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

template <int MT, int NT>
cudaError_t attend_mma(const LatentArgs& a, cudaStream_t s, bool pdl) {
  static DeviceOnce once;
  cudaError_t e = allow_smem(once, latent_attn_mma_kernel<MT, NT>, 220 * 1024);
  if (e != cudaSuccess) return e;
  return launch_pdl(latent_attn_mma_kernel<MT, NT>, dim3(a.splits, (a.heads + 16 * MT - 1) / (16 * MT), a.M), dim3(kThreads),
                    mma_smem_bytes<MT>(a.cache.row_ld), s, pdl, a);
}

// 16 heads per block (two blocks per SM at a 576-column cache row); 32 were slower, one block per SM
bool use_mma(int M, int row_ld, int tensor_cores) {
  return tensor_cores && M >= kMmaRows && mma_smem_bytes<1>(row_ld) <= 220 * 1024;
}

}  // namespace

int latent_attn_splits(int M, int heads, int row_ld, int tensor_cores, int window) {
  const bool mma = use_mma(M, row_ld, tensor_cores);
  const int groups = M * (mma ? (heads + 15) / 16 : (heads + kHG - 1) / kHG);
  // one wave of blocks: two per SM for the tensor-core form, four for the other
  return std::max(1, std::min({kMaxSplits, (window + kTK - 1) / kTK, (mma ? 296 : kLatentBlocks) / groups}));
}

cudaError_t launch_latent_absorb(const LatentArgs& a, cudaStream_t s, bool pdl) {
  if (!latent_ok(a)) return cudaErrorInvalidValue;
  if (a.cache.f32) return a.M == 1 ? absorb<float, 1>(a, s, pdl) : absorb<float, 8>(a, s, pdl);
  return a.M == 1 ? absorb<__nv_bfloat16, 1>(a, s, pdl) : absorb<__nv_bfloat16, 8>(a, s, pdl);
}

cudaError_t launch_latent_attn(const LatentArgs& a, cudaStream_t s, bool pdl) {
  if (!latent_ok(a) || a.splits < 1 || a.splits > kMaxSplits) return cudaErrorInvalidValue;
  if (use_mma(a.M, a.cache.row_ld, a.tensor_cores && !a.cache.f32)) {
    const int nt = (a.cache.kv_ld + 63) / 64;             // 8-column blocks per warp
    return nt <= 2 ? attend_mma<1, 2>(a, s, pdl) : nt <= 4 ? attend_mma<1, 4>(a, s, pdl) : nt <= 8 ? attend_mma<1, 8>(a, s, pdl) : attend_mma<1, 16>(a, s, pdl);
  }
  const bool two = a.cache.kv_ld > 2 * kThreads;
  if (a.cache.f32) return two ? attend<float, 2>(a, s, pdl) : attend<float, 1>(a, s, pdl);
  return two ? attend<__nv_bfloat16, 2>(a, s, pdl) : attend<__nv_bfloat16, 1>(a, s, pdl);
}

cudaError_t launch_latent_out(const LatentArgs& a, cudaStream_t s, bool pdl) {
  if (!latent_ok(a) || a.splits < 1 || a.splits > kMaxSplits) return cudaErrorInvalidValue;
  const int chunks = (a.vdim + kVC - 1) / kVC, kc = (a.cache.kv_ld + 255) / 256;
  auto go = [&](auto kernel, int rt) {
    return launch_pdl(kernel, dim3(a.heads, chunks, (a.M + rt - 1) / rt), dim3(kThreads), sizeof(float) * std::max(rt, 2) * a.cache.kv_ld, s, pdl, a);
  };
  if (a.M == 1) return kc == 1 ? go(latent_out_kernel<1, 1>, 1) : kc == 2 ? go(latent_out_kernel<1, 2>, 1) : go(latent_out_kernel<1, 4>, 1);
  if (a.M <= 8 || kc > 2) return kc == 1 ? go(latent_out_kernel<8, 1>, 8) : kc == 2 ? go(latent_out_kernel<8, 2>, 8) : go(latent_out_kernel<8, 4>, 8);
  return kc == 1 ? go(latent_out_kernel<16, 1>, 16) : go(latent_out_kernel<16, 2>, 16);
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
