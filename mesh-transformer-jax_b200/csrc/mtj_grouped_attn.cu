// Softmax attention of query heads over shared key / value heads, with RMS norms over the whole query and key
// projections and an optional position-dependent query temperature; keys and values are cached in pages addressed by
// the position inside the sequence.
//
//   grouped_prep_kernel      a block per row: norms, temperature, query layout, cache write
//   grouped_attn_mma_kernel  bf16 caches, a row at a time (decoding, short portions): one block = (row, key head, key
//                            range), the query heads of the group as the M dimension of mma.m16n8k16.  Every warp walks
//                            16-key pieces of its own through a cp.async ring, so the warps meet only once, at the end;
//                            the last block of a (row, key head) adds the key ranges.  (M is the group size, far
//                            below the 128 rows of a tcgen05 tile, and the bound is the cache traffic.)
//   grouped_attn_kernel      the same on CUDA cores: fp32 caches, and head sizes beyond the other
// Prompts take the tensor-core attention over the same pages (mtj_attn_tc_grouped.cu).  Scores and softmax are fp32.
#include <math.h>

#include <algorithm>

#include "mtj_common.cuh"
#include "mtj_stack_kernels.h"

namespace mtj {
namespace {

constexpr int kPrepThreads = 256;
constexpr int kPiece = 16;        // keys per step of a warp; key ranges are multiples of it
constexpr int kMaxSplits = 64;

__device__ __forceinline__ void st(float* p, float v) { *p = v; }
__device__ __forceinline__ void st(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ void st4(float* p, const float4& v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void st4(__nv_bfloat16* p, const float4& v) {
  *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
}
__device__ __forceinline__ float get(const float* p) { return *p; }
__device__ __forceinline__ float get(const __nv_bfloat16* p) { return __bfloat162float(*p); }

// position of row m inside its sequence (negative: left padding)
__device__ __forceinline__ int own_pos(const RowMap& r, const int32_t* pad, int m, int* seq) {
  *seq = r.b0 + m / r.Tc;
  return (r.pos0_dev ? *r.pos0_dev : r.pos0_host) + m % r.Tc - pad[*seq];
}
// row of position p in the caches
__device__ __forceinline__ size_t cache_row(const GroupedCache& c, int seq, int p) {
  const int page = c.page_table[static_cast<size_t>(seq) * c.ring_pages + (p / kPageTokens) % c.ring_pages];
  return static_cast<size_t>(page) * kPageTokens + p % kPageTokens;
}

__device__ __forceinline__ float prep_block_sum(float v, float* red) {
  v = warp_sum(v);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  if (lane == 0) red[warp] = v;
  __syncthreads();
  float t = 0.f;
#pragma unroll
  for (int i = 0; i < kPrepThreads / 32; ++i) t += red[i];
  __syncthreads();
  return t;
}

// n numbers (heads of `per`) scaled and weighted into heads of ld columns, columns per .. ld - 1 zero (rs < 0: plain copy)
template <typename T>
__device__ __forceinline__ void place_heads(const float* src, int n, int per, const float* w, float rs, T* dst, int ld, bool vec) {
  if (vec) {
#pragma unroll 2
    for (int i = 4 * threadIdx.x; i < n; i += 4 * kPrepThreads) {
      float4 v = *reinterpret_cast<const float4*>(src + i);
      if (w) {
        const float4 f = *reinterpret_cast<const float4*>(w + i);
        v = make_float4(v.x * rs * f.x, v.y * rs * f.y, v.z * rs * f.z, v.w * rs * f.w);
      }
      st4(dst + static_cast<size_t>(i / per) * ld + i % per, v);
    }
  } else {
    for (int i = threadIdx.x; i < n; i += kPrepThreads)
      st(dst + static_cast<size_t>(i / per) * ld + i % per, w ? src[i] * rs * w[i] : src[i]);
  }
  const int gap = ld - per, heads = n / per;
  for (int i = threadIdx.x; i < heads * gap; i += kPrepThreads) st(dst + static_cast<size_t>(i / gap) * ld + per + i % gap, 0.f);
}

template <typename T, typename TQ>
__global__ void __launch_bounds__(kPrepThreads) grouped_prep_kernel(const GroupedAttnArgs a) {
  __shared__ float red[kPrepThreads / 32];
  pdl_wait();
  pdl_launch_dependents();
  const int m = blockIdx.x, nq = a.heads * a.dim, nk = a.own_kv ? a.kv_heads * a.dim : 0;
  int seq;
  const int p = own_pos(a.rows, a.pad, m, &seq);
  const float* row = a.p1 + static_cast<size_t>(m) * a.ld_p1;
  const bool vec = ((a.dim | a.vdim | a.ld_p1) & 3) == 0;
  float qs = 0.f, ks = 0.f;
  if (vec) {
#pragma unroll 4
    for (int i = 4 * threadIdx.x; i < nq + nk; i += 4 * kPrepThreads) {
      const float4 v = *reinterpret_cast<const float4*>(row + i);
      const float s = (v.x * v.x + v.y * v.y) + (v.z * v.z + v.w * v.w);
      if (i < nq) qs += s;
      else ks += s;
    }
  } else {
    for (int i = threadIdx.x; i < nq + nk; i += kPrepThreads) {
      const float v = row[i];
      if (i < nq) qs = fmaf(v, v, qs);
      else ks = fmaf(v, v, ks);
    }
  }
  qs = prep_block_sum(qs, red);
  if (nk) ks = prep_block_sum(ks, red);
  float rq = 1.0f / sqrtf(qs / static_cast<float>(nq) + a.eps);
  if (a.q_temp_every > 0.0)
    rq *= 1.0f + a.q_temp_coef * logf(static_cast<float>(floor((max(p, 0) + 1.0) / a.q_temp_every)) + 1.0f);
  const size_t qld = static_cast<size_t>(a.heads) * a.q_cols;
  TQ* q = sizeof(TQ) == 2 ? reinterpret_cast<TQ*>(a.q_bf16) : reinterpret_cast<TQ*>(a.q_f32);
  place_heads(row, nq, a.dim, a.q_norm, rq, q + m * qld, a.q_cols, vec);
  if (!nk || p < 0) return;
  const size_t cr = cache_row(a.cache, seq, p);
  const float rk = 1.0f / sqrtf(ks / static_cast<float>(nk) + a.eps);
  place_heads(row + nq, nk, a.dim, a.k_norm, rk, static_cast<T*>(a.cache.k) + cr * a.cache.k_ld, a.cache.k_ld / a.kv_heads, vec);
  place_heads(row + nq + nk, a.kv_heads * a.vdim, a.vdim, static_cast<const float*>(nullptr), 1.0f,
              static_cast<T*>(a.cache.v) + cr * a.cache.v_ld, a.cache.v_ld / a.kv_heads, vec);
}

// ---- what the row-at-a-time kernels share: the key range of a block and the end of a (row, key head)
struct Range {
  int seq, k0, k1, lo;                // keys [max(k0, lo), k1)
};
__device__ __forceinline__ Range key_range(const GroupedAttnArgs& a, int m, int split) {
  Range r;
  const int p = own_pos(a.rows, a.pad, m, &r.seq);
  const int lo = max(0, p - a.window + 1), n = p - lo + 1;            // n <= 0: a padding row
  const int first = lo / kPiece * kPiece, per = ((max(n, 0) + lo - first + a.splits - 1) / a.splits + kPiece - 1) / kPiece * kPiece;
  r.k0 = first + split * per;                          // pieces lie inside one page
  r.k1 = min(r.k0 + per, p + 1);
  r.lo = lo;
  return r;
}
__device__ __forceinline__ float ex2(float x) {
  float y;
  asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
  return y;
}
template <bool BASE2>
__device__ __forceinline__ float weight_of(float m, float ref) {      // exp of a difference of maxima, 0 for an empty range
  return m == -INFINITY ? 0.f : BASE2 ? ex2(m - ref) : expf(m - ref);
}

// Adds the key ranges of `nh` query heads once the last block of them has arrived, a warp per head; all threads of every
// block call it behind their stores to part_o / part_ml.  ws: kMaxSplits floats of shared memory per warp.
template <bool BASE2, int THREADS>
__device__ __forceinline__ void finish_heads(const GroupedAttnArgs& a, int m, int h0, int nh, uint32_t* counter, float* ws_all) {
  __shared__ bool is_last;
  __threadfence();
  __syncthreads();
  if (threadIdx.x == 0) is_last = atomicAdd(counter, 1u) == static_cast<uint32_t>(a.splits) - 1u;
  __syncthreads();
  if (!is_last) return;
  __threadfence();
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  float* ws = ws_all + warp * kMaxSplits;
  for (int h = h0 + warp; h < h0 + nh; h += THREADS / 32) {
    const size_t base = (static_cast<size_t>(m) * a.heads + h) * a.splits;
    const float* ml = a.part_ml + 2 * base;
    constexpr int kPer = kMaxSplits / 32;
    float2 r[kPer];                                    // (maximum, denominator) of ranges lane, lane + 32
    float mx = -INFINITY, l = 0.f;
#pragma unroll
    for (int i = 0; i < kPer; ++i) {
      const int s = lane + 32 * i;
      r[i] = s < a.splits ? make_float2(__ldcg(ml + 2 * s), __ldcg(ml + 2 * s + 1)) : make_float2(-INFINITY, 0.f);
      mx = fmaxf(mx, r[i].x);
    }
    mx = warp_max(mx);
#pragma unroll
    for (int i = 0; i < kPer; ++i) {
      r[i].x = weight_of<BASE2>(r[i].x, mx);
      l = fmaf(r[i].x, r[i].y, l);
    }
    l = warp_sum(l);
    const float inv = l > 0.f ? 1.0f / l : 0.f;
    __syncwarp();                                      // the last head's weights are read
#pragma unroll
    for (int i = 0; i < kPer; ++i) ws[lane + 32 * i] = r[i].x * inv;
    __syncwarp();
    const float* po = a.part_o + base * a.vdim;
    const size_t o = static_cast<size_t>(m) * a.ld_out + h * a.vdim;
    if (((a.vdim | a.ld_out) & 3) == 0) {
      for (int c = 4 * lane; c < a.vdim; c += 128) {
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
        for (int s = 0; s < a.splits; ++s) {
          const float4 p = __ldcg(reinterpret_cast<const float4*>(po + static_cast<size_t>(s) * a.vdim + c));
          const float e = ws[s];
          v.x = fmaf(e, p.x, v.x); v.y = fmaf(e, p.y, v.y); v.z = fmaf(e, p.z, v.z); v.w = fmaf(e, p.w, v.w);
        }
        if (a.out) st4(a.out + o + c, v);
        if (a.out_bf16) st4(a.out_bf16 + o + c, v);
      }
    } else {
      for (int c = lane; c < a.vdim; c += 32) {
        float v = 0.f;
#pragma unroll 8
        for (int s = 0; s < a.splits; ++s) v = fmaf(ws[s], __ldcg(po + static_cast<size_t>(s) * a.vdim + c), v);
        if (a.out) a.out[o + c] = v;
        if (a.out_bf16) a.out_bf16[o + c] = __float2bfloat16_rn(v);
      }
    }
  }
  if (threadIdx.x == 0) *counter = 0u;
}

// ------------------------------------------------------------------------------------------- CUDA cores
constexpr int kTK = 32;           // keys per tile (= lanes)
constexpr int kHG = 8;            // query heads per block (= warps)

__host__ __device__ __forceinline__ int row_stride(int n) {        // floats; an odd number of 16-byte units
  const int s = (n + 3) & ~3;
  return (s >> 2) & 1 ? s : s + 4;
}

template <typename T, int NC>
__global__ void __launch_bounds__(32 * kHG) grouped_attn_kernel(const GroupedAttnArgs a) {
  extern __shared__ __align__(16) float ga_smem[];
  __shared__ float ws[kMaxSplits * kHG];
  const int kst = row_stride(a.dim), vst = (a.vdim + 3) & ~3;
  float* qs = ga_smem;                     // [kHG][kst]
  float* ks = qs + kHG * kst;              // [kTK][kst]
  float* vs = ks + kTK * kst;              // [kTK][vst]
  pdl_wait();
  pdl_launch_dependents();
  const int rep = a.heads / a.kv_heads, groups = (rep + kHG - 1) / kHG;
  const int m = blockIdx.z, split = blockIdx.x, g = blockIdx.y / groups, hg = blockIdx.y % groups;
  const int h0 = g * rep + hg * kHG, nh = min(kHG, rep - hg * kHG);
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const Range r = key_range(a, m, split);
  const int kc = a.cache.k_ld / a.kv_heads, vc = a.cache.v_ld / a.kv_heads;
  for (int i = threadIdx.x; i < kHG * kst; i += 32 * kHG) {
    const int h = i / kst, c = i % kst;
    qs[i] = h < nh && c < a.dim ? a.q_f32[(static_cast<size_t>(m) * a.heads + h0 + h) * a.q_cols + c] * a.scale : 0.f;
  }
  float acc[NC] = {};
  float mx = -INFINITY, l = 0.f;
  for (int kt = r.k0; kt < r.k1; kt += kTK) {
    __syncthreads();
    for (int key = warp; key < kTK; key += kHG) {
      const bool in = kt + key < r.k1 && kt + key >= r.lo;
      const size_t row = in ? cache_row(a.cache, r.seq, kt + key) : 0;
      const T* kp = static_cast<const T*>(a.cache.k) + row * a.cache.k_ld + g * kc;
      const T* vp = static_cast<const T*>(a.cache.v) + row * a.cache.v_ld + g * vc;
      for (int c = lane; c < kst; c += 32) ks[key * kst + c] = in && c < a.dim ? get(kp + c) : 0.f;
      for (int c = lane; c < vst; c += 32) vs[key * vst + c] = in && c < a.vdim ? get(vp + c) : 0.f;
    }
    __syncthreads();
    float s = 0.f, s2 = 0.f;
    const float* q = qs + warp * kst;
    const float* k = ks + lane * kst;
    for (int i = 0; i < ((a.dim + 3) & ~3); i += 4) {
      const float4 x = *reinterpret_cast<const float4*>(q + i), y = *reinterpret_cast<const float4*>(k + i);
      s = fmaf(x.x, y.x, s); s2 = fmaf(x.y, y.y, s2); s = fmaf(x.z, y.z, s); s2 = fmaf(x.w, y.w, s2);
    }
    s = kt + lane < r.k1 && kt + lane >= r.lo ? s + s2 : -INFINITY;
    const float m_new = fmaxf(mx, warp_max(s));                     // -inf: no key of the tile is seen, nor any before
    const float corr = weight_of<false>(mx, m_new), w = weight_of<false>(s, m_new);
    l = l * corr + warp_sum(w);
    mx = m_new;
#pragma unroll
    for (int c = 0; c < NC; ++c) acc[c] *= corr;
    for (int key = 0; key < kTK; ++key) {
      const float wk = __shfl_sync(0xffffffffu, w, key);
#pragma unroll
      for (int c = 0; c < NC; ++c)
        if (c * 32 + lane < a.vdim) acc[c] = fmaf(wk, vs[key * vst + c * 32 + lane], acc[c]);
    }
  }
  if (a.splits == 1) {
    const float inv = l > 0.f ? 1.0f / l : 0.f;
    if (warp < nh) {
      const size_t o = static_cast<size_t>(m) * a.ld_out + (h0 + warp) * a.vdim + lane;
#pragma unroll
      for (int c = 0; c < NC; ++c) {
        if (c * 32 + lane >= a.vdim) continue;
        if (a.out) a.out[o + c * 32] = acc[c] * inv;
        if (a.out_bf16) a.out_bf16[o + c * 32] = __float2bfloat16_rn(acc[c] * inv);
      }
    }
    return;
  }
  if (warp < nh) {
    const size_t base = (static_cast<size_t>(m) * a.heads + h0 + warp) * a.splits + split;
#pragma unroll
    for (int c = 0; c < NC; ++c)
      if (c * 32 + lane < a.vdim) a.part_o[base * a.vdim + c * 32 + lane] = acc[c];
    if (lane == 0) {
      a.part_ml[2 * base] = mx;
      a.part_ml[2 * base + 1] = l;
    }
  }
  finish_heads<false, 32 * kHG>(a, m, h0, nh, a.counters + static_cast<size_t>(m) * gridDim.y + blockIdx.y, ws);
}

// ----------------------------------------------------------------------------------------- tensor cores
constexpr int kWarps = 4;         // warps per block, each with key pieces of its own
constexpr int kHM = 16;           // query heads per block (rows of the MMA)
constexpr int kStages = 3;        // pieces in a warp's ring

__device__ __forceinline__ void cp16(uint32_t dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ void ldsm4(uint32_t* r, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm4t(uint32_t* r, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void mma16816(float* d, const uint32_t* a, const uint32_t* b) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b[0]), "r"(b[1]));
}
__host__ __device__ __forceinline__ int mma_ld(int n) { return (n + 15) / 16 * 16 + 8; }     // an odd number of 16-byte units
size_t mma_smem(int dim, int vdim) {
  return 2u * (kHM * mma_ld(dim) + static_cast<size_t>(kWarps) * kStages * kPiece * (mma_ld(dim) + mma_ld(vdim)));
}

template <int VT>
__global__ void __launch_bounds__(32 * kWarps) grouped_attn_mma_kernel(const GroupedAttnArgs a) {
  extern __shared__ __align__(16) unsigned char gm_smem[];
  __shared__ float ws[kMaxSplits * kWarps];
  __shared__ float2 wml[kWarps][kHM];
  const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int kst = mma_ld(a.dim), vst = mma_ld(a.vdim), kd = kst - 8, vd = vst - 8;
  const int kc = a.cache.k_ld / a.kv_heads, vc = a.cache.v_ld / a.kv_heads;     // cached columns per head, multiples of 8
  __nv_bfloat16* qs = reinterpret_cast<__nv_bfloat16*>(gm_smem);                 // [kHM][kst]
  __nv_bfloat16* ring = qs + kHM * kst + warp * (kStages * kPiece * (kst + vst));   // [kStages][kPiece][kst], then the values
  __nv_bfloat16* vring = ring + kStages * kPiece * kst;
  const int rep = a.heads / a.kv_heads, groups = (rep + kHM - 1) / kHM;
  const int m = blockIdx.z, split = blockIdx.x, g = blockIdx.y / groups, hg = blockIdx.y % groups;
  const int h0 = g * rep + hg * kHM, nh = min(kHM, rep - hg * kHM);
  // columns of a piece that no copy reaches stay zero
  for (int i = lane; i < kStages * kPiece; i += 32) {
    if (kc < kd) *reinterpret_cast<uint4*>(ring + i * kst + kc) = make_uint4(0u, 0u, 0u, 0u);
    if (vc < vd) *reinterpret_cast<uint4*>(vring + i * vst + vc) = make_uint4(0u, 0u, 0u, 0u);
  }
  pdl_wait();
  pdl_launch_dependents();
  const Range r = key_range(a, m, split);
  const int n_pieces = r.k1 > r.k0 ? (r.k1 - r.k0 + kPiece - 1) / kPiece : 0;
  // a lane copies the same 16 bytes of every kper-th key
  const int kv8 = kc >> 3, vv8 = vc >> 3, kper = 32 / kv8, vper = 32 / vv8;
  const int kkey = lane / kv8 < kper ? lane / kv8 : kPiece, vkey = lane / vv8 < vper ? lane / vv8 : kPiece;
  const int kcol = lane % kv8 * 8, vcol = lane % vv8 * 8;
  auto fetch = [&](int piece, int slot) {
    if (piece < n_pieces) {
      const int kt = r.k0 + piece * kPiece, n = r.k1 - kt;   // keys of the piece that exist: the rest is zero
      const size_t row = cache_row(a.cache, r.seq, kt);
      const __nv_bfloat16* ks = static_cast<const __nv_bfloat16*>(a.cache.k) + row * a.cache.k_ld + g * kc + kcol;
      const __nv_bfloat16* vs = static_cast<const __nv_bfloat16*>(a.cache.v) + row * a.cache.v_ld + g * vc + vcol;
      __nv_bfloat16 *kd2 = ring + slot * kPiece * kst + kcol, *vd2 = vring + slot * kPiece * vst + vcol;
      for (int key = kkey; key < kPiece; key += kper) {
        if (key < n) cp16(smem_u32(kd2 + key * kst), ks + key * a.cache.k_ld);
        else *reinterpret_cast<uint4*>(kd2 + key * kst) = make_uint4(0u, 0u, 0u, 0u);
      }
      for (int key = vkey; key < kPiece; key += vper) {
        if (key < n) cp16(smem_u32(vd2 + key * vst), vs + key * a.cache.v_ld);
        else *reinterpret_cast<uint4*>(vd2 + key * vst) = make_uint4(0u, 0u, 0u, 0u);
      }
    }
    cp_commit();                                            // always, so that groups count pieces
  };
#pragma unroll
  for (int i = 0; i < kStages - 1; ++i) fetch(warp + i * kWarps, i);
  for (int i = threadIdx.x; i < kHM * (kd >> 3); i += 32 * kWarps) {
    const int h = i / (kd >> 3), c = i % (kd >> 3) * 8;
    uint4 v = make_uint4(0u, 0u, 0u, 0u);
    if (h < nh && c < a.q_cols) v = *reinterpret_cast<const uint4*>(a.q_bf16 + (static_cast<size_t>(m) * a.heads + h0 + h) * a.q_cols + c);
    *reinterpret_cast<uint4*>(qs + h * kst + c) = v;
  }
  __syncthreads();
  const float c2 = a.scale * 1.4426950408889634f;
  float acc[VT][4] = {};
  float mx[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};    // rows lane / 4 and lane / 4 + 8; l: this lane's columns
  const uint32_t qa = smem_u32(qs) + 2u * ((lane & 15) * kst + (lane >> 4) * 8);
  int slot = 0;
  for (int piece = warp; piece < n_pieces; piece += kWarps) {
    fetch(piece + (kStages - 1) * kWarps, slot == 0 ? kStages - 1 : slot - 1);
    cp_wait<kStages - 1>();
    __syncwarp();
    const uint32_t ka = smem_u32(ring + slot * kPiece * kst) + 2u * (((lane & 7) + ((lane >> 4) & 1) * 8) * kst + ((lane >> 3) & 1) * 8);
    float s[2][4] = {};
    for (int k = 0; k < kd; k += 16) {
      uint32_t af[4], bf[4];
      ldsm4(af, qa + 2u * k);
      ldsm4(bf, ka + 2u * k);
      mma16816(s[0], af, bf);
      mma16816(s[1], af, bf + 2);
    }
    const int key0 = r.k0 + piece * kPiece + (lane & 3) * 2;
    float corr[2];
#pragma unroll
    for (int h = 0; h < 2; ++h) {
      float t = -INFINITY;
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          float& v = s[j][2 * h + e];
          v = key0 + 8 * j + e < r.k1 && key0 + 8 * j + e >= r.lo ? v * c2 : -INFINITY;
          t = fmaxf(t, v);
        }
      t = fmaxf(t, __shfl_xor_sync(0xffffffffu, t, 1));
      t = fmaxf(t, __shfl_xor_sync(0xffffffffu, t, 2));
      const float m_new = fmaxf(mx[h], t), ref = m_new == -INFINITY ? 0.f : m_new;      // -inf: no key is seen so far
      corr[h] = ex2(mx[h] - ref);
      mx[h] = m_new;
      float sum = 0.f;
#pragma unroll
      for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          s[j][2 * h + e] = ex2(s[j][2 * h + e] - ref);
          sum += s[j][2 * h + e];
        }
      l[h] = l[h] * corr[h] + sum;
    }
    const uint32_t pf[4] = {pack_bf16x2(s[0][0], s[0][1]), pack_bf16x2(s[0][2], s[0][3]), pack_bf16x2(s[1][0], s[1][1]), pack_bf16x2(s[1][2], s[1][3])};
    const uint32_t va = smem_u32(vring + slot * kPiece * vst) + 2u * ((lane & 15) * vst + (lane >> 4) * 8);
#pragma unroll
    for (int j = 0; j < VT; j += 2)
      if (j * 8 < vd) {
        uint32_t bf[4];
        ldsm4t(bf, va + 16u * j);
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          acc[j + e][0] *= corr[0];
          acc[j + e][1] *= corr[0];
          acc[j + e][2] *= corr[1];
          acc[j + e][3] *= corr[1];
          mma16816(acc[j + e], pf, bf + 2 * e);
        }
      }
    __syncwarp();                                             // the slot may be fetched over
    slot = slot + 1 == kStages ? 0 : slot + 1;
  }
  cp_wait<0>();
#pragma unroll
  for (int h = 0; h < 2; ++h) {
    l[h] += __shfl_xor_sync(0xffffffffu, l[h], 1);
    l[h] += __shfl_xor_sync(0xffffffffu, l[h], 2);
    if ((lane & 3) == 0) wml[warp][(lane >> 2) + 8 * h] = make_float2(mx[h], l[h]);
  }
  __syncthreads();                                            // the rings are free: they take the warps' outputs
  float* os = reinterpret_cast<float*>(qs + kHM * kst);       // [kWarps][kHM][vd]
#pragma unroll
  for (int j = 0; j < VT; ++j)
    if (j * 8 < vd) {
      float* o = os + (warp * kHM + (lane >> 2)) * vd + j * 8 + (lane & 3) * 2;
      *reinterpret_cast<float2*>(o) = make_float2(acc[j][0], acc[j][1]);
      *reinterpret_cast<float2*>(o + 8 * vd) = make_float2(acc[j][2], acc[j][3]);
    }
  __syncthreads();
  for (int i = threadIdx.x; i < nh * a.vdim; i += 32 * kWarps) {
    const int h = i / a.vdim, c = i % a.vdim;
    float top = -INFINITY, v = 0.f, sum = 0.f;
#pragma unroll
    for (int w = 0; w < kWarps; ++w) top = fmaxf(top, wml[w][h].x);
#pragma unroll
    for (int w = 0; w < kWarps; ++w) {
      const float e = weight_of<true>(wml[w][h].x, top);
      sum = fmaf(e, wml[w][h].y, sum);
      v = fmaf(e, os[(w * kHM + h) * vd + c], v);
    }
    if (a.splits == 1) {
      v = sum > 0.f ? v / sum : 0.f;
      const size_t o = static_cast<size_t>(m) * a.ld_out + (h0 + h) * a.vdim + c;
      if (a.out) a.out[o] = v;
      if (a.out_bf16) a.out_bf16[o] = __float2bfloat16_rn(v);
    } else {
      const size_t base = (static_cast<size_t>(m) * a.heads + h0 + h) * a.splits + split;
      a.part_o[base * a.vdim + c] = v;
      if (c == 0) {
        a.part_ml[2 * base] = top;
        a.part_ml[2 * base + 1] = sum;
      }
    }
  }
  if (a.splits > 1)
    finish_heads<true, 32 * kWarps>(a, m, h0, nh, a.counters + static_cast<size_t>(m) * gridDim.y + blockIdx.y, ws);
}

bool use_mma(const GroupedAttnArgs& a) { return a.q_bf16 && !a.cache.f32 && a.dim <= 256 && a.vdim <= 256; }

template <int VT>
cudaError_t attend_mma(const GroupedAttnArgs& a, cudaStream_t s, bool pdl) {
  static DeviceOnce once;
  const size_t smem = mma_smem(a.dim, a.vdim);
  if (smem > 220 * 1024) return cudaErrorInvalidValue;
  cudaError_t e = once.run([&] {
    return cudaFuncSetAttribute(grouped_attn_mma_kernel<VT>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024);
  });
  if (e != cudaSuccess) return e;
  const int rep = a.heads / a.kv_heads;
  return launch_pdl(grouped_attn_mma_kernel<VT>, dim3(a.splits, a.kv_heads * ((rep + kHM - 1) / kHM), a.M), dim3(32 * kWarps), smem, s, pdl, a);
}

template <typename T, int NC>
cudaError_t attend(const GroupedAttnArgs& a, cudaStream_t s, bool pdl) {
  static DeviceOnce once;
  const size_t smem = sizeof(float) * ((kHG + kTK) * static_cast<size_t>(row_stride(a.dim)) + kTK * static_cast<size_t>((a.vdim + 3) & ~3));
  if (smem > 220 * 1024) return cudaErrorInvalidValue;
  cudaError_t e = once.run([&] {
    return cudaFuncSetAttribute(grouped_attn_kernel<T, NC>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024);
  });
  if (e != cudaSuccess) return e;
  const int rep = a.heads / a.kv_heads;
  return launch_pdl(grouped_attn_kernel<T, NC>, dim3(a.splits, a.kv_heads * ((rep + kHG - 1) / kHG), a.M), dim3(32 * kHG), smem, s, pdl, a);
}

template <typename T>
cudaError_t attend_cols(const GroupedAttnArgs& a, cudaStream_t s, bool pdl) {
  if (a.vdim <= 64) return attend<T, 2>(a, s, pdl);
  if (a.vdim <= 128) return attend<T, 4>(a, s, pdl);
  return attend<T, 16>(a, s, pdl);
}

bool grouped_ok(const GroupedAttnArgs& a) {
  return a.M > 0 && a.heads > 0 && a.kv_heads > 0 && a.heads % a.kv_heads == 0 && a.dim > 0 && a.dim <= kGroupedMaxDim && a.vdim > 0 &&
         a.vdim <= kGroupedMaxDim && a.window > 0 && a.rows.Tc > 0 && a.cache.k_ld % a.kv_heads == 0 && a.cache.v_ld % a.kv_heads == 0 &&
         (a.cache.k_ld / a.kv_heads & 7) == 0 && (a.cache.v_ld / a.kv_heads & 7) == 0 && a.q_cols >= a.dim && (a.q_cols & 7) == 0 &&
         (a.q_bf16 != nullptr) != (a.q_f32 != nullptr);
}

}  // namespace

int grouped_counters(int heads, int kv_heads) { return kv_heads * ((heads / kv_heads + kHG - 1) / kHG); }

int grouped_attn_splits(int M, int heads, int kv_heads, int window) {
  const int groups = M * kv_heads * ((heads / kv_heads + kHM - 1) / kHM);
  const int most = std::max(1, std::min(kMaxSplits, (window + kPageTokens - 1) / kPageTokens));
  // two blocks fit an SM: the fewest ranges whose last wave wastes little, merging counted as one more key in fifty
  int best = 1;
  double cost = 1e30;
  for (int s = 1; s <= most && (s == 1 || static_cast<int64_t>(groups) * s <= kGroupedBlocks); ++s) {
    const double c = ((static_cast<int64_t>(groups) * s + 295) / 296) * (1.0 / s + 0.02);
    if (c < cost * 0.999) {
      cost = c;
      best = s;
    }
  }
  return best;
}

cudaError_t launch_grouped_prep(const GroupedAttnArgs& a, cudaStream_t s, bool pdl) {
  if (!grouped_ok(a)) return cudaErrorInvalidValue;
  if (a.cache.f32) {
    if (a.q_bf16) return cudaErrorInvalidValue;
    return launch_pdl(grouped_prep_kernel<float, float>, dim3(a.M), dim3(kPrepThreads), 0, s, pdl, a);
  }
  return a.q_bf16 ? launch_pdl(grouped_prep_kernel<__nv_bfloat16, __nv_bfloat16>, dim3(a.M), dim3(kPrepThreads), 0, s, pdl, a)
                  : launch_pdl(grouped_prep_kernel<__nv_bfloat16, float>, dim3(a.M), dim3(kPrepThreads), 0, s, pdl, a);
}

cudaError_t launch_grouped_attn(const GroupedAttnArgs& a, cudaStream_t s, bool pdl) {
  if (!grouped_ok(a) || a.splits < 1 || a.splits > kMaxSplits || a.M > 65535) return cudaErrorInvalidValue;
  if (use_mma(a)) return a.vdim <= 64 ? attend_mma<8>(a, s, pdl) : a.vdim <= 128 ? attend_mma<16>(a, s, pdl) : attend_mma<32>(a, s, pdl);
  if (!a.q_f32) return cudaErrorInvalidValue;
  return a.cache.f32 ? attend_cols<float>(a, s, pdl) : attend_cols<__nv_bfloat16>(a, s, pdl);
}

}  // namespace mtj
