// Matrix-state recurrences over long prompts, in chunks of 16 rows on the tensor cores.  With G_i the logarithm of the
// decay from the start of a chunk through its row i, S0 the state in front of the chunk and C its last row:
//   SSD     o_i = e^(G_i) C_i S0 + sum_{j <= i} e^(G_i - G_j) dt_j (C_i . B_j) x_j + D x_i
//           S   = e^(G_C) S0 + sum_j e^(G_C - G_j) dt_j B_j x_j^T
//   delta   u = T (V - K~ S0), T = (I + diag(beta) L)^-1 diag(beta), L_ij = k_i . e^(G_i - G_j) k_j (j < i),  K~_i = e^(G_i) k_i
//           o_i = (e^(G_i) q_i) S0 + sum_{j <= i} (q_i . e^(G_i - G_j) k_j) u_j
//           S   = e^(G_C) S0 + sum_j (e^(G_C - G_j) k_j) u_j^T
// where the delta rule's G is per key channel.  Every decay is the product of per-row factors, none is divided by
// another, so nothing overflows and rows that forget at once are exact.
//
// What does not depend on the state is computed for all chunks at once and left as one record per (chunk, head) in the
// layout the scan reads: delta_prep_kernel (K~, the scaled queries and keys, T, the masked products q.k) and
// ssd_prep_kernel (the masked products C.B and the rows' decays).  In the scans two warps share 16 value columns of a
// head, each keeping the S^T [16, keys / 2] of half the keys in fp32 accumulators, which are at the same time the left
// operands of the next products; they add their partial sums through shared memory, once a chunk.  Records and rows
// come through rings.  Operands that are not exact in bf16 are split into two bf16 numbers (the second the rounding error
// of the first) and multiplied as hi.hi + hi.lo + lo.hi with fp32 accumulation: about 16 mantissa bits, so the state
// keeps its 32-bit character.  (mma.sync: the M dimension is 16 columns of a state that must stay in registers between
// dependent products.)
#include <math.h>

#include <algorithm>

#include "mtj_matrix_state.cuh"

namespace mtj {
namespace {

constexpr int kC = kMatrixChunk;     // rows per chunk
constexpr int kSq = kC + 8;          // row stride of a 16 x 16 matrix, an odd number of 16-byte units
static_assert(kC == 16, "one MMA tile");

__device__ __forceinline__ void ldsm4(uint32_t* r, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm4t(uint32_t* r, uint32_t addr) {
  asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void mma(float* d, const uint32_t* a, const uint32_t* b) {
  asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
               : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
               : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b[0]), "r"(b[1]));
}
// two numbers as packed bf16 pairs: the rounded values and their rounding errors
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pack_bf16x2(x, y);
  lo = pack_bf16x2(x - bf16_lo(hi), y - bf16_hi(hi));
}
// A operand (16 rows, 16 columns of K) from two neighbouring 16 x 8 accumulator tiles
__device__ __forceinline__ void split_a(const float* t0, const float* t1, uint32_t* hi, uint32_t* lo) {
  split2(t0[0], t0[1], hi[0], lo[0]);
  split2(t0[2], t0[3], hi[1], lo[1]);
  split2(t1[0], t1[1], hi[2], lo[2]);
  split2(t1[2], t1[3], hi[3], lo[3]);
}
// lane offsets (elements) into a row-major matrix: as B operand with the rows as N (both 8-row tiles), as A operand or,
// transposed, as B operand with the rows as K
__device__ __forceinline__ int rows_as_n(int lane, int ld) { return ((lane & 7) + ((lane >> 4) & 1) * 8) * ld + ((lane >> 3) & 1) * 8; }
__device__ __forceinline__ int rows_as_m(int lane, int ld) { return (lane & 15) * ld + (lane >> 4) * 8; }

__device__ __forceinline__ void zero_front(const MatrixStateArgs& a, const MsSpan& sp, int i, int head, int c0, int cols, int threads) {
  for (int t = threadIdx.x; t < (a.rows.Tc - sp.n) * cols; t += threads) {
    const int c = c0 + t % cols;
    if (c < a.vdim) a.out[static_cast<size_t>(i * a.rows.Tc + t / cols) * a.ld_out + head * a.vdim + c] = 0.f;
  }
}

// S^T of 16 columns and NT * 8 keys from key0 on: tile n holds keys key0 + 8 n .. + 7
template <int NT>
__device__ __forceinline__ void load_state(const MatrixStateArgs& a, const float* state, int key0, int col, int lane, bool have, float (*S)[4]) {
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int key = key0 + 8 * n + (lane & 3) * 2 + (e & 1), c = col + (lane >> 2) + (e >> 1) * 8;
      S[n][e] = have && key < a.dim && c < a.vdim ? state[static_cast<size_t>(key) * a.vdim + c] : 0.f;
    }
}
template <int NT>
__device__ __forceinline__ void store_state(const MatrixStateArgs& a, float* state, int key0, int col, int lane, const float (*S)[4]) {
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int key = key0 + 8 * n + (lane & 3) * 2 + (e & 1), c = col + (lane >> 2) + (e >> 1) * 8;
      if (key < a.dim && c < a.vdim) state[static_cast<size_t>(key) * a.vdim + c] = S[n][e];
    }
}
// The values of this lane's accumulator places -- rows (lane & 3) * 2 + {0, 1} (+ 8), columns lane / 4 (+ 8) of a chunk --
// as loaded, one chunk ahead.  Rows past the end repeat the last one and columns past the head's the last one: their
// weights are zero, their results are not stored.
struct Values {
  unsigned short r[4][2];            // [columns lane / 4 and + 8 of rows 0 .. 7, then of rows 8 .. 15][row of the pair]
  __device__ __forceinline__ void load(const __nv_bfloat16* v, int ld, int nt, int cols_left, int lane) {
#pragma unroll
    for (int i = 0; i < 4; ++i) {
      const int t = (lane & 3) * 2 + (i >> 1) * 8, c = max(0, min((lane >> 2) + (i & 1) * 8, cols_left - 1));
      const unsigned short* p = reinterpret_cast<const unsigned short*>(v) + c;
      r[i][0] = p[min(t, nt - 1) * ld];
      r[i][1] = p[min(t + 1, nt - 1) * ld];
    }
  }
  __device__ __forceinline__ void pack(uint32_t* out) const {
#pragma unroll
    for (int i = 0; i < 4; ++i) out[i] = r[i][0] | (static_cast<uint32_t>(r[i][1]) << 16);
  }
};
__device__ __forceinline__ void pair_sync(int id) { asm volatile("bar.sync %0, 64;" ::"r"(id) : "memory"); }
// one 8-row tile of outputs
__device__ __forceinline__ void store_tile(float* out, int ld, int t0, int nt, int cols_left, int lane, const float* o) {
#pragma unroll
  for (int e = 0; e < 4; ++e) {
    const int t = t0 + (lane & 3) * 2 + (e & 1), c = (lane >> 2) + (e >> 1) * 8;
    if (t < nt && c < cols_left) out[t * ld + c] = o[e];
  }
}

// ------------------------------------------------------------------------------------------------ delta rule
template <int DP>
struct Record {                      // of one (chunk, head); byte offsets
  static constexpr int LD = DP + 8;
  static constexpr int kMat = kC * LD * 2, kSmall = kC * kSq * 2;
  static constexpr int kKt = 0, kQt = 2 * kMat, kKh = 4 * kMat, kT = 6 * kMat, kM = kT + 2 * kSmall, kE = kM + 2 * kSmall;
  static constexpr int kBytes = kE + DP * 4;          // hi then lo of every matrix; a multiple of 16
};

template <int DP>
struct PrepSmem {
  float k[kC][DP], q[kC][DP], g[kC][DP];
  float L[kC][kC + 4], M[kC][kC + 4];                 // products, rows i, columns j
  float beta[kC];
};

__device__ __forceinline__ float dot4(const float4& x, const float4& y, float s) {
  return fmaf(x.w, y.w, fmaf(x.z, y.z, fmaf(x.y, y.y, fmaf(x.x, y.x, s))));
}

// elements n .. n + 3 of a row, zeros from `have` on
__device__ __forceinline__ float4 four(const float* p, int n, int have, bool vec) {
  if (vec) return n < have ? *reinterpret_cast<const float4*>(p + n) : make_float4(0.f, 0.f, 0.f, 0.f);
  return make_float4(n < have ? p[n] : 0.f, n + 1 < have ? p[n + 1] : 0.f, n + 2 < have ? p[n + 2] : 0.f, n + 3 < have ? p[n + 3] : 0.f);
}
__device__ __forceinline__ float4 four(const __nv_bfloat16* p, int n, int have, bool vec) {
  if (vec) {
    const uint2 w = n < have ? *reinterpret_cast<const uint2*>(p + n) : make_uint2(0u, 0u);
    return make_float4(bf16_lo(w.x), bf16_hi(w.x), bf16_lo(w.y), bf16_hi(w.y));
  }
  return make_float4(n < have ? __bfloat162float(p[n]) : 0.f, n + 1 < have ? __bfloat162float(p[n + 1]) : 0.f,
                     n + 2 < have ? __bfloat162float(p[n + 2]) : 0.f, n + 3 < have ? __bfloat162float(p[n + 3]) : 0.f);
}

// One block of 4 warps per (chunk, head).
template <int DP>
__global__ void __launch_bounds__(128) delta_prep_kernel(const MatrixStateArgs a) {
  using Rec = Record<DP>;
  extern __shared__ __align__(16) unsigned char dp_smem[];
  PrepSmem<DP>& sm = *reinterpret_cast<PrepSmem<DP>*>(dp_smem);
  const int chunk = blockIdx.x, head = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const MsSpan sp = ms_span(a, blockIdx.z);
  const int nt = min(kC, sp.n - chunk * kC);
  if (nt <= 0) return;
  const int kh = head / (a.heads / a.key_heads);
  const float A = a.A[head];
  const __nv_bfloat16* u = static_cast<const __nv_bfloat16*>(a.u);
  // a warp per row, a lane four neighbouring channels
  constexpr int N4 = (DP + 127) / 128;
  const int kcol = a.k0 + kh * a.dim, qcol = a.q0 + kh * a.dim, dcol = head * a.dim;
  const bool vec = ((a.dim | kcol | qcol | a.ld_u | a.ld_decay) & 3) == 0;
  float4 bias[N4];
#pragma unroll
  for (int c = 0; c < N4; ++c) bias[c] = four(a.decay_b + dcol, c * 128 + 4 * lane, a.dim, vec);
#pragma unroll
  for (int i = 0; i < kC / 4; ++i) {
    const int t = warp + 4 * i;
    const size_t m = static_cast<size_t>(sp.row0 + chunk * kC + min(t, nt - 1));
    const __nv_bfloat16* row = u + m * a.ld_u;
    const int have = t < nt ? a.dim : 0;
    float4 kv[N4], qv[N4], gv[N4];
    float ks = 0.f, qs = 0.f;
#pragma unroll
    for (int c = 0; c < N4; ++c) {
      const int n = c * 128 + 4 * lane;
      kv[c] = four(row + kcol, n, have, vec);
      qv[c] = four(row + qcol, n, have, vec);
      gv[c] = four(a.decay + m * a.ld_decay + dcol, n, have, vec);
    }
#pragma unroll
    for (int c = 0; c < N4; ++c) {
      ks = dot4(kv[c], kv[c], ks);
      qs = dot4(qv[c], qv[c], qs);
    }
    const float kr = 1.0f / sqrtf(warp_sum(ks) + kUnitEps), qr = a.q_scale / sqrtf(warp_sum(qs) + kUnitEps);
#pragma unroll
    for (int c = 0; c < N4; ++c) {
      const int n = c * 128 + 4 * lane;
      if (n >= DP) continue;
      auto g = [&](float raw, float b) { return t < nt ? MsFn<__nv_bfloat16>::exp(A * MsFn<__nv_bfloat16>::softplus(raw + b)) : 1.0f; };
      *reinterpret_cast<float4*>(&sm.k[t][n]) = make_float4(kv[c].x * kr, kv[c].y * kr, kv[c].z * kr, kv[c].w * kr);
      *reinterpret_cast<float4*>(&sm.q[t][n]) = make_float4(qv[c].x * qr, qv[c].y * qr, qv[c].z * qr, qv[c].w * qr);
      *reinterpret_cast<float4*>(&sm.g[t][n]) = make_float4(g(gv[c].x, bias[c].x), g(gv[c].y, bias[c].y), g(gv[c].z, bias[c].z), g(gv[c].w, bias[c].w));
    }
    if (lane == 0) sm.beta[t] = t < nt ? MsFn<__nv_bfloat16>::sigmoid(a.beta[m * a.ld_beta + head]) : 0.f;
  }
  __syncthreads();
  // L_ij and M_ij, lanes over the key channels (four neighbours each); a warp takes columns j of a balanced total
  // length and walks the rows in fours, whose eight sums are brought together by a transposing reduction
#pragma unroll 1
  for (int s = 0; s < 4; ++s) {
    const int j = s == 0 ? warp : s == 1 ? 15 - warp : s == 2 ? 4 + warp : 11 - warp;
    float4 d[N4];
#pragma unroll
    for (int c = 0; c < N4; ++c)
      d[c] = c * 128 + 4 * lane < DP ? *reinterpret_cast<const float4*>(&sm.k[j][c * 128 + 4 * lane]) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 1
    for (int i0 = 0; i0 < kC; i0 += 4) {
      float v[8];                                     // L of four rows, then M
#pragma unroll
      for (int r = 0; r < 4; ++r) {
        const int i = i0 + r;
        v[r] = v[4 + r] = 0.f;
        if (i >= j) {
#pragma unroll
          for (int c = 0; c < N4; ++c) {
            const int n = c * 128 + 4 * lane;
            if (n < DP) {
              if (i > j) {
                const float4 g = *reinterpret_cast<const float4*>(&sm.g[i][n]);
                d[c].x *= g.x; d[c].y *= g.y; d[c].z *= g.z; d[c].w *= g.w;
                v[r] = dot4(*reinterpret_cast<const float4*>(&sm.k[i][n]), d[c], v[r]);
              }
              v[4 + r] = dot4(*reinterpret_cast<const float4*>(&sm.q[i][n]), d[c], v[4 + r]);
            }
          }
        }
      }
      if (i0 + 3 >= j) {
#pragma unroll
        for (int w = 4; w > 0; w >>= 1) {             // lane bits 16, 8, 4 pick one of the eight
          const bool up = lane & (4 * w);
#pragma unroll
          for (int r = 0; r < w; ++r) {
            const float send = up ? v[r] : v[r + w], keep = up ? v[r + w] : v[r];
            v[r] = keep + __shfl_xor_sync(0xffffffffu, send, 4 * w);
          }
        }
        v[0] += __shfl_xor_sync(0xffffffffu, v[0], 2);
        v[0] += __shfl_xor_sync(0xffffffffu, v[0], 1);
      }
      if ((lane & 3) == 0) {
        const int which = lane >> 2, i = i0 + (which & 3);
        (which < 4 ? sm.L : sm.M)[i][j] = v[0];       // zero above the diagonal, L zero on it too
      }
    }
  }
  __syncthreads();
  unsigned char* rec = static_cast<unsigned char*>(a.chunk_records) +
                       ((static_cast<size_t>(blockIdx.z) * gridDim.x + chunk) * a.heads + head) * Rec::kBytes;
  auto put2 = [&](int at, int row, int col, float x, float y) {
    uint32_t hi, lo;
    split2(x, y, hi, lo);
    *reinterpret_cast<uint32_t*>(rec + at + (row * kSq + col) * 2) = hi;
    *reinterpret_cast<uint32_t*>(rec + at + Rec::kSmall + (row * kSq + col) * 2) = lo;
  };
  auto put4 = [&](int at, int row, int col, const float4& v) {
    uint2 hi, lo;
    split2(v.x, v.y, hi.x, lo.x);
    split2(v.z, v.w, hi.y, lo.y);
    *reinterpret_cast<uint2*>(rec + at + (row * Rec::LD + col) * 2) = hi;
    *reinterpret_cast<uint2*>(rec + at + Rec::kMat + (row * Rec::LD + col) * 2) = lo;
  };
  if (warp == 3) {
    // T column by column: lane c < 16 solves for column c
    const int c = lane & 15;
    float T[kC];
#pragma unroll
    for (int i = 0; i < kC; ++i) {
      float v = i == c ? 1.0f : 0.f;
#pragma unroll
      for (int j = 0; j < kC; ++j)
        if (j < i) v = fmaf(-sm.L[i][j], T[j], v);
      T[i] = sm.beta[i] * v;
    }
#pragma unroll
    for (int i = 0; i < kC; ++i) {
      const float other = __shfl_down_sync(0xffffffffu, T[i], 1);
      if (lane < 16 && !(lane & 1)) put2(Rec::kT, i, c, T[i], other);
    }
    for (int i = lane; i < kC * kC / 2; i += 32) {
      const int r = i / (kC / 2), cc = i % (kC / 2) * 2;
      put2(Rec::kM, r, cc, sm.M[r][cc], sm.M[r][cc + 1]);
    }
    return;
  }
  // warp 0: K~ and the whole chunk's decay, warp 1: the scaled queries (prefix products), warp 2: the keys for the new
  // state (suffix products)
#pragma unroll
  for (int c = 0; c < N4; ++c) {
    const int n = c * 128 + 4 * lane;
    if (n >= DP) continue;
    float4 p = make_float4(1.f, 1.f, 1.f, 1.f);
    auto times = [&](const float4& x) { return make_float4(x.x * p.x, x.y * p.y, x.z * p.z, x.w * p.w); };
    if (warp < 2) {
#pragma unroll
      for (int i = 0; i < kC; ++i) {
        p = times(*reinterpret_cast<const float4*>(&sm.g[i][n]));
        put4(warp ? Rec::kQt : Rec::kKt, i, n, times(*reinterpret_cast<const float4*>(warp ? &sm.q[i][n] : &sm.k[i][n])));
      }
      if (warp == 0) *reinterpret_cast<float4*>(rec + Rec::kE + n * 4) = p;
    } else {
#pragma unroll
      for (int i = kC - 1; i >= 0; --i) {
        put4(Rec::kKh, i, n, times(*reinterpret_cast<const float4*>(&sm.k[i][n])));
        p = times(*reinterpret_cast<const float4*>(&sm.g[i][n]));
      }
    }
  }
}

__device__ __forceinline__ void bulk_copy(uint32_t dst, const void* src, uint32_t bytes, uint32_t bar) {
  asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
               ::"r"(dst), "l"(src), "r"(bytes), "r"(bar)
               : "memory");
}
__device__ __forceinline__ void arrive(uint32_t bar) { asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(bar) : "memory"); }

constexpr int kRing = 3;

// One block = (head, 16 NG columns, sequence): two scan warps per 16 columns and one that fetches records.
template <int DP, int NG>
__global__ void __launch_bounds__(32 * (2 * NG + 1)) delta_chunk_kernel(const MatrixStateArgs a, int chunks_max) {
  using Rec = Record<DP>;
  constexpr int NW = 2 * NG, NT = DP / 16;               // warps; 8-key tiles per warp
  extern __shared__ __align__(128) unsigned char dc_smem[];
  __shared__ __align__(16) float4 swap[2][NW][3][32];     // partial sums for the partner, two chunks in turn
  __shared__ __align__(8) uint64_t bars[2 * kRing];
  __shared__ uint32_t failed;
  const int head = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const uint32_t full = smem_u32(bars), empty = full + 8 * kRing, base = smem_u32(dc_smem);
  if (threadIdx.x == 0) {
    for (int i = 0; i < kRing; ++i) {
      mbar_init(full + 8 * i, 1);
      mbar_init(empty + 8 * i, NW);
    }
    mbar_fence_init();
    failed = 0;
  }
  __syncthreads();
  const MsSpan sp = ms_span(a, blockIdx.z);
  const int chunks = (sp.n + kC - 1) / kC, c0 = blockIdx.y * 16 * NG;
  if (warp == NW) {
    if (lane == 0) {
      const unsigned char* rec = static_cast<const unsigned char*>(a.chunk_records) +
                                 (static_cast<size_t>(blockIdx.z) * chunks_max * a.heads + head) * Rec::kBytes;
      int issued = 0;
      for (int k = 0; k < chunks; ++k) {
        const int s = k % kRing;
        if (k >= kRing && !mbar_wait(empty + 8 * s, ((k / kRing) - 1) & 1)) {
          atomicOr(&failed, 1u);
          break;
        }
        mbar_expect_tx(full + 8 * s, Rec::kBytes);
        bulk_copy(base + s * Rec::kBytes, rec + static_cast<size_t>(k) * a.heads * Rec::kBytes, Rec::kBytes, full + 8 * s);
        issued = k + 1;
      }
      for (int k = max(0, issued - kRing); k < issued; ++k) mbar_wait(full + 8 * (k % kRing), (k / kRing) & 1);   // no copy outlives the block
    }
  } else {
    const int grp = warp >> 1, half = warp & 1, col = c0 + grp * 16, left = a.vdim - col, key0 = half * (DP / 2);
    float* state = a.state + (static_cast<size_t>(sp.seq) * a.heads + head) * a.dim * a.vdim;
    float S[NT][4];
    load_state<NT>(a, state, key0, col, lane, sp.start > 0 && sp.n > 0, S);
    zero_front(a, sp, blockIdx.z, head, c0, 16 * NG, 32 * NW);
    const __nv_bfloat16* v = static_cast<const __nv_bfloat16*>(a.u) + static_cast<size_t>(sp.row0) * a.ld_u + a.v0 + head * a.vdim + min(col, a.vdim - 1);
    float* out = a.out + static_cast<size_t>(sp.row0) * a.ld_out + head * a.vdim + col;
    Values vals;
    if (chunks > 0) vals.load(v, a.ld_u, min(kC, sp.n), left, lane);
    const int on = (rows_as_n(lane, Rec::LD) + key0) * 2, ot = (rows_as_m(lane, Rec::LD) + key0) * 2, os = rows_as_n(lane, kSq) * 2;
    bool ok = true;                                      // a wait that runs out is remembered; the pair barriers go on
    for (int k = 0; k < chunks; ++k) {
      const int s = k % kRing, nt = min(kC, sp.n - k * kC);
      if (ok) ok = mbar_wait(full + 8 * s, (k / kRing) & 1);
      const uint32_t r = base + s * Rec::kBytes;
      uint32_t cur[4];
      vals.pack(cur);
      if (k + 1 < chunks) vals.load(v + static_cast<size_t>(k + 1) * kC * a.ld_u, a.ld_u, min(kC, sp.n - (k + 1) * kC), left, lane);
      float R[3][2][4] = {}, O[3][2][4] = {};            // the three products of the split operands
#pragma unroll
      for (int ks = 0; ks < NT / 2; ++ks) {
        uint32_t hi[4], lo[4], bh[4], bl[4];
        split_a(S[2 * ks], S[2 * ks + 1], hi, lo);
        ldsm4(bh, r + Rec::kKt + on + 32 * ks);
        ldsm4(bl, r + Rec::kKt + Rec::kMat + on + 32 * ks);
#pragma unroll
        for (int t = 0; t < 2; ++t) {
          mma(R[0][t], hi, bh + 2 * t);
          mma(R[1][t], hi, bl + 2 * t);
          mma(R[2][t], lo, bh + 2 * t);
        }
        ldsm4(bh, r + Rec::kQt + on + 32 * ks);
        ldsm4(bl, r + Rec::kQt + Rec::kMat + on + 32 * ks);
#pragma unroll
        for (int t = 0; t < 2; ++t) {
          mma(O[0][t], hi, bh + 2 * t);
          mma(O[1][t], hi, bl + 2 * t);
          mma(O[2][t], lo, bh + 2 * t);
        }
      }
#pragma unroll
      for (int t = 0; t < 2; ++t)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
          R[0][t][e] += R[1][t][e] + R[2][t][e];
          O[0][t][e] += O[1][t][e] + O[2][t][e];
        }
      // the other half of the keys: both warps need all of R, of the outputs each finishes the tile `half`
      float4* mine = swap[k & 1][warp][0] + lane;
      const float4* theirs = swap[k & 1][warp ^ 1][0] + lane;
      mine[0] = make_float4(R[0][0][0], R[0][0][1], R[0][0][2], R[0][0][3]);
      mine[32] = make_float4(R[0][1][0], R[0][1][1], R[0][1][2], R[0][1][3]);
      mine[64] = half ? make_float4(O[0][0][0], O[0][0][1], O[0][0][2], O[0][0][3]) : make_float4(O[0][1][0], O[0][1][1], O[0][1][2], O[0][1][3]);
      pair_sync(1 + grp);
      uint32_t hi[4], lo[4], bh[4], bl[4];
      const float4 r0 = theirs[0], r1 = theirs[32], po = theirs[64];
      {
        float X[2][4];                                   // V - K~ S0, transposed
        const float rt[2][4] = {{r0.x, r0.y, r0.z, r0.w}, {r1.x, r1.y, r1.z, r1.w}};
#pragma unroll
        for (int t = 0; t < 2; ++t)
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const uint32_t p = cur[2 * t + (e >> 1)];
            X[t][e] = ((e & 1) ? bf16_hi(p) : bf16_lo(p)) - (R[0][t][e] + rt[t][e]);
          }
        split_a(X[0], X[1], hi, lo);
      }
      float U[3][2][4] = {};
      ldsm4(bh, r + Rec::kT + os);
      ldsm4(bl, r + Rec::kT + Rec::kSmall + os);
#pragma unroll
      for (int t = 0; t < 2; ++t) {
        mma(U[0][t], hi, bh + 2 * t);
        mma(U[1][t], hi, bl + 2 * t);
        mma(U[2][t], lo, bh + 2 * t);
      }
#pragma unroll
      for (int t = 0; t < 2; ++t)
#pragma unroll
        for (int e = 0; e < 4; ++e) U[0][t][e] += U[1][t][e] + U[2][t][e];
      split_a(U[0][0], U[0][1], hi, lo);
#pragma unroll
      for (int p = 0; p < NT / 2; ++p) {                 // the new state
        ldsm4t(bh, r + Rec::kKh + ot + 32 * p);
        ldsm4t(bl, r + Rec::kKh + Rec::kMat + ot + 32 * p);
#pragma unroll
        for (int t = 0; t < 2; ++t) {
          float* st = S[2 * p + t];
          float ex, ey;
          asm volatile("ld.shared.v2.f32 {%0, %1}, [%2];" : "=f"(ex), "=f"(ey) : "r"(r + Rec::kE + (key0 + 8 * (2 * p + t) + (lane & 3) * 2) * 4) : "memory");
          st[0] *= ex; st[1] *= ey; st[2] *= ex; st[3] *= ey;
        }
#pragma unroll
        for (int t = 0; t < 2; ++t) {
          mma(S[2 * p + t], hi, bh + 2 * t);
          mma(S[2 * p + t], hi, bl + 2 * t);
          mma(S[2 * p + t], lo, bh + 2 * t);
        }
      }
      ldsm4(bh, r + Rec::kM + os);
      ldsm4(bl, r + Rec::kM + Rec::kSmall + os);
      __syncwarp();
      if (lane == 0) arrive(empty + 8 * s);              // the record is read
      float y[4];
#pragma unroll
      for (int e = 0; e < 4; ++e) y[e] = half ? O[0][1][e] : O[0][0][e];
      y[0] += po.x; y[1] += po.y; y[2] += po.z; y[3] += po.w;
      const uint32_t mh[2] = {half ? bh[2] : bh[0], half ? bh[3] : bh[1]}, ml[2] = {half ? bl[2] : bl[0], half ? bl[3] : bl[1]};
      mma(y, hi, mh);
      mma(y, hi, ml);
      mma(y, lo, mh);
      store_tile(out + static_cast<size_t>(k) * kC * a.ld_out, a.ld_out, half * 8, nt, left, lane, y);
    }
    if (!ok) atomicOr(&failed, 1u);
    if (sp.n > 0 && __all_sync(0xffffffffu, ok)) store_state<NT>(a, state, key0, col, lane, S);
  }
  __syncthreads();
  if (threadIdx.x == 0 && failed && a.dev_err) atomicOr(a.dev_err, kDevErrTimeout);
}

// ------------------------------------------------------------------------------------------------------ SSD
__device__ __forceinline__ void cp16(uint32_t dst, const void* src) {
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

struct SsdRecord {                   // of one (chunk, head); byte offsets
  static constexpr int kSmall = kC * kSq * 2;          // masked products [i][j], hi then lo
  static constexpr int kG = 2 * kSmall;                // floats: e^(G_i) [16], e^(G_C - G_j) dt_j [16], e^(G_C)
  static constexpr int kBytes = kG + 4 * 36;
};
template <int DP>
struct SsdTiles {                    // of one (chunk, key head): B then C, zero-padded; they follow all head records
  static constexpr int LD = DP + 8, kMat = kC * LD * 2, kBytes = 2 * kMat;
};
static_assert(SsdRecord::kBytes % 16 == 0, "whole pieces");

// 16 rows of `dim` columns -> [kC][LD] in shared memory by `threads` threads; rows from nt on are zero
__device__ __forceinline__ void fetch_rows(__nv_bfloat16* dst, int LD, const __nv_bfloat16* src, int ld, int dim, int nt, bool vec, int t, int threads) {
  if (vec) {
    const int per = dim >> 3;
    for (int i = t; i < kC * per; i += threads) {
      const int row = i / per, c = i % per * 8;
      __nv_bfloat16* d = dst + row * LD + c;
      if (row < nt) cp16(smem_u32(d), src + static_cast<size_t>(row) * ld + c);
      else *reinterpret_cast<uint4*>(d) = make_uint4(0u, 0u, 0u, 0u);
    }
  } else {
    for (int i = t; i < kC * dim; i += threads) {
      const int row = i / dim, c = i % dim;
      dst[row * LD + c] = row < nt ? src[static_cast<size_t>(row) * ld + c] : __float2bfloat16_rn(0.f);
    }
  }
}

// One block of 4 warps per (chunk, key head): C B^T once, then the records of the heads that share it.
template <int DP>
__global__ void __launch_bounds__(128) ssd_prep_kernel(const MatrixStateArgs a) {
  constexpr int LD = DP + 8;
  __shared__ __align__(16) __nv_bfloat16 tile[2][kC * LD];           // B, C
  const int chunk = blockIdx.x, kh = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const MsSpan sp = ms_span(a, blockIdx.z);
  const int nt = min(kC, sp.n - chunk * kC);
  if (nt <= 0) return;
  const size_t row0 = static_cast<size_t>(sp.row0 + chunk * kC);
  const __nv_bfloat16* u = static_cast<const __nv_bfloat16*>(a.u) + row0 * a.ld_u;
  const int kb = a.k0 + kh * a.dim, qb = a.q0 + kh * a.dim, rep = a.heads / a.key_heads;
  const bool vec = ((a.dim | kb | qb | a.ld_u) & 7) == 0;
  if (a.dim < DP)
    for (int i = threadIdx.x; i < 2 * kC * LD / 8; i += 128) reinterpret_cast<uint4*>(tile[0])[i] = make_uint4(0u, 0u, 0u, 0u);
  __syncthreads();
  fetch_rows(tile[0], LD, u + kb, a.ld_u, a.dim, nt, vec, threadIdx.x, 128);
  fetch_rows(tile[1], LD, u + qb, a.ld_u, a.dim, nt, vec, threadIdx.x, 128);
  cp_commit();
  cp_wait<0>();
  __syncthreads();
  unsigned char* tiles = static_cast<unsigned char*>(a.chunk_records) + static_cast<size_t>(gridDim.z) * gridDim.x * a.heads * SsdRecord::kBytes +
                         ((static_cast<size_t>(blockIdx.z) * gridDim.x + chunk) * a.key_heads + kh) * SsdTiles<DP>::kBytes;
  for (int i = threadIdx.x; i < SsdTiles<DP>::kBytes / 16; i += 128) reinterpret_cast<uint4*>(tiles)[i] = reinterpret_cast<const uint4*>(tile[0])[i];
  float P[2][4] = {};                                    // C B^T [i, j]
  const uint32_t rb = smem_u32(tile[0]) + rows_as_n(lane, LD) * 2, rc = smem_u32(tile[1]) + rows_as_m(lane, LD) * 2;
#pragma unroll
  for (int ks = 0; ks < DP / 16; ++ks) {
    uint32_t ca[4], bn[4];
    ldsm4(ca, rc + 32 * ks);
    ldsm4(bn, rb + 32 * ks);
    mma(P[0], ca, bn);
    mma(P[1], ca, bn + 2);
  }
  for (int head = kh * rep + warp; head < (kh + 1) * rep; head += 4) {
    const int t = lane & 15;
    const float dt = t < nt ? MsFn<__nv_bfloat16>::softplus(a.decay[(row0 + t) * a.ld_decay + head] + a.decay_b[head]) : 0.f;
    float G = a.A[head] * dt;                            // running sum over the chunk's rows, lane = row
#pragma unroll
    for (int o = 1; o < 16; o <<= 1) {
      const float up = __shfl_up_sync(0xffffffffu, G, o, 16);
      if (t >= o) G += up;
    }
    const float last = __shfl_sync(0xffffffffu, G, 15);
    unsigned char* rec = static_cast<unsigned char*>(a.chunk_records) +
                         ((static_cast<size_t>(blockIdx.z) * gridDim.x + chunk) * a.heads + head) * SsdRecord::kBytes;
    float* fl = reinterpret_cast<float*>(rec + SsdRecord::kG);
    if (lane < 16) {
      fl[t] = __expf(G);
      fl[16 + t] = __expf(last - G) * dt;
      if (t == 0) fl[32] = __expf(last);
    }
    float Gj[4], dj[4];                                  // rows j = (lane & 3) * 2 + {0, 1} (+ 8)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int j = (lane & 3) * 2 + (e & 1) + (e >> 1) * 8;
      Gj[e] = __shfl_sync(0xffffffffu, G, j);
      dj[e] = __shfl_sync(0xffffffffu, dt, j);
    }
#pragma unroll
    for (int i8 = 0; i8 < 2; ++i8) {
      const int i = (lane >> 2) + 8 * i8;
      const float Gi = __shfl_sync(0xffffffffu, G, i);
#pragma unroll
      for (int j8 = 0; j8 < 2; ++j8) {
        float w[2];
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int j = (lane & 3) * 2 + e + 8 * j8;
          w[e] = j <= i ? P[j8][2 * i8 + e] * __expf(Gi - Gj[2 * j8 + e]) * dj[2 * j8 + e] : 0.f;
        }
        uint32_t hi, lo;
        split2(w[0], w[1], hi, lo);
        const int at = (i * kSq + (lane & 3) * 2 + 8 * j8) * 2;
        *reinterpret_cast<uint32_t*>(rec + at) = hi;
        *reinterpret_cast<uint32_t*>(rec + SsdRecord::kSmall + at) = lo;
      }
    }
  }
}

// One block = (head, 16 NG columns, sequence): two scan warps per 16 columns and one that fetches tiles and records.
template <int DP, int NG>
__global__ void __launch_bounds__(32 * (2 * NG + 1)) ssd_chunk_kernel(const MatrixStateArgs a, int chunks_max) {
  using Tiles = SsdTiles<DP>;
  constexpr int LD = Tiles::LD, NW = 2 * NG, NT = DP / 16, kStages = 4, kStage = Tiles::kBytes + SsdRecord::kBytes;
  extern __shared__ __align__(128) unsigned char sd_smem[];
  __shared__ __align__(16) float4 swap[2][NW][32];
  __shared__ __align__(8) uint64_t bars[2 * kStages];
  __shared__ uint32_t failed;
  const int head = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const uint32_t full = smem_u32(bars), empty = full + 8 * kStages, base = smem_u32(sd_smem);
  if (threadIdx.x == 0) {
    for (int i = 0; i < kStages; ++i) {
      mbar_init(full + 8 * i, 1);
      mbar_init(empty + 8 * i, NW);
    }
    mbar_fence_init();
    failed = 0;
  }
  __syncthreads();
  const MsSpan sp = ms_span(a, blockIdx.z);
  const int chunks = (sp.n + kC - 1) / kC, c0 = blockIdx.y * 16 * NG;
  if (warp == NW) {
    if (lane == 0) {
      const unsigned char* rec = static_cast<const unsigned char*>(a.chunk_records);
      const unsigned char* tiles = rec + static_cast<size_t>(gridDim.z) * chunks_max * a.heads * SsdRecord::kBytes +
                                   (static_cast<size_t>(blockIdx.z) * chunks_max * a.key_heads + head / (a.heads / a.key_heads)) * Tiles::kBytes;
      rec += (static_cast<size_t>(blockIdx.z) * chunks_max * a.heads + head) * SsdRecord::kBytes;
      int issued = 0;
      for (int k = 0; k < chunks; ++k) {
        const int s = k % kStages;
        if (k >= kStages && !mbar_wait(empty + 8 * s, ((k / kStages) - 1) & 1)) {
          atomicOr(&failed, 1u);
          break;
        }
        mbar_expect_tx(full + 8 * s, kStage);
        bulk_copy(base + s * kStage, tiles + static_cast<size_t>(k) * a.key_heads * Tiles::kBytes, Tiles::kBytes, full + 8 * s);
        bulk_copy(base + s * kStage + Tiles::kBytes, rec + static_cast<size_t>(k) * a.heads * SsdRecord::kBytes, SsdRecord::kBytes, full + 8 * s);
        issued = k + 1;
      }
      for (int k = max(0, issued - kStages); k < issued; ++k) mbar_wait(full + 8 * (k % kStages), (k / kStages) & 1);   // no copy outlives the block
    }
  } else {
    const int grp = warp >> 1, half = warp & 1, key0 = half * (DP / 2), col = c0 + grp * 16, left = a.vdim - col;
    const __nv_bfloat16* u = static_cast<const __nv_bfloat16*>(a.u) + static_cast<size_t>(sp.row0) * a.ld_u;
    const float D = a.D[head];
    float* state = a.state + (static_cast<size_t>(sp.seq) * a.heads + head) * a.dim * a.vdim;
    float S[NT][4];
    load_state<NT>(a, state, key0, col, lane, sp.start > 0 && sp.n > 0, S);
    zero_front(a, sp, blockIdx.z, head, c0, 16 * NG, 32 * NW);
    const __nv_bfloat16* v = u + a.v0 + head * a.vdim + min(col, a.vdim - 1);
    float* out = a.out + static_cast<size_t>(sp.row0) * a.ld_out + head * a.vdim + col;
    Values vals;
    if (chunks > 0) vals.load(v, a.ld_u, min(kC, sp.n), left, lane);
    const int on = (rows_as_n(lane, LD) + key0) * 2, om = (rows_as_m(lane, LD) + key0) * 2, os = rows_as_n(lane, kSq) * 2;
    bool ok = true;                                        // a wait that runs out is remembered; the pair barriers go on
    for (int k = 0; k < chunks; ++k) {
      const int s = k % kStages, nt = min(kC, sp.n - k * kC);
      if (ok) ok = mbar_wait(full + 8 * s, (k / kStages) & 1);
      const uint32_t rb = base + s * kStage, rc = rb + Tiles::kMat, rr = rb + Tiles::kBytes;
      const float* fl = reinterpret_cast<const float*>(sd_smem + s * kStage + Tiles::kBytes + SsdRecord::kG);
      uint32_t x[4];
      vals.pack(x);
      if (k + 1 < chunks) vals.load(v + static_cast<size_t>(k + 1) * kC * a.ld_u, a.ld_u, min(kC, sp.n - (k + 1) * kC), left, lane);
      float O[2][2][4] = {};                               // S0^T C^T by the split of S0
#pragma unroll
      for (int ks = 0; ks < NT / 2; ++ks) {
        uint32_t hi[4], lo[4], cn[4];
        split_a(S[2 * ks], S[2 * ks + 1], hi, lo);
        ldsm4(cn, rc + on + 32 * ks);
#pragma unroll
        for (int t = 0; t < 2; ++t) {
          mma(O[0][t], hi, cn + 2 * t);
          mma(O[1][t], lo, cn + 2 * t);
        }
      }
#pragma unroll
      for (int t = 0; t < 2; ++t)
#pragma unroll
        for (int e = 0; e < 4; ++e) O[0][t][e] += O[1][t][e];
      // of the outputs this warp finishes the tile `half`; the partner gets the partial sums of the other
      swap[k & 1][warp][lane] = half ? make_float4(O[0][0][0], O[0][0][1], O[0][0][2], O[0][0][3])
                                     : make_float4(O[0][1][0], O[0][1][1], O[0][1][2], O[0][1][3]);
      uint32_t uh[4], ul[4];
#pragma unroll
      for (int t = 0; t < 2; ++t) {
        const float2 f = *reinterpret_cast<const float2*>(fl + 16 + 8 * t + (lane & 3) * 2);
#pragma unroll
        for (int h = 0; h < 2; ++h) split2(bf16_lo(x[2 * t + h]) * f.x, bf16_hi(x[2 * t + h]) * f.y, uh[2 * t + h], ul[2 * t + h]);
      }
      const float el = fl[32];
#pragma unroll
      for (int n = 0; n < NT; ++n) {
        S[n][0] *= el; S[n][1] *= el; S[n][2] *= el; S[n][3] *= el;
      }
#pragma unroll
      for (int p = 0; p < NT / 2; ++p) {
        uint32_t b[4];
        ldsm4t(b, rb + om + 32 * p);
#pragma unroll
        for (int t = 0; t < 2; ++t) {
          mma(S[2 * p + t], uh, b + 2 * t);
          mma(S[2 * p + t], ul, b + 2 * t);
        }
      }
      uint32_t mh[4], ml[4];
      ldsm4(mh, rr + os);
      ldsm4(ml, rr + SsdRecord::kSmall + os);
      const float2 eg = *reinterpret_cast<const float2*>(fl + 8 * half + (lane & 3) * 2);
      __syncwarp();
      if (lane == 0) arrive(empty + 8 * s);                // the stage is read
      pair_sync(1 + grp);
      const float4 po = swap[k & 1][warp ^ 1][lane];
      const uint32_t x0 = half ? x[2] : x[0], x1 = half ? x[3] : x[1];
      float y[4];
      y[0] = fmaf(D, bf16_lo(x0), ((half ? O[0][1][0] : O[0][0][0]) + po.x) * eg.x);
      y[1] = fmaf(D, bf16_hi(x0), ((half ? O[0][1][1] : O[0][0][1]) + po.y) * eg.y);
      y[2] = fmaf(D, bf16_lo(x1), ((half ? O[0][1][2] : O[0][0][2]) + po.z) * eg.x);
      y[3] = fmaf(D, bf16_hi(x1), ((half ? O[0][1][3] : O[0][0][3]) + po.w) * eg.y);
      const uint32_t th[2] = {half ? mh[2] : mh[0], half ? mh[3] : mh[1]}, tl[2] = {half ? ml[2] : ml[0], half ? ml[3] : ml[1]};
      mma(y, x, th);
      mma(y, x, tl);
      store_tile(out + static_cast<size_t>(k) * kC * a.ld_out, a.ld_out, half * 8, nt, left, lane, y);
    }
    if (!ok) atomicOr(&failed, 1u);
    if (sp.n > 0 && __all_sync(0xffffffffu, ok)) store_state<NT>(a, state, key0, col, lane, S);
  }
  __syncthreads();
  if (threadIdx.x == 0 && failed && a.dev_err) atomicOr(a.dev_err, kDevErrTimeout);
}

template <typename K>
cudaError_t allow_smem(DeviceOnce& once, K kernel, int bytes) {
  return once.run([&] { return cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes); });
}

template <int DP, int NG>
cudaError_t delta_cols(const MatrixStateArgs& a, int chunks, cudaStream_t s) {
  constexpr int smem = kRing * Record<DP>::kBytes;
  static_assert(smem <= 200 * 1024 && Record<DP>::kBytes % 16 == 0, "shared memory");
  static DeviceOnce once;
  cudaError_t e = allow_smem(once, delta_chunk_kernel<DP, NG>, smem);
  if (e != cudaSuccess) return e;
  delta_chunk_kernel<DP, NG><<<dim3(a.heads, (a.vdim + 16 * NG - 1) / (16 * NG), a.nseq), 32 * (2 * NG + 1), smem, s>>>(a, chunks);
  return cudaGetLastError();
}

template <int DP>
cudaError_t delta(const MatrixStateArgs& a, cudaStream_t s) {
  constexpr int prep = static_cast<int>(sizeof(PrepSmem<DP>));
  static DeviceOnce once;
  cudaError_t e = allow_smem(once, delta_prep_kernel<DP>, prep);
  if (e != cudaSuccess) return e;
  const int chunks = (a.rows.Tc + kC - 1) / kC;
  delta_prep_kernel<DP><<<dim3(chunks, a.heads, a.nseq), 128, prep, s>>>(a);
  e = cudaGetLastError();
  if (e != cudaSuccess) return e;
  // as few columns per block as still give every SM a block
  const int64_t cols = static_cast<int64_t>(a.heads) * a.nseq * ((a.vdim + 15) / 16);
  return cols <= 148 * 2 ? delta_cols<DP, 2>(a, chunks, s) : delta_cols<DP, 4>(a, chunks, s);
}

template <int DP, int NG>
cudaError_t ssd_cols(const MatrixStateArgs& a, int chunks, cudaStream_t s) {
  constexpr int smem = 4 * (SsdTiles<DP>::kBytes + SsdRecord::kBytes);
  static_assert(smem <= 200 * 1024 && SsdTiles<DP>::kBytes % 16 == 0, "shared memory");
  static DeviceOnce once;
  cudaError_t e = allow_smem(once, ssd_chunk_kernel<DP, NG>, smem);
  if (e != cudaSuccess) return e;
  ssd_chunk_kernel<DP, NG><<<dim3(a.heads, (a.vdim + 16 * NG - 1) / (16 * NG), a.nseq), 32 * (2 * NG + 1), smem, s>>>(a, chunks);
  return cudaGetLastError();
}

template <int DP>
cudaError_t ssd(const MatrixStateArgs& a, cudaStream_t s) {
  const int chunks = (a.rows.Tc + kC - 1) / kC;
  ssd_prep_kernel<DP><<<dim3(chunks, a.key_heads, a.nseq), 128, 0, s>>>(a);
  const cudaError_t e = cudaGetLastError();
  if (e != cudaSuccess) return e;
  const int64_t cols = static_cast<int64_t>(a.heads) * a.nseq * ((a.vdim + 15) / 16);
  return cols <= 148 * 2 ? ssd_cols<DP, 2>(a, chunks, s) : ssd_cols<DP, 4>(a, chunks, s);
}

}  // namespace

int64_t matrix_chunk_bytes(int heads, int key_heads, int dim, int delta) {
  const int64_t h = heads, g = key_heads;
  if (delta) return h * (dim <= 32 ? Record<32>::kBytes : dim <= 64 ? Record<64>::kBytes : dim <= 128 ? Record<128>::kBytes : Record<256>::kBytes);
  return h * SsdRecord::kBytes + g * (dim <= 32 ? SsdTiles<32>::kBytes : dim <= 64 ? SsdTiles<64>::kBytes : dim <= 128 ? SsdTiles<128>::kBytes : SsdTiles<256>::kBytes);
}

cudaError_t launch_matrix_chunks(const MatrixStateArgs& a, cudaStream_t s) {
  if (!matrix_state_ok(a) || !a.u_bf16 || a.nseq > 65535 || a.heads > 65535) return cudaErrorInvalidValue;
  if (!a.chunk_records || (reinterpret_cast<uintptr_t>(a.chunk_records) & 15)) return cudaErrorInvalidValue;
  if (a.delta) return a.dim <= 32 ? delta<32>(a, s) : a.dim <= 64 ? delta<64>(a, s) : a.dim <= 128 ? delta<128>(a, s) : delta<256>(a, s);
  return a.dim <= 32 ? ssd<32>(a, s) : a.dim <= 64 ? ssd<64>(a, s) : a.dim <= 128 ? ssd<128>(a, s) : ssd<256>(a, s);
}

}  // namespace mtj
