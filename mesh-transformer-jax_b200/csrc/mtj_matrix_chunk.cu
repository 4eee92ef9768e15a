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
// What does not depend on the state (delta: K~, the scaled queries and keys, T, the masked products) is computed for
// all chunks at once by delta_prep_kernel and left as one record per (chunk, head) in the layout the scan reads.  In
// the scan a warp owns 16 value columns of a head and keeps its S^T [16, keys] in fp32 accumulators, which are at the
// same time the left operands of the next products; records come by bulk copies through a ring.  Operands that are not
// exact in bf16 are split into two bf16 numbers (the second the rounding error of the first) and multiplied as hi.hi +
// hi.lo + lo.hi with fp32 accumulation: about 16 mantissa bits, so the state keeps its 32-bit character.
// (mma.sync: the M dimension is 16 columns of a state that must stay in registers between dependent products.)
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

// S^T of 16 columns: tile n holds keys 8 n .. 8 n + 7
template <int DP>
__device__ __forceinline__ void load_state(const MatrixStateArgs& a, const float* state, int col, int lane, bool have, float (*S)[4]) {
#pragma unroll
  for (int n = 0; n < DP / 8; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int key = 8 * n + (lane & 3) * 2 + (e & 1), c = col + (lane >> 2) + (e >> 1) * 8;
      S[n][e] = have && key < a.dim && c < a.vdim ? state[static_cast<size_t>(key) * a.vdim + c] : 0.f;
    }
}
template <int DP>
__device__ __forceinline__ void store_state(const MatrixStateArgs& a, float* state, int col, int lane, const float (*S)[4]) {
#pragma unroll
  for (int n = 0; n < DP / 8; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int key = 8 * n + (lane & 3) * 2 + (e & 1), c = col + (lane >> 2) + (e >> 1) * 8;
      if (key < a.dim && c < a.vdim) state[static_cast<size_t>(key) * a.vdim + c] = S[n][e];
    }
}
// The values of this lane's accumulator places: rows (lane & 3) * 2 + {0, 1} (+ 8), columns lane / 4 (+ 8) of a chunk, as
// packed bf16 pairs of neighbouring rows: v[0], v[1] = columns lane / 4 and + 8 of rows 0 .. 7, v[2], v[3] of rows 8 .. 15.
__device__ __forceinline__ void load_values(const __nv_bfloat16* v, int ld, int nt, int cols_left, int lane, uint32_t* out) {
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int t = (lane & 3) * 2 + (i >> 1) * 8, c = (lane >> 2) + (i & 1) * 8;
    const unsigned short* p = reinterpret_cast<const unsigned short*>(v) + static_cast<size_t>(t) * ld + c;
    const uint32_t x = c < cols_left && t < nt ? *p : 0u, y = c < cols_left && t + 1 < nt ? p[ld] : 0u;
    out[i] = x | (y << 16);
  }
}
__device__ __forceinline__ void store_outputs(float* out, int ld, int nt, int cols_left, int lane, const float (*o)[4]) {
#pragma unroll
  for (int t8 = 0; t8 < 2; ++t8)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int t = (lane & 3) * 2 + (e & 1) + t8 * 8, c = (lane >> 2) + (e >> 1) * 8;
      if (t < nt && c < cols_left) out[static_cast<size_t>(t) * ld + c] = o[t8][e];
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
  float k[kC][DP + 1], q[kC][DP + 1], g[kC][DP + 1];
  float L[kC][kC + 4], M[kC][kC + 4];                 // products, rows i, columns j
  float beta[kC];
};

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
  constexpr int NC = DP / 32;
#pragma unroll
  for (int i = 0; i < kC / 4; ++i) {                  // a warp per row
    const int t = warp + 4 * i;
    const size_t m = static_cast<size_t>(sp.row0 + chunk * kC + min(t, nt - 1));
    const __nv_bfloat16* row = u + m * a.ld_u;
    float kv[NC], qv[NC], gv[NC], ks = 0.f, qs = 0.f;
#pragma unroll
    for (int c = 0; c < NC; ++c) {
      const int n = c * 32 + lane;
      const bool in = t < nt && n < a.dim;
      kv[c] = in ? __bfloat162float(row[a.k0 + kh * a.dim + n]) : 0.f;
      qv[c] = in ? __bfloat162float(row[a.q0 + kh * a.dim + n]) : 0.f;
      gv[c] = in ? a.decay[m * a.ld_decay + head * a.dim + n] + a.decay_b[head * a.dim + n] : 0.f;
    }
#pragma unroll
    for (int c = 0; c < NC; ++c) {
      ks = fmaf(kv[c], kv[c], ks);
      qs = fmaf(qv[c], qv[c], qs);
    }
    const float kr = 1.0f / sqrtf(warp_sum(ks) + kUnitEps), qr = a.q_scale / sqrtf(warp_sum(qs) + kUnitEps);
#pragma unroll
    for (int c = 0; c < NC; ++c) {
      const int n = c * 32 + lane;
      sm.k[t][n] = kv[c] * kr;
      sm.q[t][n] = qv[c] * qr;
      sm.g[t][n] = t < nt ? MsFn<__nv_bfloat16>::exp(A * MsFn<__nv_bfloat16>::softplus(gv[c])) : 1.0f;
    }
    if (lane == 0) sm.beta[t] = t < nt ? MsFn<__nv_bfloat16>::sigmoid(a.beta[m * a.ld_beta + head]) : 0.f;
  }
  for (int i = threadIdx.x; i < kC * kC; i += 128) {
    if (i / kC < i % kC) sm.M[i / kC][i % kC] = 0.f;
    if (i / kC <= i % kC) sm.L[i / kC][i % kC] = 0.f;
  }
  __syncthreads();
  // L_ij and M_ij for i = j .. 15, lanes over the key channels; a warp takes columns j of a balanced total length
#pragma unroll 1
  for (int s = 0; s < 4; ++s) {
    const int j = s == 0 ? warp : s == 1 ? 15 - warp : s == 2 ? 4 + warp : 11 - warp;
    float d[NC], mine_l = 0.f, mine_m = 0.f;
#pragma unroll
    for (int c = 0; c < NC; ++c) d[c] = sm.k[j][c * 32 + lane];
#pragma unroll 2
    for (int i = j; i < kC; ++i) {
      float l = 0.f, m = 0.f;
#pragma unroll
      for (int c = 0; c < NC; ++c) {
        const int n = c * 32 + lane;
        if (i > j) d[c] *= sm.g[i][n];
        l = fmaf(sm.k[i][n], d[c], l);
        m = fmaf(sm.q[i][n], d[c], m);
      }
      // both sums at once: the lower half of the warp goes on with l, the upper with m
      const float send = lane < 16 ? m : l, keep = lane < 16 ? l : m;
      float v = keep + __shfl_xor_sync(0xffffffffu, send, 16);
#pragma unroll
      for (int o = 8; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
      if ((lane & 15) == i) mine_l = v;               // lane i keeps l, lane 16 + i keeps m
    }
    mine_m = __shfl_down_sync(0xffffffffu, mine_l, 16);
    if (lane < 16 && lane >= j) {
      if (lane > j) sm.L[lane][j] = mine_l;
      sm.M[lane][j] = mine_m;
    }
  }
  __syncthreads();
  unsigned char* rec = static_cast<unsigned char*>(a.chunk_records) +
                       ((static_cast<size_t>(blockIdx.z) * gridDim.x + chunk) * a.heads + head) * Rec::kBytes;
  auto put = [&](int at, int bytes, int row, int ld, int col, float x, float y) {
    uint32_t hi, lo;
    split2(x, y, hi, lo);
    *reinterpret_cast<uint32_t*>(rec + at + (row * ld + col) * 2) = hi;
    *reinterpret_cast<uint32_t*>(rec + at + bytes + (row * ld + col) * 2) = lo;
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
      if (lane < 16 && !(lane & 1)) put(Rec::kT, Rec::kSmall, i, kSq, c, T[i], other);
    }
    for (int i = lane; i < kC * kC / 2; i += 32) {
      const int r = i / (kC / 2), cc = i % (kC / 2) * 2;
      put(Rec::kM, Rec::kSmall, r, kSq, cc, sm.M[r][cc], sm.M[r][cc + 1]);
    }
  }
  // scaled keys and queries: jobs of two neighbouring channels, prefix products (K~, Q~, the whole chunk's decay) or
  // suffix products (keys for the new state)
  for (int job = threadIdx.x; job < DP; job += 128) {
    const int n = job % (DP / 2) * 2;
    float px = 1.0f, py = 1.0f;
    if (job < DP / 2) {
#pragma unroll
      for (int i = 0; i < kC; ++i) {
        px *= sm.g[i][n];
        py *= sm.g[i][n + 1];
        put(Rec::kKt, Rec::kMat, i, Rec::LD, n, sm.k[i][n] * px, sm.k[i][n + 1] * py);
        put(Rec::kQt, Rec::kMat, i, Rec::LD, n, sm.q[i][n] * px, sm.q[i][n + 1] * py);
      }
      *reinterpret_cast<float2*>(rec + Rec::kE + n * 4) = make_float2(px, py);
    } else {
#pragma unroll
      for (int i = kC - 1; i >= 0; --i) {
        put(Rec::kKh, Rec::kMat, i, Rec::LD, n, sm.k[i][n] * px, sm.k[i][n + 1] * py);
        px *= sm.g[i][n];
        py *= sm.g[i][n + 1];
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

// One block = (head, 16 NW columns, sequence): NW scan warps and one that fetches records.
template <int DP, int NW>
__global__ void __launch_bounds__(32 * (NW + 1)) delta_chunk_kernel(const MatrixStateArgs a, int chunks_max) {
  using Rec = Record<DP>;
  extern __shared__ __align__(128) unsigned char dc_smem[];
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
  const int chunks = (sp.n + kC - 1) / kC, c0 = blockIdx.y * 16 * NW;
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
    const int col = c0 + warp * 16, left = a.vdim - col;
    float* state = a.state + (static_cast<size_t>(sp.seq) * a.heads + head) * a.dim * a.vdim;
    float S[DP / 8][4];
    load_state<DP>(a, state, col, lane, sp.start > 0 && sp.n > 0, S);
    zero_front(a, sp, blockIdx.z, head, c0, 16 * NW, 32 * NW);
    const __nv_bfloat16* v = static_cast<const __nv_bfloat16*>(a.u) + static_cast<size_t>(sp.row0) * a.ld_u + a.v0 + head * a.vdim + col;
    float* out = a.out + static_cast<size_t>(sp.row0) * a.ld_out + head * a.vdim + col;
    uint32_t vals[4] = {0u, 0u, 0u, 0u};
    if (chunks > 0) load_values(v, a.ld_u, min(kC, sp.n), left, lane, vals);
    const int on = rows_as_n(lane, Rec::LD) * 2, ot = rows_as_m(lane, Rec::LD) * 2, os = rows_as_n(lane, kSq) * 2;
    bool ok = true;
    for (int k = 0; k < chunks && ok; ++k) {
      const int s = k % kRing, nt = min(kC, sp.n - k * kC);
      ok = mbar_wait(full + 8 * s, (k / kRing) & 1);
      ok = __all_sync(0xffffffffu, ok);
      if (!ok) break;
      const uint32_t r = base + s * Rec::kBytes;
      uint32_t cur[4] = {vals[0], vals[1], vals[2], vals[3]};
      if (k + 1 < chunks) load_values(v + static_cast<size_t>(k + 1) * kC * a.ld_u, a.ld_u, sp.n - (k + 1) * kC, left, lane, vals);
      float R[3][2][4] = {}, O[3][2][4] = {};            // the three products of the split operands
#pragma unroll
      for (int ks = 0; ks < DP / 16; ++ks) {
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
      uint32_t hi[4], lo[4], bh[4], bl[4];
      {
        float X[2][4];                                   // V - K~ S0, transposed
#pragma unroll
        for (int t = 0; t < 2; ++t)
#pragma unroll
          for (int e = 0; e < 4; ++e) {
            const uint32_t p = cur[2 * t + (e >> 1)];
            X[t][e] = ((e & 1) ? bf16_hi(p) : bf16_lo(p)) - (R[0][t][e] + (R[1][t][e] + R[2][t][e]));
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
      for (int p = 0; p < DP / 16; ++p) {                // the new state
        ldsm4t(bh, r + Rec::kKh + ot + 32 * p);
        ldsm4t(bl, r + Rec::kKh + Rec::kMat + ot + 32 * p);
#pragma unroll
        for (int t = 0; t < 2; ++t) {
          float* st = S[2 * p + t];
          float ex, ey;
          asm volatile("ld.shared.v2.f32 {%0, %1}, [%2];" : "=f"(ex), "=f"(ey) : "r"(r + Rec::kE + (8 * (2 * p + t) + (lane & 3) * 2) * 4) : "memory");
          st[0] *= ex; st[1] *= ey; st[2] *= ex; st[3] *= ey;
          mma(st, hi, bh + 2 * t);
          mma(st, hi, bl + 2 * t);
          mma(st, lo, bh + 2 * t);
        }
      }
      ldsm4(bh, r + Rec::kM + os);
      ldsm4(bl, r + Rec::kM + Rec::kSmall + os);
      __syncwarp();
      if (lane == 0) arrive(empty + 8 * s);              // the record is read
#pragma unroll
      for (int t = 0; t < 2; ++t) {
        mma(O[0][t], hi, bh + 2 * t);
        mma(O[1][t], hi, bl + 2 * t);
        mma(O[2][t], lo, bh + 2 * t);
#pragma unroll
        for (int e = 0; e < 4; ++e) O[0][t][e] += O[1][t][e] + O[2][t][e];
      }
      store_outputs(out + static_cast<size_t>(k) * kC * a.ld_out, a.ld_out, nt, left, lane, O[0]);
    }
    if (!ok && lane == 0) atomicOr(&failed, 1u);
    if (sp.n > 0 && ok) store_state<DP>(a, state, col, lane, S);
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

template <int DP, int NW>
__global__ void __launch_bounds__(32 * NW) ssd_chunk_kernel(const MatrixStateArgs a) {
  constexpr int LD = DP + 8, kTile = kC * LD, kThreads = 32 * NW;
  extern __shared__ __align__(16) __nv_bfloat16 sd_smem[];             // [kRing][B | C][kC][LD]
  const int head = blockIdx.x, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const MsSpan sp = ms_span(a, blockIdx.z);
  const int chunks = (sp.n + kC - 1) / kC, c0 = blockIdx.y * 16 * NW, col = c0 + warp * 16, left = a.vdim - col;
  const int kh = head / (a.heads / a.key_heads);
  const __nv_bfloat16* u = static_cast<const __nv_bfloat16*>(a.u) + static_cast<size_t>(sp.row0) * a.ld_u;
  const int kb = a.k0 + kh * a.dim, qb = a.q0 + kh * a.dim;
  const bool vec = ((a.dim | kb | qb | a.ld_u) & 7) == 0;
  for (int i = threadIdx.x; i < kRing * 2 * kTile / 8; i += kThreads) reinterpret_cast<uint4*>(sd_smem)[i] = make_uint4(0u, 0u, 0u, 0u);
  __syncthreads();
  auto fetch = [&](int k) {
    if (k < chunks) {
      __nv_bfloat16* dst = sd_smem + (k % kRing) * 2 * kTile;
      const int nt = min(kC, sp.n - k * kC);
      const __nv_bfloat16* src = u + static_cast<size_t>(k) * kC * a.ld_u;
      if (vec) {
        const int per = a.dim >> 3;
        for (int i = threadIdx.x; i < 2 * kC * per; i += kThreads) {
          const int which = i / (kC * per), t = i / per % kC, c = i % per * 8;
          __nv_bfloat16* d = dst + which * kTile + t * LD + c;
          if (t < nt) cp16(smem_u32(d), src + static_cast<size_t>(t) * a.ld_u + (which ? qb : kb) + c);
          else *reinterpret_cast<uint4*>(d) = make_uint4(0u, 0u, 0u, 0u);
        }
      } else {
        for (int i = threadIdx.x; i < 2 * kC * a.dim; i += kThreads) {
          const int which = i / (kC * a.dim), t = i / a.dim % kC, c = i % a.dim;
          dst[which * kTile + t * LD + c] = t < nt ? src[static_cast<size_t>(t) * a.ld_u + (which ? qb : kb) + c] : __float2bfloat16_rn(0.f);
        }
      }
    }
    cp_commit();                                         // always, so that groups count chunks
  };
  fetch(0);
  fetch(1);
  const float A = a.A[head], D = a.D[head], bias = a.decay_b[head];
  float* state = a.state + (static_cast<size_t>(sp.seq) * a.heads + head) * a.dim * a.vdim;
  float S[DP / 8][4];
  load_state<DP>(a, state, col, lane, sp.start > 0 && sp.n > 0, S);
  zero_front(a, sp, blockIdx.z, head, c0, 16 * NW, kThreads);
  const __nv_bfloat16* v = u + a.v0 + head * a.vdim + col;
  float* out = a.out + static_cast<size_t>(sp.row0) * a.ld_out + head * a.vdim + col;
  const float* raw = a.decay + static_cast<size_t>(sp.row0) * a.ld_decay + head;
  uint32_t vals[4] = {0u, 0u, 0u, 0u};
  float dt_raw = 0.f;
  if (chunks > 0) {
    load_values(v, a.ld_u, min(kC, sp.n), left, lane, vals);
    if ((lane & 15) < sp.n) dt_raw = raw[static_cast<size_t>(lane & 15) * a.ld_decay];
  }
  const int on = rows_as_n(lane, LD) * 2, om = rows_as_m(lane, LD) * 2;
  for (int k = 0; k < chunks; ++k) {
    const int nt = min(kC, sp.n - k * kC);
    cp_wait<1>();
    __syncthreads();                                     // chunk k has arrived for everyone; chunk k - 1 is read
    fetch(k + 2);
    const uint32_t rb = smem_u32(sd_smem + (k % kRing) * 2 * kTile), rc = rb + kTile * 2;
    const uint32_t x[4] = {vals[0], vals[1], vals[2], vals[3]};
    const float dt = (lane & 15) < nt ? MsFn<__nv_bfloat16>::softplus(dt_raw + bias) : 0.f;
    if (k + 1 < chunks) {
      const int more = sp.n - (k + 1) * kC;
      load_values(v + static_cast<size_t>(k + 1) * kC * a.ld_u, a.ld_u, more, left, lane, vals);
      if ((lane & 15) < more) dt_raw = raw[static_cast<size_t>((k + 1) * kC + (lane & 15)) * a.ld_decay];
    }
    float G = A * dt;                                    // running sum over the chunk's rows, lane = row
#pragma unroll
    for (int o = 1; o < 16; o <<= 1) {
      const float up = __shfl_up_sync(0xffffffffu, G, o, 16);
      if ((lane & 15) >= o) G += up;
    }
    const float last = __shfl_sync(0xffffffffu, G, 15);
    const float Gr[2] = {__shfl_sync(0xffffffffu, G, lane >> 2), __shfl_sync(0xffffffffu, G, (lane >> 2) + 8)};
    float Gc[4], dc[4];                                  // rows (lane & 3) * 2 + {0, 1} (+ 8)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int t = (lane & 3) * 2 + (e & 1) + (e >> 1) * 8;
      Gc[e] = __shfl_sync(0xffffffffu, G, t);
      dc[e] = __shfl_sync(0xffffffffu, dt, t);
    }
    float P[2][4] = {}, O[2][2][4] = {};                 // C B^T [i, j]; S0^T C^T by the split of S0
#pragma unroll
    for (int ks = 0; ks < DP / 16; ++ks) {
      uint32_t hi[4], lo[4], ca[4], cn[4], bn[4];
      split_a(S[2 * ks], S[2 * ks + 1], hi, lo);
      ldsm4(cn, rc + on + 32 * ks);
      ldsm4(ca, rc + om + 32 * ks);
      ldsm4(bn, rb + on + 32 * ks);
#pragma unroll
      for (int t = 0; t < 2; ++t) {
        mma(O[0][t], hi, cn + 2 * t);
        mma(O[1][t], lo, cn + 2 * t);
        mma(P[t], ca, bn + 2 * t);
      }
    }
    // masked and decayed products as the right operand: the accumulator layout of [i, j] is that of an operand with j as K
    uint32_t mh[2][2], ml[2][2];
#pragma unroll
    for (int i8 = 0; i8 < 2; ++i8)
#pragma unroll
      for (int j8 = 0; j8 < 2; ++j8) {
        float w[2];
#pragma unroll
        for (int e = 0; e < 2; ++e) {
          const int i = (lane >> 2) + 8 * i8, j = (lane & 3) * 2 + e + 8 * j8;
          w[e] = j <= i ? P[j8][2 * i8 + e] * __expf(Gr[i8] - Gc[2 * j8 + e]) * dc[2 * j8 + e] : 0.f;
        }
        split2(w[0], w[1], mh[i8][j8], ml[i8][j8]);
      }
    float o[2][4];
    uint32_t uh[4], ul[4];
#pragma unroll
    for (int t = 0; t < 2; ++t) {
      const float e0 = __expf(Gc[2 * t]), e1 = __expf(Gc[2 * t + 1]);
      const float f0 = __expf(last - Gc[2 * t]) * dc[2 * t], f1 = __expf(last - Gc[2 * t + 1]) * dc[2 * t + 1];
#pragma unroll
      for (int h = 0; h < 2; ++h) {
        const float x0 = bf16_lo(x[2 * t + h]), x1 = bf16_hi(x[2 * t + h]);
        o[t][2 * h] = fmaf(D, x0, (O[0][t][2 * h] + O[1][t][2 * h]) * e0);
        o[t][2 * h + 1] = fmaf(D, x1, (O[0][t][2 * h + 1] + O[1][t][2 * h + 1]) * e1);
        split2(x0 * f0, x1 * f1, uh[2 * t + h], ul[2 * t + h]);
      }
    }
    const float el = __expf(last);
#pragma unroll
    for (int p = 0; p < DP / 16; ++p) {
      uint32_t b[4];
      ldsm4t(b, rb + om + 32 * p);
#pragma unroll
      for (int t = 0; t < 2; ++t) {
        float* st = S[2 * p + t];
        st[0] *= el; st[1] *= el; st[2] *= el; st[3] *= el;
        mma(st, uh, b + 2 * t);
        mma(st, ul, b + 2 * t);
      }
    }
#pragma unroll
    for (int t = 0; t < 2; ++t) {
      mma(o[t], x, mh[t]);
      mma(o[t], x, ml[t]);
    }
    store_outputs(out + static_cast<size_t>(k) * kC * a.ld_out, a.ld_out, nt, left, lane, o);
  }
  if (sp.n > 0) store_state<DP>(a, state, col, lane, S);
}

template <typename K>
cudaError_t allow_smem(DeviceOnce& once, K kernel, int bytes) {
  return once.run([&] { return cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes); });
}

template <int DP, int NW>
cudaError_t delta_cols(const MatrixStateArgs& a, int chunks, cudaStream_t s) {
  constexpr int smem = kRing * Record<DP>::kBytes;
  static_assert(smem <= 220 * 1024 && Record<DP>::kBytes % 16 == 0, "shared memory");
  static DeviceOnce once;
  cudaError_t e = allow_smem(once, delta_chunk_kernel<DP, NW>, smem);
  if (e != cudaSuccess) return e;
  delta_chunk_kernel<DP, NW><<<dim3(a.heads, (a.vdim + 16 * NW - 1) / (16 * NW), a.nseq), 32 * (NW + 1), smem, s>>>(a, chunks);
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
  return cols <= 148 * 4 ? delta_cols<DP, 2>(a, chunks, s) : delta_cols<DP, 4>(a, chunks, s);
}

template <int DP>
cudaError_t ssd(const MatrixStateArgs& a, cudaStream_t s) {
  constexpr int smem = kRing * 2 * kC * (DP + 8) * 2, NW = 4;
  static DeviceOnce once;
  cudaError_t e = allow_smem(once, ssd_chunk_kernel<DP, NW>, smem);
  if (e != cudaSuccess) return e;
  ssd_chunk_kernel<DP, NW><<<dim3(a.heads, (a.vdim + 16 * NW - 1) / (16 * NW), a.nseq), 32 * NW, smem, s>>>(a);
  return cudaGetLastError();
}

}  // namespace

int64_t matrix_chunk_record_bytes(int dim) {
  return dim <= 32 ? Record<32>::kBytes : dim <= 64 ? Record<64>::kBytes : dim <= 128 ? Record<128>::kBytes : Record<256>::kBytes;
}

cudaError_t launch_matrix_chunks(const MatrixStateArgs& a, cudaStream_t s) {
  if (!matrix_state_ok(a) || !a.u_bf16 || a.nseq > 65535 || a.heads > 65535) return cudaErrorInvalidValue;
  if (a.delta) {
    if (!a.chunk_records || (reinterpret_cast<uintptr_t>(a.chunk_records) & 15)) return cudaErrorInvalidValue;
    return a.dim <= 32 ? delta<32>(a, s) : a.dim <= 64 ? delta<64>(a, s) : a.dim <= 128 ? delta<128>(a, s) : delta<256>(a, s);
  }
  return a.dim <= 32 ? ssd<32>(a, s) : a.dim <= 64 ? ssd<64>(a, s) : a.dim <= 128 ? ssd<128>(a, s) : ssd<256>(a, s);
}

}  // namespace mtj
