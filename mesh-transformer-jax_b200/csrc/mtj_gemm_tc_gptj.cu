// Instances of the tensor-core GEMM with the GPT-J epilogues.
#include "mtj_gemm_tc.cuh"

namespace mtj {

cudaError_t launch_gemm_tc_gptj(GemvEpilogue epi, bool wide, const CUtensorMap& mw, const CUtensorMap& mx,
                                const CUtensorMap* ml, const GemmTcArgs& a, cudaStream_t s, bool pdl) {
  if (wide) {
    switch (epi) {
      case kEpiInProj: return launch_tc_persist<kEpiInProj>(mw, mx, a, s);
      case kEpiOut: return launch_tc_persist<kEpiOut>(mw, mx, a, s);
      case kEpiLogitsCE:
        if (!a.ce_gmax || !a.ce_gsum || !a.ce_tlogit || !a.ce_hit || !a.ce_targets || a.ce_ld < a.M) return cudaErrorInvalidValue;
        return launch_tc_persist<kEpiLogitsCE>(mw, mx, a, s);
      default: return launch_tc_persist<kEpiLogits>(mw, mx, a, s);
    }
  }
  if (ml) {
    // hi + lo activations: token tiles of 32 or 64 rows only (few-sequence decode)
    const int bnl = gemm_tc_token_tile_for(a.M);
    if (bnl == 32) {
      switch (epi) {
        case kEpiInProj: return launch_tc<32, 4, kEpiInProj, true>(mw, mx, a, s, pdl, ml);
        case kEpiOut: return launch_tc<32, 4, kEpiOut, true>(mw, mx, a, s, pdl, ml);
        default: return launch_tc<32, 4, kEpiLogits, true>(mw, mx, a, s, pdl, ml);
      }
    }
    if (bnl == 64) {
      switch (epi) {
        case kEpiInProj: return launch_tc<64, 3, kEpiInProj, true>(mw, mx, a, s, pdl, ml);
        case kEpiOut: return launch_tc<64, 3, kEpiOut, true>(mw, mx, a, s, pdl, ml);
        default: return launch_tc<64, 3, kEpiLogits, true>(mw, mx, a, s, pdl, ml);
      }
    }
    return cudaErrorInvalidValue;
  }
  // Few token rows (batched decode) stream the weights once: a narrower token tile leaves room for a
  // deeper TMA ring, i.e. more weight bytes in flight per block.
  const int bn = gemm_tc_token_tile_for(a.M);
  if (bn == 32) {
    switch (epi) {
      case kEpiInProj: return launch_tc<32, 5, kEpiInProj>(mw, mx, a, s, pdl);
      case kEpiOut: return launch_tc<32, 5, kEpiOut>(mw, mx, a, s, pdl);
      default: return launch_tc<32, 5, kEpiLogits>(mw, mx, a, s, pdl);
    }
  }
  if (bn == 64) {
    switch (epi) {
      case kEpiInProj: return launch_tc<64, 4, kEpiInProj>(mw, mx, a, s, pdl);
      case kEpiOut: return launch_tc<64, 4, kEpiOut>(mw, mx, a, s, pdl);
      default: return launch_tc<64, 4, kEpiLogits>(mw, mx, a, s, pdl);
    }
  }
  switch (epi) {
    case kEpiInProj: return launch_tc<128, 3, kEpiInProj>(mw, mx, a, s, pdl);
    case kEpiOut: return launch_tc<128, 3, kEpiOut>(mw, mx, a, s, pdl);
    default: return launch_tc<128, 3, kEpiLogits>(mw, mx, a, s, pdl);
  }
}

}  // namespace mtj
