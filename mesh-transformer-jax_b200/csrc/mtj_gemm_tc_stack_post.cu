// Further instances of the tensor-core GEMM for layer-stack models: squared-relu feed-forwards and capped logits.  A
// file of its own so that it compiles beside the others.
#include "mtj_gemm_tc.cuh"

namespace mtj {

cudaError_t launch_gemm_tc_stack_post(GemvEpilogue epi, bool wide, const CUtensorMap& mw, const CUtensorMap& mx,
                                      const GemmTcArgs& a, cudaStream_t s, bool pdl) {
  if (a.partial || a.bias || (epi == kEpiRelu2 ? !a.out_bf16 : !a.out || a.softcap <= 0.f)) return cudaErrorInvalidValue;
  if (wide) return epi == kEpiRelu2 ? launch_tc_persist<kEpiRelu2>(mw, mx, a, s) : launch_tc_persist<kEpiSoftcap>(mw, mx, a, s);
  switch (gemm_tc_token_tile_for(a.M)) {
    case 32: return epi == kEpiRelu2 ? launch_tc<32, 5, kEpiRelu2>(mw, mx, a, s, pdl) : launch_tc<32, 5, kEpiSoftcap>(mw, mx, a, s, pdl);
    case 64: return epi == kEpiRelu2 ? launch_tc<64, 4, kEpiRelu2>(mw, mx, a, s, pdl) : launch_tc<64, 4, kEpiSoftcap>(mw, mx, a, s, pdl);
    default: return epi == kEpiRelu2 ? launch_tc<128, 3, kEpiRelu2>(mw, mx, a, s, pdl) : launch_tc<128, 3, kEpiSoftcap>(mw, mx, a, s, pdl);
  }
}

}  // namespace mtj
