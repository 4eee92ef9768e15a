// Instances of the tensor-core GEMM with the epilogues that layer-stack models use: plain (fp32 and / or bf16
// result) and SwiGLU over interleaved (gate, up) weight rows.  A file of its own so that it compiles beside the
// GPT-J instances.
#include "mtj_gemm_tc.cuh"

namespace mtj {

cudaError_t launch_gemm_tc_stack(GemvEpilogue epi, bool wide, const CUtensorMap& mw, const CUtensorMap& mx,
                                 const GemmTcArgs& a, cudaStream_t s, bool pdl) {
  if (epi == kEpiSwiGLU ? (!a.out_bf16 || (a.N & 1) || a.partial || a.bias) : (!a.out && !a.out_bf16 && !a.partial))
    return cudaErrorInvalidValue;
  if (wide) return epi == kEpiPlain ? launch_tc_persist<kEpiPlain>(mw, mx, a, s) : launch_tc_persist<kEpiSwiGLU>(mw, mx, a, s);
  switch (gemm_tc_token_tile_for(a.M)) {
    case 32: return epi == kEpiPlain ? launch_tc<32, 5, kEpiPlain>(mw, mx, a, s, pdl) : launch_tc<32, 5, kEpiSwiGLU>(mw, mx, a, s, pdl);
    case 64: return epi == kEpiPlain ? launch_tc<64, 4, kEpiPlain>(mw, mx, a, s, pdl) : launch_tc<64, 4, kEpiSwiGLU>(mw, mx, a, s, pdl);
    default: return epi == kEpiPlain ? launch_tc<128, 3, kEpiPlain>(mw, mx, a, s, pdl) : launch_tc<128, 3, kEpiSwiGLU>(mw, mx, a, s, pdl);
  }
}

}  // namespace mtj
