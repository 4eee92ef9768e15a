// Weak stand-ins for the kernels of the GPT-J family and of tensor parallelism, for a library that holds only the
// units of layer-stack models (build.py --family stack).  A full build links the real ones over these.
#include "mtj_comm.h"
#include "mtj_gemm_tc.cuh"

namespace mtj {

#define MTJ_WEAK __attribute__((weak))
#define MTJ_ABSENT { return cudaErrorNotSupported; }
#define MTJ_NO_COMM { *err = "this build has no tensor parallelism"; return 1; }

MTJ_WEAK cudaError_t launch_gemm_tc_gptj(GemvEpilogue, bool, const CUtensorMap&, const CUtensorMap&, const CUtensorMap*,
                                         const GemmTcArgs&, cudaStream_t, bool) MTJ_ABSENT
MTJ_WEAK cudaError_t launch_decode_mega(const MegaArgs&, cudaStream_t, int*) MTJ_ABSENT
MTJ_WEAK cudaError_t launch_decode_attn(const DecodeAttnArgs&, cudaStream_t, bool) MTJ_ABSENT
MTJ_WEAK int decode_attn_splits(int) { return 1 << 20; }      // more than mtj_create accepts: no GPT-J handles
MTJ_WEAK cudaError_t launch_prefill_attn(const PrefillAttnArgs&, cudaStream_t) MTJ_ABSENT
MTJ_WEAK cudaError_t launch_prefill_attn_tc(const void*, const void*, const void*, const PrefillAttnTcArgs&,
                                            cudaStream_t) MTJ_ABSENT
MTJ_WEAK int32_t comm_unique_id(uint8_t*, std::string* err) MTJ_NO_COMM
MTJ_WEAK int32_t comm_init(const uint8_t*, int, int, void**, std::string* err) MTJ_NO_COMM
MTJ_WEAK void comm_destroy(void*) {}
MTJ_WEAK int32_t comm_all_reduce(void*, float*, size_t, bool, cudaStream_t, std::string* err) MTJ_NO_COMM
MTJ_WEAK int32_t comm_all_gather(void*, const float*, float*, size_t, cudaStream_t, std::string* err) MTJ_NO_COMM
MTJ_WEAK cudaError_t launch_p2p_allreduce(const P2pArgs&, int, cudaStream_t, bool) MTJ_ABSENT
MTJ_WEAK cudaError_t launch_tp_push_reduce(const TpReduceArgs&, int, cudaStream_t, bool) MTJ_ABSENT
MTJ_WEAK cudaError_t launch_tp_argmax(const TpArgmaxArgs&, int, cudaStream_t, bool) MTJ_ABSENT
MTJ_WEAK cudaError_t launch_residual_stats(float*, const float*, float*, int, int, bool, cudaStream_t, bool) MTJ_ABSENT
MTJ_WEAK cudaError_t launch_gather_rows(const float*, float*, int, int, int, cudaStream_t) MTJ_ABSENT

}  // namespace mtj
