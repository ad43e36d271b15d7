// Stand-ins for the packed-weight units (oxb_mmq_*.cu, oxb_gemv.cu) in the core build of the library, which models with
// bf16 / f32 weights need and which compiles in a fraction of the time: a packed-weight call reports an error.
#include "mmq_dispatch.h"

namespace oxb {
#define OXB_NO_MMQ(name) \
  int name(OXB_MMQ_ARGS) { return (int)cudaErrorNotSupported; }
OXB_NO_MMQ(gemm_mmq_q4_k)
OXB_NO_MMQ(gemm_mmq_q6_k)
OXB_NO_MMQ(gemm_mmq_q8_0)
OXB_NO_MMQ(gemm_mmq_q4_0)
OXB_NO_MMQ(gemm_mmq_nvfp4)
OXB_NO_MMQ(gemm_mmq_fp8b)
int gemv_quant_run(int, const uint8_t*, size_t, const __nv_bfloat16*, int, __nv_bfloat16*, int, const float*, int, int, int, int, int,
                   cudaStream_t) {
  return (int)cudaErrorNotSupported;
}
}  // namespace oxb
