#include "mix_common.cuh"
namespace scmx {
bool latent_attn_tc_supported(int64_t, int64_t, int, int, int, float) { return false; }
int latent_attn_tc(const bf16_t*, int64_t, const bf16_t*, int64_t, const bf16_t*, int64_t, int64_t, int64_t, int64_t, int64_t, int, int, int, int, float, bf16_t*, int32_t*, cudaStream_t) { return SCMX_ELIMIT; }
}
