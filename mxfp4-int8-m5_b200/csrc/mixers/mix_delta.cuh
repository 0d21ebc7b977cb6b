// Arguments of the gated delta rule over a prompt portion, shared by its token-by-token and tensor-core forms.
#pragma once
#include "mix_common.cuh"

namespace scmx {

struct DeltaArgs {
    const void *q, *k, *v;    // [n, ld*]: heads side by side, after convolution and SiLU
    const void* b;            // [n, ldb] logits of beta
    const void* a;            // [n, lda] decay logits: storage type, one per head; or float, one per head and key channel
    const float *nA, *dtb;    // -exp(A_log) [H]; dt_bias [H] or [H d]
    float* state;             // [H, d, dv]
    float* o;                 // [n, H, dv]
    int64_t n, ldq, ldk, ldv, ldb, lda;
    int H, G, d, dv;
};

bool delta_tc_supported(int64_t n, int H, int d, int dv, int64_t ldv);
int64_t delta_tc_scratch(int64_t n, int H, int d, int dv);
int delta_tc(const DeltaArgs& a, bool channel, void* scratch, int32_t* status, cudaStream_t st);

}  // namespace scmx
