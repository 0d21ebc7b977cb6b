#include "mix_delta.cuh"
namespace scmx {
bool delta_tc_supported(int64_t, int, int, int, int64_t) { return false; }
int64_t delta_tc_scratch(int64_t, int, int) { return 0; }
int delta_tc(const DeltaArgs&, bool, void*, int32_t*, cudaStream_t) { return SCMX_ELIMIT; }
}
