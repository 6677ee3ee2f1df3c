#include "tkv_latent.cuh"
namespace tkv {
bool two_part_tc_shape(const TwoPartAttn&, int) { return false; }
int launch_two_part_tc(const TwoPartAttn&, int64_t, int, cudaStream_t) { return fail(TKV_ERR_UNSUPPORTED, "not built"); }
}
