#include "tkv_moe.cuh"
namespace tkv {
bool moe_tc_shape(const GroupedGemm&, int) { return false; }
int launch_moe_tc(const GroupedGemm&, cudaStream_t) { return fail(TKV_ERR_UNSUPPORTED, "not built"); }
}
