#include "tkv_moe.cuh"
namespace tkv {
bool moe_stream_shape(const GroupedGemm&, int) { return false; }
int launch_moe_stream(const GroupedGemm&, cudaStream_t) { return fail(TKV_ERR_UNSUPPORTED, "not built"); }
}
