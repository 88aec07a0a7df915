#include "../../include/dejavu_b200_routed.h"
#include "hybrid_moe.cuh"
namespace djv {
bool moe_grouped_tc_supported(int, const GroupedArgs &) { return false; }
int moe_grouped_tc(const GroupedArgs &, cudaStream_t) { return DJV_ERR_UNSUPPORTED; }
}  // namespace djv
extern "C" unsigned djv_moe_timeouts(void) { return 0; }
