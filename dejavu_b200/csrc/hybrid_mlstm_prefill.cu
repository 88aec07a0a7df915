#include "../../include/dejavu_b200_routed.h"
#include "hybrid_mlstm.cuh"
namespace djv {
bool mlstm_tc_supported(int, int, int) { return false; }
int mlstm_tc_chunk_state(const MlstmArgs &, cudaStream_t) { return DJV_ERR_UNSUPPORTED; }
int mlstm_tc_chunk_out(const MlstmArgs &, cudaStream_t) { return DJV_ERR_UNSUPPORTED; }
}  // namespace djv
extern "C" unsigned djv_mlstm_timeouts(void) { return 0; }
