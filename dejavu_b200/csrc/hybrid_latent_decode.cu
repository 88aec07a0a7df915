#include "../../include/dejavu_b200_routed.h"
#include "hybrid_latent.cuh"
namespace djv {
bool latent_attend_mma_supported(const LatentDecodeArgs &, bool) { return false; }
int latent_attend_mma(const LatentDecodeArgs &, cudaStream_t) { return DJV_ERR_UNSUPPORTED; }
}  // namespace djv
