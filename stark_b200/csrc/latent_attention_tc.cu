// stub
#include "layered.cuh"
namespace sb {
bool latent_prefill_tc_supports(const LatentShape &) { return false; }
stark_b200_status latent_prefill_tc_launch(const LatentArgs &, cudaStream_t) { return STARK_B200_UNSUPPORTED; }
}
