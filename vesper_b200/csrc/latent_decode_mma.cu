#include "hybrid.cuh"
namespace vb200 {
bool latent_mma_supported(const vb200_latent_args&) { return false; }
int launch_latent_split_mma(cudaStream_t, const vb200_latent_args&, const LatentPlan&, const float*, float*, int*) { return VB200_ERR_UNSUPPORTED; }
}
