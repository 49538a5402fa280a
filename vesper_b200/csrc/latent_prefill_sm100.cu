#include "hybrid.cuh"
namespace vb200 {
bool latent_sm100_supported(const vb200_latent_args&) { return false; }
int launch_latent_prefill_sm100(cudaStream_t, const vb200_latent_args&, int*) { return VB200_ERR_UNSUPPORTED; }
}
