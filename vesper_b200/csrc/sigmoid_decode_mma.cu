#include "hybrid.cuh"
namespace vb200 {
bool sig_decode_mma_supported(const vb200_sigattn_args&) { return false; }
int launch_sig_decode_mma(cudaStream_t, const vb200_sigattn_args&, const SigPlan&, const void*, float*, int*) { return VB200_ERR_UNSUPPORTED; }
}
