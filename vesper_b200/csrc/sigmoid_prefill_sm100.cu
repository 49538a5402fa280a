#include "hybrid.cuh"
namespace vb200 {
bool sig_prefill_sm100_supported(const vb200_sigattn_args&) { return false; }
int launch_sig_prefill_sm100(cudaStream_t, const vb200_sigattn_args&, const SigPlan&, const void*, int*) { return VB200_ERR_UNSUPPORTED; }
}
