#include "hybrid.cuh"
namespace vb200 {
bool ssd_chunk_supported(const vb200_ssd_args&) { return false; }
int launch_ssd_chunks(cudaStream_t, const vb200_ssd_args&, const SsdPlan&, const void*, void*, float*) { return VB200_ERR_UNSUPPORTED; }
}
