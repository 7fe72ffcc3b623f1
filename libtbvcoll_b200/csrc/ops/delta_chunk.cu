// delta_chunk.cu
#include "delta.cuh"
namespace delta_ops {
bool chunk_fits(const Params&) { return false; }
cudaError_t chunk_scan(const Params&, const int*, int, bool*, cudaStream_t) { return cudaErrorNotSupported; }
}  // namespace delta_ops
