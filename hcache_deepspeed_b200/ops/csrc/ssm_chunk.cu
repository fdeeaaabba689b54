#include "ssm.cuh"
namespace hds {
bool ssm_chunk_supported(const SsmArgs&, int) { return false; }
int ssm_chunk_launch(const SsmArgs&, int, cudaStream_t) { return HDS_ERR_UNSUPPORTED; }
}  // namespace hds
