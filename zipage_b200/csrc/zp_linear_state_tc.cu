#include "zp_linear_state.cuh"
namespace zp {
bool linear_chunk_supports(const LinearArgs&) { return false; }
size_t linear_chunk_workspace(int, int, int, int) { return 0; }
int linear_chunk(const LinearArgs&, cudaStream_t) { return ZP_ERR_UNSUPPORTED; }
}
