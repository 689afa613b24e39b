#include "zp_moe.cuh"
namespace zp {
bool grouped_tc_supports(const GroupedArgs&, int) { return false; }
int grouped_gemm_tc(const GroupedArgs&, cudaStream_t) { return ZP_ERR_UNSUPPORTED; }
}  // namespace zp
