// Arguments shared by the grouped (per-expert) matrix product kernels.
#pragma once
#include "zp_common.cuh"

namespace zp {

// out[p, n] = act(sum_k x[r(p), k] w[e, n, k]) for the places p = offsets[e] .. offsets[e + 1] of each expert e;
// r(p) = rows[p], or p itself when rows is NULL.  With ZP_ACT_SILU_MUL the rows of w come in blocks of 16 gates and 16
// ups, and out[p, i] = silu(s_p gate_i) * (s_p up_i), [places, Nout / 2], s_p = row_scale[p] (NULL = 1).
struct GroupedArgs {
  const void* x;
  const int32_t* rows;
  const void* w;             // [E, Nout, K]
  const int32_t* offsets;    // [E + 1]
  const float* row_scale;
  void* out;                 // [places, Nout]
  int64_t x_stride;          // elements between rows of x
  int src_rows, places, E, Nout, K, act;
};

// tcgen05 kernel (zp_moe_tc.cu)
bool grouped_tc_supports(const GroupedArgs& a, int dtype);
int grouped_gemm_tc(const GroupedArgs& a, cudaStream_t st);

}  // namespace zp
