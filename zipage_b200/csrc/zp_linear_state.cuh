// Arguments and gate arithmetic shared by the kernels of linear attention with a decaying matrix state.
#pragma once
#include "zp_common.cuh"

namespace zp {

// One step of a linear-attention recurrence over a batch of sequences.  Per head, with a fp32 state S [dim, vdim]:
//   S_t = diag(a_t) S_(t-1) + k_t v_t^T;   o_t = S_t^T q_t (+ D v_t)
// The kind says where the decays a_t, keys and queries come from; z is a fp32 projection of the layer's input:
//   FORGET  a = l + (1 - l) sigmoid(z + bias) per channel, k = 1 - a, q = silu(q)          (l = lower)
//   POWER   a = sigmoid(z + bias)^rtau per channel, q and k as projected, q times qscale
//   SCALAR  dt = softplus(z + bias) per head, a = exp(-exp(A_log) dt), k times dt, D v_t added to o_t; G groups of
//           heads share q and k
// taps > 0: q, k and v are the projection itself and a causal convolution over the last `taps` tokens with bias and silu comes
// first; channels: v [H, vdim] | k [G, dim] | q [G, dim].  Its earlier inputs are in `ring` [slots, taps, channels], position p
// in row p % taps, so that a decoded token's row is never one that another block of the launch still reads.
// Rows of sequence b are cu_q[b] .. cu_q[b + 1] (NULL: row b alone); context_lens[b] counts its tokens including these, so a
// sequence whose context equals its rows starts from the zero state whatever its slot holds.  Context 0 marks a padding row.
using LinearArgs = zp_linear_state_params;

struct LinearSeq { int row0, count, ctx, slot; bool fresh; };
__device__ __forceinline__ LinearSeq linear_seq(const LinearArgs& a, int b) {
  LinearSeq s;
  s.row0 = a.cu_seqlens_q ? a.cu_seqlens_q[b] : b;
  s.count = a.cu_seqlens_q ? a.cu_seqlens_q[b + 1] - s.row0 : 1;
  s.ctx = a.context_lens[b];
  s.slot = a.slots[b];
  if (s.ctx < s.count || s.slot < 0 || s.slot >= a.n_slots) s.count = 0;
  s.fresh = s.ctx == s.count;
  return s;
}

__device__ __forceinline__ float ls_softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float ls_sigmoid(float z) { return 1.f / (1.f + expf(-z)); }

// chunked tensor-core kernels (zp_linear_state_tc.cu)
constexpr int LC_C = 64;                           // tokens of a chunk
bool linear_chunk_supports(const LinearArgs& a);
size_t linear_chunk_workspace(int total_rows, int B, int H, int dim);
int linear_chunk(const LinearArgs& a, cudaStream_t st);

}  // namespace zp
