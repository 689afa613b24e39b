// Arguments and gate arithmetic shared by the gated delta rule kernels.
#pragma once
#include "zp_common.cuh"

namespace zp {

// One step of a gated delta rule over a batch of sequences.  Per value head, with unit keys and queries (the head's
// share of q | k through a norm of one), a decay g_t = exp(-exp(A) softplus(a_t + dt)), a step b_t = sigmoid(beta_t) and a
// fp32 state S [dim, vdim]:
//   u_t = b_t (v_t - g_t S_(t-1)^T k_t);   S_t = g_t S_(t-1) + k_t u_t^T;   o_t = S_t^T q_t dim^(-1/2)
//   out = o_t / rms(o_t) * weight * silu(gate_t) * out_scale
// x holds the rows q [G, dim] | k [G, dim] | v [H, vdim], head h with the keys of head h / (H / G).  taps > 0: x is the
// projection itself, and a causal convolution over the last `taps` tokens and silu come first; its earlier inputs are in
// `ring` [slots, taps, channels], position p in row p % taps, so that a decoded token's row is never one that another
// block of the same launch still reads.  taps = 0: x has been through zp_short_conv.
// Rows of sequence b are cu_q[b] .. cu_q[b + 1] (NULL: row b alone); context_lens[b] counts its tokens including these, so a
// sequence whose context equals its rows starts from the zero state whatever its slot holds.  Context 0 marks a padding row.
struct DeltaArgs {
  const void* x; const void* gate;      // row strides x_stride, gate_stride
  const float* ab;                      // [rows, 2 H]: a, then beta
  const float *A_log, *dt_bias;         // [H]
  const float* norm_weight;             // [vdim]
  const float* conv_w;                  // [taps, channels]
  void* ring;
  const int32_t* cu_q; const int32_t* context_lens; const int32_t* slots;
  float* S;                             // [slots, H, dim, VP]
  void* out;
  int B, H, G, dim, vdim, VP, n_slots, taps, VT;
  int64_t x_stride, gate_stride, ab_stride, out_stride;
  float eps, out_scale;
};

constexpr float DELTA_UNIT_EPS = 1e-6f;

__device__ __forceinline__ float softplus(float z) { return fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))); }
__device__ __forceinline__ float delta_log_decay(const DeltaArgs& a, int64_t row, int h) {
  return -expf(a.A_log[h]) * softplus(a.ab[row * a.ab_stride + h] + a.dt_bias[h]);
}
__device__ __forceinline__ float delta_beta(const DeltaArgs& a, int64_t row, int h) {
  return 1.f / (1.f + expf(-a.ab[row * a.ab_stride + a.H + h]));
}

struct DeltaSeq { int row0, count, ctx, slot; bool fresh; };
__device__ __forceinline__ DeltaSeq delta_seq(const DeltaArgs& a, int b) {
  DeltaSeq s;
  s.row0 = a.cu_q ? a.cu_q[b] : b;
  s.count = a.cu_q ? a.cu_q[b + 1] - s.row0 : 1;
  s.ctx = a.context_lens[b];
  s.slot = a.slots[b];
  if (s.ctx < s.count || s.slot < 0 || s.slot >= a.n_slots) s.count = 0;
  s.fresh = s.ctx == s.count;
  return s;
}

// chunked tensor-core kernels (zp_delta_tc.cu)
constexpr int DC_C = 64;                           // tokens of a chunk
bool delta_chunk_supports(const DeltaArgs& a, int dtype);
size_t delta_chunk_workspace(int total_rows, int B, int H);
int delta_chunk(const DeltaArgs& a, int total_rows, void* workspace, cudaStream_t st);

}  // namespace zp
