// Arguments and gate arithmetic shared by the matrix-memory (mLSTM) kernels.
#pragma once
#include "zp_common.cuh"

namespace zp {

// One step of a matrix-memory mixer over a batch of sequences.  Per head, with a log input gate i_t, a
// log forget gate f_t, a running maximum m (initially 0) and a fp32 state (S [dim, vdim], n [dim]):
//   m_t = max(f_t + m_(t-1), i_t)
//   S_t = exp(f_t + m_(t-1) - m_t) S_(t-1) + exp(i_t - m_t) k_t v_t^T        (n_t with k_t alone)
//   o_t = S_t^T q_t / (max(|n_t . q_t|, exp(-m_t)) + 1e-6)
//   out = o_t / rms(o_t) * weight * sigmoid(g_t)
// Rows of sequence b are cu_q[b] .. cu_q[b + 1] (NULL: row b alone); context_lens[b] counts its tokens
// including these, so a sequence whose context equals its rows starts from the zero state whatever its
// slot holds.  Context 0 marks a padding row of a fixed-size batch.
struct MlstmArgs {
  const void* q; const void* k; const void* v; const void* g;   // [rows, H * dim | H * vdim], common row stride
  const float* gates;       // [rows, 2 H] pre-activations: input gates, then forget gates
  const float* gate_bias;   // [2 H]
  const float* norm_weight; // [H * vdim]
  const int32_t* cu_q; const int32_t* context_lens; const int32_t* slots;
  float* S; float* n; float* m;   // [slots, H, dim, VP], [slots, H, dim], [slots, H]
  void* out;
  int B, H, dim, vdim, VP, n_slots, VT;
  int64_t row_stride, gates_stride, out_stride;
  float qscale, cap, eps;
};

constexpr float MLSTM_DEN_EPS = 1e-6f;

__device__ __forceinline__ float soft_cap(float x, float cap) { return cap * tanhf(x / cap); }
__device__ __forceinline__ float log_sigmoid(float x) { return fminf(x, 0.f) - log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ float log_input_gate(const MlstmArgs& a, int64_t row, int h) {
  return soft_cap(a.gates[row * a.gates_stride + h] + a.gate_bias[h], a.cap);
}
__device__ __forceinline__ float log_forget_gate(const MlstmArgs& a, int64_t row, int h) {
  return log_sigmoid(soft_cap(a.gates[row * a.gates_stride + a.H + h] + a.gate_bias[a.H + h], a.cap));
}

struct MlstmSeq { int row0, count, ctx, slot; bool fresh; };
__device__ __forceinline__ MlstmSeq mlstm_seq(const MlstmArgs& a, int b) {
  MlstmSeq s;
  s.row0 = a.cu_q ? a.cu_q[b] : b;
  s.count = a.cu_q ? a.cu_q[b + 1] - s.row0 : 1;
  s.ctx = a.context_lens[b];
  s.slot = a.slots[b];
  if (s.ctx < s.count || s.slot < 0 || s.slot >= a.n_slots) s.count = 0;
  s.fresh = s.ctx == s.count;
  return s;
}

// ---- thread-block clusters along the value dims: per-row sums over the whole head ---------------
__device__ __forceinline__ uint32_t cluster_rank() { uint32_t r; asm("mov.u32 %0, %%cluster_ctarank;" : "=r"(r)); return r; }
__device__ __forceinline__ uint32_t cluster_size() { uint32_t r; asm("mov.u32 %0, %%cluster_nctarank;" : "=r"(r)); return r; }
__device__ __forceinline__ void cluster_sync() {
  asm volatile("barrier.cluster.arrive.release.aligned;\n barrier.cluster.wait.acquire.aligned;" ::: "memory");
}
// a float of the same shared-memory variable in another block of the cluster
__device__ __forceinline__ float ld_cluster(const float* p, uint32_t rank) {
  uint32_t a = static_cast<uint32_t>(__cvta_generic_to_shared(p)), ra;
  float v;
  asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(ra) : "r"(a), "r"(rank));
  asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(ra) : "memory");
  return v;
}

}  // namespace zp
