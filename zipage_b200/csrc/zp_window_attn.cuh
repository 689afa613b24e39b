// Arguments shared by the attention kernels with masks, soft caps, distance biases, sinks and output gates (SIMT, mma.sync, tcgen05).
#pragma once
#include "zp_common.cuh"

namespace zp {

// Queries of one step, each sequence's newest tokens, over its paged keys.  Rows of sequence b are
// cu_q[b] .. cu_q[b + 1] (absolute rows of q / out), or row b alone when cu_q is NULL; its context
// (keys up to and including this step's tokens) is context_lens[b], so row r sits at position
// context - count + r and sees the keys j <= position with position - j < window (window > 0) and, with chunk > 0,
// those of its own chunk, floor(j / chunk) = floor(position / chunk); the keys j < keep are seen in any case.  With slopes,
// slopes[h] * (position - j) is taken off a score.  A head's sink is one more term of its softmax's
// denominator, exp(sink[h]).  The result is multiplied by out_scale and by sigmoid(gate), one gate per head or per entry.
struct WinArgs {
  const void* q; const void* k; const void* v;   // q [rows, Hq, D] with a row stride; paged caches [P, BS, Hkv, KP | VP]
  const int32_t* cu_q; const int32_t* context_lens; const int32_t* table;
  void* out; float* part;
  int B, NBmax, Hq, Hkv, D, DV, KP, VP, BS, window, n_pages, nsplit;
  int64_t q_stride;      // elements between rows of q
  int64_t out_stride;    // elements between rows of out
  float scale, softcap;  // softcap 0 = none
  int chunk;             // 0 = none
  int keep;              // first keys that every later query sees
  const float* slopes;   // [Hq] or NULL
  const float* sink;     // [Hq] or NULL
  const void* gate;      // rows of T: [Hq] (WIN_GATE_HEAD) or [Hq, DV] (WIN_GATE_ENTRY)
  int64_t gate_stride;
  int gate_mode;
  float out_scale;
};

// Rows, position of the first row and context of sequence b.
struct WinSeq { int row0, count, ctx, pos0; };
__device__ __forceinline__ WinSeq win_seq(const WinArgs& a, int b) {
  WinSeq s;
  s.row0 = a.cu_q ? a.cu_q[b] : b;
  s.count = a.cu_q ? a.cu_q[b + 1] - s.row0 : 1;
  s.ctx = a.context_lens[b];
  s.pos0 = s.ctx - s.count;
  if (s.pos0 < 0) s.count = 0;   // a padding row of a fixed-size batch (context 0) has no query
  return s;
}
// first key position that a query at `pos` sees
__device__ __forceinline__ int win_first(const WinArgs& a, int pos) {
  const int w = a.window > 0 ? max(0, pos - a.window + 1) : 0;
  return a.chunk > 0 ? max(w, pos - pos % a.chunk) : w;
}
// Tiles of `tk` keys that queries from position `first_pos` to `last_pos` see: `kept` tiles with the kept keys, then those
// from t0 on.
struct WinTiles {
  int kept, t0, n;
  __device__ __forceinline__ int tile(int j) const { return j < kept ? j : t0 + j - kept; }
};
__device__ __forceinline__ WinTiles win_tiles(const WinArgs& a, int first_pos, int last_pos, int tk) {
  WinTiles w;
  w.t0 = win_first(a, first_pos) / tk;
  w.kept = min((a.keep + tk - 1) / tk, w.t0);
  w.n = w.kept + last_pos / tk - w.t0 + 1;
  return w;
}
// slope of head h in log2 units
__device__ __forceinline__ float win_slope2(const WinArgs& a, int h) { return a.slopes ? a.slopes[h] * 1.4426950408889634f : 0.f; }
enum { WIN_GATE_NONE = 0, WIN_GATE_HEAD = 1, WIN_GATE_ENTRY = 2 };
__device__ __forceinline__ float win_sigmoid(float z) { return 1.f / (1.f + __expf(-z)); }
// what the output of head h in `row` (absolute) is multiplied by: the factor of all entries, ...
template <typename T> __device__ __forceinline__ float win_head_factor(const WinArgs& a, int64_t row, int h) {
  if (a.gate_mode != WIN_GATE_HEAD) return a.out_scale;
  return a.out_scale * win_sigmoid(Elem<T>::to_f32(reinterpret_cast<const T*>(a.gate)[row * a.gate_stride + h]));
}
// ... and the one of entry d
template <typename T> __device__ __forceinline__ float win_entry_factor(const WinArgs& a, int64_t row, int h, int d) {
  if (a.gate_mode != WIN_GATE_ENTRY) return 1.f;
  return win_sigmoid(Elem<T>::to_f32(reinterpret_cast<const T*>(a.gate)[row * a.gate_stride + (int64_t)h * a.DV + d]));
}
// the sink of a head in log2 units
__device__ __forceinline__ float win_sink2(const WinArgs& a, int h) { return a.sink ? a.sink[h] * 1.4426950408889634f : -INFINITY; }

// page of key position `key` of sequence b, kept inside the pool whatever the table holds
__device__ __forceinline__ int win_page(const WinArgs& a, int b, int key) {
  const int col = min(key / a.BS, a.NBmax - 1);
  return min(max(a.table[(int64_t)b * a.NBmax + col], 0), a.n_pages - 1);
}

}  // namespace zp
