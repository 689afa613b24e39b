// Arguments shared by the sliding-window / soft-capped attention kernels (SIMT and mma.sync).
#pragma once
#include "zp_common.cuh"

namespace zp {

// Queries of one step, each sequence's newest tokens, over its paged keys.  Rows of sequence b are
// cu_q[b] .. cu_q[b + 1] (absolute rows of q / out), or row b alone when cu_q is NULL; its context
// (keys up to and including this step's tokens) is context_lens[b], so row r sits at position
// context - count + r and sees the keys j with 0 <= position - j < window.
struct WinArgs {
  const void* q; const void* k; const void* v;   // q [rows, Hq, D] with a row stride; paged caches [P, BS, Hkv, KP | VP]
  const int32_t* cu_q; const int32_t* context_lens; const int32_t* table;
  void* out; float* part;
  int B, NBmax, Hq, Hkv, D, DV, KP, VP, BS, window, n_pages, nsplit;
  int64_t q_stride;      // elements between rows of q
  int64_t out_stride;    // elements between rows of out
  float scale, softcap;  // softcap 0 = none
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
  return a.window > 0 ? max(0, pos - a.window + 1) : 0;
}
// page of key position `key` of sequence b, kept inside the pool whatever the table holds
__device__ __forceinline__ int win_page(const WinArgs& a, int b, int key) {
  const int col = min(key / a.BS, a.NBmax - 1);
  return min(max(a.table[(int64_t)b * a.NBmax + col], 0), a.n_pages - 1);
}

}  // namespace zp
