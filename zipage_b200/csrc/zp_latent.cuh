// Arguments of the attention kernels that meet cached latents directly.
#pragma once
#include "zp_common.cuh"

namespace zp {

// Rows, positions and contexts of the sequences as in WinArgs (zp_window_attn.cuh).
struct LatentArgs {
  const void* q;             // [rows, H, KP]
  const void* cache;         // [n_pages, BS, KP]
  const int32_t* cu_q; const int32_t* context_lens; const int32_t* table;
  void* out;                 // [rows, H, R]
  float* part;               // spans' sums [rows * H, nsplit, R], then (reference, row sum) [rows * H, nsplit, 2]
  int B, NBmax, H, R, KP, BS, n_pages, nsplit;
  int64_t pairs;             // rows * H
  float scale;
};

struct LatSeq { int row0, count, ctx, pos0; };
__device__ __forceinline__ LatSeq lat_seq(const LatentArgs& a, int b) {
  LatSeq s;
  s.row0 = a.cu_q ? a.cu_q[b] : b;
  s.count = a.cu_q ? a.cu_q[b + 1] - s.row0 : 1;
  s.ctx = a.context_lens[b];
  s.pos0 = s.ctx - s.count;
  if (s.pos0 < 0) s.count = 0;   // a padding row of a fixed-size batch (context 0) has no query
  return s;
}
// page of key position `key` of sequence b, kept inside the pool whatever the table holds
__device__ __forceinline__ int lat_page(const LatentArgs& a, int b, int key) {
  const int col = min(key / a.BS, a.NBmax - 1);
  return min(max(a.table[(int64_t)b * a.NBmax + col], 0), a.n_pages - 1);
}

// zp_latent_decode_tc.cu
bool latent_decode_tc_supports(const LatentArgs& a, int dtype);
int latent_decode_splits(int B, int max_q, int H, int span);
int latent_decode_tc(const LatentArgs& a, int max_q, int total_rows, cudaStream_t st);

}  // namespace zp
