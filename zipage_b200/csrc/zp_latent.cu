// Row kernels of latent attention (keys and values of all heads are products of one small cached latent):
//   * from a token's down projections: the query latent RMS-normed, the key/value latent RMS-normed, the
//     shared key part rotated, both written to the token's cache row (and to a dense row),
//   * rotation of the queries' rotated part, in place or into the rows that meet the latents directly,
//   * the dense copy of sequences' cached rows.
// Norms, angles and rotations are fp32; angles come from fp64 turns per position, reduced to a fraction of
// a turn before the conversion.
#include "zp_latent.cuh"

namespace zp {

constexpr int LP_THREADS = 128;

// cos and sin of position * turns (in turns)
__device__ __forceinline__ void turn_cs(int64_t pos, double turns, float& c, float& s) {
  const double t = (double)pos * turns;
  sincospif(2.f * (float)(t - rint(t)), &s, &c);
}

// v (n entries) -> T(v * rsqrt(mean(v^2) + eps) * w) at each of dst0 / dst1 (may be NULL)
template <typename T>
__device__ __forceinline__ void rms_part(const T* __restrict__ v, int n, const float* __restrict__ w, float eps, T* dst0, T* dst1,
                                         float* red, bool vec) {
  constexpr int EPV = 16 / sizeof(T);
  float ss = 0.f;
  if (vec) {
    for (int c = threadIdx.x * EPV; c < n; c += LP_THREADS * EPV) {
      const int4 raw = ld16(v + c);
      const T* e = reinterpret_cast<const T*>(&raw);
#pragma unroll
      for (int j = 0; j < EPV; ++j) { const float f = Elem<T>::to_f32(e[j]); ss = fmaf(f, f, ss); }
    }
  } else {
    for (int c = threadIdx.x; c < n; c += LP_THREADS) { const float f = Elem<T>::to_f32(v[c]); ss = fmaf(f, f, ss); }
  }
  const float r = 1.f / sqrtf(block_sum(ss, red) / (float)n + eps);
  if (vec) {
    for (int c = threadIdx.x * EPV; c < n; c += LP_THREADS * EPV) {
      const int4 raw = ld16(v + c);
      const T* e = reinterpret_cast<const T*>(&raw);
      int4 o;
      T* oe = reinterpret_cast<T*>(&o);
#pragma unroll
      for (int j = 0; j < EPV; ++j) oe[j] = Elem<T>::from_f32(Elem<T>::to_f32(e[j]) * r * w[c + j]);
      if (dst0) st16(dst0 + c, o);
      if (dst1) st16(dst1 + c, o);
    }
  } else {
    for (int c = threadIdx.x; c < n; c += LP_THREADS) {
      const T o = Elem<T>::from_f32(Elem<T>::to_f32(v[c]) * r * w[c]);
      if (dst0) dst0[c] = o;
      if (dst1) dst1[c] = o;
    }
  }
}

// One block per token: y [q_rank | kv_rank | rot] -> cq, cache row [kv_rank | rot | padding] and dense row.
template <typename T>
__global__ void __launch_bounds__(LP_THREADS)
latent_prepare_kernel(const T* __restrict__ y, int64_t ld, const int64_t* __restrict__ positions,
                      const double* __restrict__ turns, const float* __restrict__ wq, const float* __restrict__ wkv,
                      T* __restrict__ cq, T* __restrict__ cache, T* __restrict__ dense, const int32_t* __restrict__ slot_mapping,
                      int q_rank, int kv_rank, int rot, int KP, int64_t n_slots, float eps, int vec_q, int vec_kv) {
  __shared__ float red[32];
  const int64_t i = blockIdx.x;
  const T* row = y + i * ld;
  rms_part<T>(row, q_rank, wq, eps, cq + i * q_rank, (T*)nullptr, red, vec_q);
  if (kv_rank == 0) return;
  row += q_rank;
  const int64_t slot = slot_mapping[i];
  T* c0 = slot >= 0 && slot < n_slots ? cache + slot * KP : nullptr;
  T* c1 = dense ? dense + i * KP : nullptr;
  rms_part<T>(row, kv_rank, wkv, eps, c0, c1, red, vec_kv);
  const int64_t pos = positions[i];
  for (int t = threadIdx.x; 2 * t < rot; t += LP_THREADS) {
    float c, s;
    turn_cs(pos, turns[t], c, s);
    const float u = Elem<T>::to_f32(row[kv_rank + 2 * t]), v = Elem<T>::to_f32(row[kv_rank + 2 * t + 1]);
    const T a = Elem<T>::from_f32(u * c - v * s), b = Elem<T>::from_f32(v * c + u * s);
    if (c0) { c0[kv_rank + 2 * t] = a; c0[kv_rank + 2 * t + 1] = b; }
    if (c1) { c1[kv_rank + 2 * t] = a; c1[kv_rank + 2 * t + 1] = b; }
  }
  if (c1)
    for (int t = kv_rank + rot + threadIdx.x; t < KP; t += LP_THREADS) c1[t] = Elem<T>::from_f32(0.f);
}

// One block per token: the last `rot` entries of each head of q [H, dim + rot] turned; written in place, or
// (q_lat given) to entries kv_rank .. kv_rank + rot of q_lat [H, KP], whose padding becomes zero.
template <typename T>
__global__ void __launch_bounds__(LP_THREADS)
latent_rotate_q_kernel(T* __restrict__ q, int64_t ld, const int64_t* __restrict__ positions, const double* __restrict__ turns,
                       T* __restrict__ q_lat, int H, int dim, int rot, int kv_rank, int KP) {
  extern __shared__ float2 cs[];
  const int64_t i = blockIdx.x, pos = positions[i];
  const int half = rot / 2;
  for (int t = threadIdx.x; t < half; t += LP_THREADS) turn_cs(pos, turns[t], cs[t].x, cs[t].y);
  __syncthreads();
  T* row = q + i * ld;
  for (int k = threadIdx.x; k < H * half; k += LP_THREADS) {
    const int h = k / half, t = k - h * half;
    T* p = row + h * (dim + rot) + dim + 2 * t;
    const float u = Elem<T>::to_f32(p[0]), v = Elem<T>::to_f32(p[1]);
    T* o = q_lat ? q_lat + (i * H + h) * KP + kv_rank + 2 * t : p;
    o[0] = Elem<T>::from_f32(u * cs[t].x - v * cs[t].y);
    o[1] = Elem<T>::from_f32(v * cs[t].x + u * cs[t].y);
  }
  if (q_lat) {
    const int pad = KP - kv_rank - rot;
    for (int k = threadIdx.x; k < H * pad; k += LP_THREADS)
      q_lat[(i * H + k / pad) * KP + kv_rank + rot + k % pad] = Elem<T>::from_f32(0.f);
  }
}

// One warp per row of dense [total, KP]: key cu_k[b] + j <- position j of sequence b.
__global__ void __launch_bounds__(256)
gather_rows_kernel(const int4* __restrict__ cache, const int32_t* __restrict__ table, const int32_t* __restrict__ cu_k,
                   int4* __restrict__ dense, int B, int NBmax, int BS, int n_pages, int vecs, int total) {
  const int i = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
  if (i >= total) return;
  int lo = 0, hi = B - 1;                 // last b with cu_k[b] <= i
  while (lo < hi) {
    const int mid = (lo + hi + 1) >> 1;
    if (cu_k[mid] <= i) lo = mid; else hi = mid - 1;
  }
  const int j = i - cu_k[lo];
  const int page = min(max(table[(int64_t)lo * NBmax + min(j / BS, NBmax - 1)], 0), n_pages - 1);
  const int4* src = cache + ((int64_t)page * BS + j % BS) * vecs;
  for (int c = lane; c < vecs; c += 32) dense[(int64_t)i * vecs + c] = src[c];
}

}  // namespace zp

extern "C" int zp_latent_prepare(const void* y, int64_t row_stride, const int64_t* positions, const double* turns,
                                 const float* q_weight, const float* kv_weight, void* cq, void* cache, void* dense,
                                 const int32_t* slot_mapping, int n_tokens, int q_rank, int kv_rank, int rot, int KP,
                                 int64_t n_slots, float eps, int dtype, void* stream) {
  if (n_tokens == 0) return ZP_OK;
  ZP_REQUIRE(y && q_weight && cq, "zp_latent_prepare: null pointer");
  ZP_REQUIRE(q_rank > 0 && kv_rank >= 0 && rot >= 0 && rot % 2 == 0, "zp_latent_prepare: bad sizes");
  ZP_REQUIRE(kv_rank == 0 || (positions && kv_weight && cache && slot_mapping && KP >= kv_rank + rot && (rot == 0 || turns)),
             "zp_latent_prepare: a key/value latent without its cache, weight or positions");
  const int epv = 16 / (int)zp::dtype_size(dtype);
  const int vec_q = q_rank % epv == 0 && row_stride % epv == 0 && ((uintptr_t)y | (uintptr_t)cq) % 16 == 0;
  const int vec_kv = vec_q && kv_rank % epv == 0 && KP % epv == 0 && ((uintptr_t)cache | (uintptr_t)dense) % 16 == 0;
  ZP_DISPATCH_DTYPE(dtype, T, {
    zp::latent_prepare_kernel<T><<<n_tokens, zp::LP_THREADS, 0, (cudaStream_t)stream>>>(
        (const T*)y, row_stride, positions, turns, q_weight, kv_weight, (T*)cq, (T*)cache, (T*)dense, slot_mapping, q_rank, kv_rank,
        rot, KP, n_slots, eps, vec_q, vec_kv);
  });
  return zp::check_launch("zp_latent_prepare");
}

extern "C" int zp_latent_rotate_q(void* q, int64_t row_stride, const int64_t* positions, const double* turns, void* q_lat,
                                  int n_tokens, int H, int dim, int rot, int kv_rank, int KP, int dtype, void* stream) {
  if (n_tokens == 0 || (rot == 0 && !q_lat)) return ZP_OK;
  ZP_REQUIRE(q && positions && (turns || rot == 0), "zp_latent_rotate_q: null pointer");
  ZP_REQUIRE(H > 0 && dim >= 0 && rot >= 0 && rot % 2 == 0 && rot <= 4096 && (!q_lat || KP >= kv_rank + rot), "zp_latent_rotate_q: bad sizes");
  ZP_DISPATCH_DTYPE(dtype, T, {
    zp::latent_rotate_q_kernel<T><<<n_tokens, zp::LP_THREADS, rot / 2 * sizeof(float2), (cudaStream_t)stream>>>(
        (T*)q, row_stride, positions, turns, (T*)q_lat, H, dim, rot, kv_rank, KP);
  });
  return zp::check_launch("zp_latent_rotate_q");
}

extern "C" int zp_gather_rows(const void* cache, const int32_t* block_table, const int32_t* cu_seqlens_k, void* dense, int B,
                              int NBmax, int BS, int n_pages, int row_bytes, int total, void* stream) {
  if (total == 0 || B == 0) return ZP_OK;
  ZP_REQUIRE(cache && block_table && cu_seqlens_k && dense, "zp_gather_rows: null pointer");
  ZP_REQUIRE(NBmax > 0 && BS > 0 && n_pages > 0 && row_bytes > 0 && row_bytes % 16 == 0 && ((uintptr_t)cache | (uintptr_t)dense) % 16 == 0,
             "zp_gather_rows: rows must be whole 16-byte pieces");
  zp::gather_rows_kernel<<<(total + 7) / 8, 256, 0, (cudaStream_t)stream>>>(
      (const int4*)cache, block_table, cu_seqlens_k, (int4*)dense, B, NBmax, BS, n_pages, row_bytes / 16, total);
  return zp::check_launch("zp_gather_rows");
}

extern "C" size_t zp_latent_attention_workspace_bytes(int total_rows, int B, int max_seqlen_q, int H, int R, int span) {
  if (total_rows < 1 || B < 1 || max_seqlen_q < 1 || H < 1) return 0;
  const int ns = zp::latent_decode_splits(B, max_seqlen_q, H, span);
  return ns > 1 ? (size_t)total_rows * H * ns * (R + 2) * sizeof(float) : 0;
}

extern "C" int zp_latent_attention(const void* q, const void* cache, const int32_t* cu_seqlens_q, const int32_t* context_lens,
                                   const int32_t* block_table, void* out, int B, int max_seqlen_q, int total_rows, int NBmax, int H,
                                   int R, int KP, int BS, int n_pages, float scale, int impl, int dtype, void* workspace,
                                   size_t workspace_bytes, void* stream) {
  if (B == 0 || (cu_seqlens_q && max_seqlen_q == 0)) return ZP_OK;
  ZP_REQUIRE(q && cache && context_lens && block_table && out, "zp_latent_attention: null pointer");
  ZP_REQUIRE(H > 0 && R > 0 && R <= 1024 && R <= KP && KP % 16 == 0 && KP <= 2048, "zp_latent_attention: %d of %d entries", R, KP);
  ZP_REQUIRE(BS > 0 && BS % 64 == 0 && NBmax > 0 && n_pages > 0 && B <= 65535 && total_rows > 0, "zp_latent_attention: bad sizes");
  const int max_q = cu_seqlens_q ? max_seqlen_q : 1;
  zp::LatentArgs a;
  a.q = q; a.cache = cache; a.cu_q = cu_seqlens_q; a.context_lens = context_lens; a.table = block_table; a.out = out;
  a.part = nullptr; a.B = B; a.NBmax = NBmax; a.H = H; a.R = R; a.KP = KP; a.BS = BS; a.n_pages = n_pages;
  a.pairs = (int64_t)total_rows * H; a.scale = scale;
  const bool tc = zp::latent_decode_tc_supports(a, dtype) && (int64_t)max_q * H <= 65535 * 16ll;
  if (impl == ZP_IMPL_TCGEN05 && !tc) {
    zp::set_error("zp_latent_attention: the tcgen05 kernel needs bf16, rows of at most 640 entries and 16-byte aligned tensors");
    return ZP_ERR_UNSUPPORTED;
  }
  if (tc && impl != ZP_IMPL_SIMT) {
    a.nsplit = zp::latent_decode_splits(B, max_q, H, NBmax * BS);
    if (a.nsplit > 1) {
      const size_t need = (size_t)a.pairs * a.nsplit * (R + 2) * sizeof(float);
      ZP_REQUIRE(workspace && workspace_bytes >= need, "zp_latent_attention: workspace of %zu bytes, %zu needed", workspace_bytes, need);
      a.part = reinterpret_cast<float*>(workspace);
    }
    return zp::latent_decode_tc(a, max_q, total_rows, (cudaStream_t)stream);
  }
  // one shared key/value head whose values are the first R entries of its keys
  return zp_window_attention(q, cache, cache, cu_seqlens_q, context_lens, block_table, out, B, max_seqlen_q, NBmax, H, 1, KP, R, KP,
                             KP, BS, n_pages, (int64_t)H * KP, (int64_t)H * R, scale, 0.f, 0, 0, 0, nullptr, nullptr, nullptr, 0, 0, 1.f, total_rows, ZP_IMPL_SIMT, dtype,
                             nullptr, 0, stream);
}
