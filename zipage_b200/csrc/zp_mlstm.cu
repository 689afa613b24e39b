// Matrix-memory (mLSTM) mixer, token by token: the decode kernel, also used for prompts in fp32.
//
// HBM-bound: a decoded token reads and writes the head's whole fp32 state once.  One block per (head,
// sequence), or, for small batches, per value tile of a head; the blocks of a head then form a cluster,
// because the output norm needs the sum of squares over all value dims (exchanged through distributed shared
// memory).  A thread owns four
// adjacent value columns and every nrg-th row of the state, so a warp moves whole rows of a tile with
// 16-byte accesses.  Gates, state update, read-out, normaliser, head norm and output gate are one
// launch.  With several tokens per sequence the block loops; each thread re-reads only what it wrote.
#include "zp_mlstm.cuh"

namespace zp {

constexpr int ML_THREADS = 256;
constexpr int ML_BATCH = 4;    // state rows of a batch; two batches are in flight per thread

template <typename T>
__global__ void __launch_bounds__(ML_THREADS, 2) mlstm_recurrent_kernel(const MlstmArgs a) {
  extern __shared__ __align__(16) float sm[];
  __shared__ float red[32];
  __shared__ float xsum[2];      // this block's sum of squares, by token parity
  const int vt = blockIdx.x, h = blockIdx.y, b = blockIdx.z, tid = threadIdx.x;
  const MlstmSeq sq = mlstm_seq(a, b);
  if (sq.count == 0) return;     // the same decision in every block of the cluster
  const int c0 = vt * a.VT, ncg = a.VT / 4, nrg = ML_THREADS / ncg;
  float* sq_ = sm;               // [dim] q
  float* sk = sq_ + a.dim;       // [dim] k
  float* sn = sk + a.dim;        // [dim] n, this block's copy
  float* part = sm + ((3 * a.dim + 3) & ~3);   // [nrg][VT] partial read-outs
  const int cg = tid % ncg, rg = tid / ncg;
  const int col = c0 + 4 * cg;
  const bool mine = rg < nrg && col < a.VP;
  const int64_t head = (int64_t)sq.slot * a.H + h;
  float* S = a.S + head * a.dim * a.VP + col;
  float m = sq.fresh ? 0.f : a.m[head];
  for (int d = tid; d < a.dim; d += ML_THREADS) sn[d] = sq.fresh ? 0.f : a.n[head * a.dim + d];
  bool zero = sq.fresh;
  const T* qb = reinterpret_cast<const T*>(a.q);
  const T* kb = reinterpret_cast<const T*>(a.k);
  const T* vb = reinterpret_cast<const T*>(a.v);
  const T* gb = reinterpret_cast<const T*>(a.g);

  for (int t = 0; t < sq.count; ++t) {
    const int64_t row = sq.row0 + t;
    // two batches of state rows alternate: one is updated while the other's loads are in flight, the
    // first while the gates are computed
    float4 sa[ML_BATCH], sb[ML_BATCH];
    const int step = nrg * ML_BATCH;
    auto load_rows = [&](float4 (&s)[ML_BATCH], int r0) {
#pragma unroll
      for (int u = 0; u < ML_BATCH; ++u) {
        const int r = r0 + u * nrg;
        s[u] = (r < a.dim && !zero) ? *reinterpret_cast<const float4*>(S + (int64_t)r * a.VP) : make_float4(0.f, 0.f, 0.f, 0.f);
      }
    };
    if (mine) load_rows(sa, rg);
    const float gi = log_input_gate(a, row, h), gf = log_forget_gate(a, row, h);
    const float m_new = fmaxf(gf + m, gi);
    const float keep = expf(gf + m - m_new), add = expf(gi - m_new);
    m = m_new;
    float nq = 0.f;
    for (int d = tid; d < a.dim; d += ML_THREADS) {
      const float qv = Elem<T>::to_f32(qb[row * a.row_stride + (int64_t)h * a.dim + d]) * a.qscale;
      const float kv = Elem<T>::to_f32(kb[row * a.row_stride + (int64_t)h * a.dim + d]);
      const float nn = fmaf(keep, sn[d], add * kv);
      sq_[d] = qv; sk[d] = kv; sn[d] = nn;
      nq = fmaf(nn, qv, nq);
    }
    nq = block_sum(nq, red);     // (its barriers also publish q and k)
    if (mine) {
      float v[4], acc[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
      for (int j = 0; j < 4; ++j)
        v[j] = col + j < a.vdim ? add * Elem<T>::to_f32(vb[row * a.row_stride + (int64_t)h * a.vdim + col + j]) : 0.f;
      auto update_rows = [&](float4 (&s)[ML_BATCH], int r0) {
#pragma unroll
        for (int u = 0; u < ML_BATCH; ++u) {
          const int r = r0 + u * nrg;
          if (r < a.dim) {
            const float kr = sk[r], qr = sq_[r];
            s[u].x = fmaf(keep, s[u].x, kr * v[0]); s[u].y = fmaf(keep, s[u].y, kr * v[1]);
            s[u].z = fmaf(keep, s[u].z, kr * v[2]); s[u].w = fmaf(keep, s[u].w, kr * v[3]);
            acc[0] = fmaf(s[u].x, qr, acc[0]); acc[1] = fmaf(s[u].y, qr, acc[1]);
            acc[2] = fmaf(s[u].z, qr, acc[2]); acc[3] = fmaf(s[u].w, qr, acc[3]);
            *reinterpret_cast<float4*>(S + (int64_t)r * a.VP) = s[u];
          }
        }
      };
      for (int r0 = rg; r0 < a.dim; r0 += 2 * step) {
        load_rows(sb, r0 + step);
        update_rows(sa, r0);
        load_rows(sa, r0 + 2 * step);
        update_rows(sb, r0 + step);
      }
      *reinterpret_cast<float4*>(part + rg * a.VT + 4 * cg) = make_float4(acc[0], acc[1], acc[2], acc[3]);
    }
    zero = false;
    __syncthreads();
    const float den = 1.f / (fmaxf(fabsf(nq), expf(-m)) + MLSTM_DEN_EPS);
    float o[4], ss = 0.f;        // columns tid, tid + 256, ... of the tile (VT <= 1024)
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int c = tid + j * ML_THREADS;
      o[j] = 0.f;
      if (c < a.VT && c0 + c < a.vdim) {
        for (int r = 0; r < nrg; ++r) o[j] += part[r * a.VT + c];
        o[j] *= den;
        ss = fmaf(o[j], o[j], ss);
      }
    }
    ss = block_sum(ss, red);
    if (cluster_size() > 1) {
      if (tid == 0) xsum[t & 1] = ss;
      cluster_sync();
      ss = 0.f;
      for (uint32_t r = 0; r < cluster_size(); ++r) ss += ld_cluster(&xsum[t & 1], r);
    }
    const float rr = 1.f / sqrtf(ss / (float)a.vdim + a.eps);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int c = tid + j * ML_THREADS;
      if (c < a.VT && c0 + c < a.vdim) {
        const int64_t e = (int64_t)h * a.vdim + c0 + c;
        const float g = Elem<T>::to_f32(gb[row * a.row_stride + e]);
        reinterpret_cast<T*>(a.out)[row * a.out_stride + e] =
            Elem<T>::from_f32(o[j] * rr * a.norm_weight[e] / (1.f + expf(-g)));
      }
    }
    __syncthreads();             // q, k and the partial sums are rewritten by the next token
  }
  if (cluster_size() > 1) cluster_sync();   // peers may still be reading xsum; n and m were read by all before
  if (vt == 0) {
    for (int d = tid; d < a.dim; d += ML_THREADS) a.n[head * a.dim + d] = sn[d];
    if (tid == 0) a.m[head] = m;
  }
}

template <typename T>
static int launch_recurrent(MlstmArgs a, cudaStream_t st) {
  // a whole head per block, or, when the batch leaves most SMs without one, up to eight value tiles
  int tiles = (a.VP + 1023) / 1024;
  while (2 * tiles <= 8 && (int64_t)a.B * a.H * tiles < 148 * 2 && a.VP / tiles > 64) tiles *= 2;
  a.VT = ((a.VP + tiles - 1) / tiles + 3) & ~3;
  tiles = (a.VP + a.VT - 1) / a.VT;
  const int nrg = ML_THREADS / (a.VT / 4);
  const size_t smem = sizeof(float) * (((3 * a.dim + 3) & ~3) + (size_t)nrg * a.VT);
  cudaLaunchConfig_t cfg = {};
  cfg.gridDim = dim3(tiles, a.H, a.B);
  cfg.blockDim = dim3(ML_THREADS);
  cfg.dynamicSmemBytes = smem;
  cfg.stream = st;
  cudaLaunchAttribute at[1];
  at[0].id = cudaLaunchAttributeClusterDimension;
  at[0].val.clusterDim.x = tiles; at[0].val.clusterDim.y = 1; at[0].val.clusterDim.z = 1;
  cfg.attrs = at; cfg.numAttrs = 1;
  cudaError_t e = cudaLaunchKernelEx(&cfg, mlstm_recurrent_kernel<T>, a);
  if (e != cudaSuccess) { set_error("zp_mlstm: %s", cudaGetErrorString(e)); return ZP_ERR_CUDA; }
  return check_launch("zp_mlstm");
}

// chunked tensor-core prefill (zp_mlstm_chunk.cu)
bool mlstm_chunk_supports(const MlstmArgs& a, int dtype);
int mlstm_chunk(const MlstmArgs& a, cudaStream_t st);
// its tcgen05 form (zp_mlstm_tc.cu)
bool mlstm_tc_supports(const MlstmArgs& a, int total_rows, int dtype);
int mlstm_tc(const MlstmArgs& a, int total_rows, cudaStream_t st);

}  // namespace zp

extern "C" int zp_mlstm(const void* q, const void* k, const void* v, const void* g, const float* gates,
                        const float* gate_bias, const float* norm_weight, const int32_t* cu_seqlens_q,
                        const int32_t* context_lens, const int32_t* slots, float* state, float* state_n,
                        float* state_m, void* out, int B, int H, int dim, int vdim, int VP, int n_slots,
                        int64_t row_stride, int64_t gates_stride, int64_t out_stride, float qscale, float gate_cap,
                        float eps, int total_rows, int impl, int dtype, void* stream) {
  if (B == 0) return ZP_OK;
  ZP_REQUIRE(q && k && v && g && gates && gate_bias && norm_weight && context_lens && slots && state && state_n &&
                 state_m && out, "zp_mlstm: null pointer");
  ZP_REQUIRE(H > 0 && dim > 0 && dim <= 2048 && vdim > 0 && VP >= vdim && VP % 4 == 0 && VP <= 8192 && n_slots > 0,
             "zp_mlstm: bad sizes");
  ZP_REQUIRE(B <= 65535 && H <= 65535 && gate_cap > 0.f, "zp_mlstm: bad sizes");
  ZP_REQUIRE((uintptr_t)state % 16 == 0, "zp_mlstm: the state must be 16-byte aligned");
  zp::MlstmArgs a;
  a.q = q; a.k = k; a.v = v; a.g = g; a.gates = gates; a.gate_bias = gate_bias; a.norm_weight = norm_weight;
  a.cu_q = cu_seqlens_q; a.context_lens = context_lens; a.slots = slots; a.S = state; a.n = state_n; a.m = state_m;
  a.out = out; a.B = B; a.H = H; a.dim = dim; a.vdim = vdim; a.VP = VP; a.n_slots = n_slots; a.VT = 0;
  a.row_stride = row_stride; a.gates_stride = gates_stride; a.out_stride = out_stride;
  a.qscale = qscale; a.cap = gate_cap; a.eps = eps;
  cudaStream_t st = (cudaStream_t)stream;
  const bool tc = cu_seqlens_q && zp::mlstm_tc_supports(a, total_rows, dtype);
  if (impl == ZP_IMPL_TCGEN05 && !tc) {
    zp::set_error("zp_mlstm: the tcgen05 kernel needs bf16 portions, a key size of 128, a value size that is a multiple of "
                  "128 and 16-byte aligned rows");
    return ZP_ERR_UNSUPPORTED;
  }
  // (chunks of 128 tokens: not for portions of a few)
  if (tc && (impl == ZP_IMPL_TCGEN05 || (impl == ZP_IMPL_AUTO && total_rows >= 64 * B))) return zp::mlstm_tc(a, total_rows, st);
  if (cu_seqlens_q && impl != ZP_IMPL_SIMT && zp::mlstm_chunk_supports(a, dtype)) return zp::mlstm_chunk(a, st);
  ZP_DISPATCH_DTYPE(dtype, T, { return zp::launch_recurrent<T>(a, st); });
  return ZP_OK;
}
