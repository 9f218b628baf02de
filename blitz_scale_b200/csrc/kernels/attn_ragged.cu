// Paged attention of a ragged batch on the CUDA cores, general form: any head size, fp32 or 16-bit, any group size,
// sliding window with kept first tokens, soft-capped scores and a per-head sink in the softmax denominator.
//
//   visible(i, j) = j <= i and (i - j < window or j < keep_first)          window 0: everything
//   score         = cap * tanh(scale * q.k / cap)                           cap 0: scale * q.k
//   score        += bias[h][min(i - j, bias_len - 1)]                       no bias: nothing
//   out           = sum_j e^score_j v_j / (e^sink + sum_j e^score_j)        no sink: the plain softmax
//   out           = sigmoid(gate) * out                                     no gate: as it is
//
// `chunked`: the window is a chunk, visible(i, j) = j <= i and floor(i / window) = floor(j / window).  `sigmoid`: no softmax,
// out = sum_j sigmoid(score_j) v_j.
//
// Keys and values may differ in size, and values may be the first columns of the keys' rows (v_row: their pitch).
// It serves the 32-bit mode and head sizes that the tensor-core kernels do not take.  A warp owns one (token, query
// head): keys go over the lanes 32 at a time for the scores, head dimensions go over the lanes for the weighted sum.
// Only the blocks of 32 keys with a visible key are read.  Everything is fp32.
#include "launch.cuh"
#include "ptx.cuh"
#include "scalar.cuh"

namespace blitz {

constexpr int kRgWarps = 8;
constexpr int kRgMaxDim = 512;        // of a value head (accumulators in registers)
constexpr int kRgMaxQueryDim = 1024;  // of a query head (shared memory)

struct RaggedAttnParams {
  const void* q;
  const void *k_pool, *v_pool;  // row of token `off` of page n: n * page_rows + off
  const void* gate;             // [tokens][gate_stride], a column per query head, or null
  void* out;
  int64_t q_stride, out_stride, gate_stride;
  const int32_t* pos;
  const int32_t* tok_indptr;   // [rows + 1]; null: row t is token t
  const int32_t* page_indptr;  // [rows + 1]
  const int32_t* page_indices;
  const void* sink;
  const void* bias;   // [q_heads][bias_len] by distance, the last entry for all longer ones; or null
  int bias_len, v_row;
  int num_tokens, rows, q_heads, kv_heads, dim, vdim, page_size, page_rows, max_pages, window, keep_first, chunked, sigmoid;
  float scale, softcap;
  int* status;
};

template <typename T>
__global__ void __launch_bounds__(kRgWarps * 32) attn_ragged_kernel(const RaggedAttnParams p) {
  ptx::griddep_launch_dependents();
  ptx::griddep_wait();
  extern __shared__ float sq_all[];
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int64_t item = static_cast<int64_t>(blockIdx.x) * kRgWarps + warp;
  if (item >= static_cast<int64_t>(p.num_tokens) * p.q_heads) return;
  const int t = static_cast<int>(item / p.q_heads), h = static_cast<int>(item % p.q_heads);
  float* sq = sq_all + warp * p.dim;
  const int b = p.tok_indptr ? row_of_token(p.tok_indptr, p.rows, t) : t;
  const int pg0 = p.page_indptr[b], npages = p.page_indptr[b + 1] - pg0;
  const int D = p.dim, DV = p.vdim, i = p.pos[t];
  T* out = reinterpret_cast<T*>(p.out) + t * p.out_stride + static_cast<int64_t>(h) * DV;
  if (npages <= 0) {  // padding row
    for (int d = lane; d < DV; d += 32) stf<T>(out + d, 0.f);
    return;
  }
  const T* q = reinterpret_cast<const T*>(p.q) + t * p.q_stride + static_cast<int64_t>(h) * D;
  for (int d = lane; d < D; d += 32) sq[d] = ldf<T>(q + d) * p.scale;
  __syncwarp();
  const int kvh = h / (p.q_heads / p.kv_heads);
  const int64_t krow = static_cast<int64_t>(p.kv_heads) * D, vrow = static_cast<int64_t>(p.kv_heads) * p.v_row;
  const T* bias = p.bias ? reinterpret_cast<const T*>(p.bias) + static_cast<int64_t>(h) * p.bias_len : nullptr;
  const T* k_pool = reinterpret_cast<const T*>(p.k_pool) + static_cast<int64_t>(kvh) * D;
  const T* v_pool = reinterpret_cast<const T*>(p.v_pool) + static_cast<int64_t>(kvh) * p.v_row;
  // key j's row in the pools; -1 where the page table does not reach (reported)
  auto key_row = [&](int j) -> int {
    const int slot = j / p.page_size;
    const int page = slot < npages ? p.page_indices[pg0 + slot] : -1;
    if (page < 0 || page >= p.max_pages) {
      if (p.status) atomicCAS(p.status, 0, kStatusBadIndex);
      return -1;
    }
    return page * p.page_rows + j % p.page_size;
  };
  float acc[kRgMaxDim / 32];
#pragma unroll
  for (int d = 0; d < kRgMaxDim / 32; ++d) acc[d] = 0.f;
  float m = -INFINITY, l = 0.f;
  if (p.sink) {
    m = ldf<T>(reinterpret_cast<const T*>(p.sink) + h);
    l = 1.f;
  }
  const int lo = p.window > 0 ? (p.chunked ? i - i % p.window : max(0, i - p.window + 1)) : 0;  // first key of the window
  const int first = min(p.keep_first, lo);                     // kept keys in front of it
  const int nkeys = first + (i - lo + 1);                      // kept keys, then the window's
  for (int base = 0; base < nkeys; base += 32) {
    const int n = base + lane;
    const int row = n < nkeys ? key_row(n < first ? n : lo + n - first) : -1;
    float s = -INFINITY;
    if (row >= 0) {
      const T* kr = k_pool + row * krow;
      s = 0.f;
      for (int d = 0; d < D; ++d) s += sq[d] * ldf<T>(kr + d);
      if (p.softcap > 0.f) s = p.softcap * tanhf(s / p.softcap);
      if (bias) s += ldf<T>(bias + min(i - (n < first ? n : lo + n - first), p.bias_len - 1));
    }
    float w;
    if (p.sigmoid) {
      w = row >= 0 ? sigmoid_f(s) : 0.f;
      l = 1.f;
    } else {
      const float mx = fmaxf(m, warp_max(s));
      if (mx == -INFINITY) continue;
      const float corr = expf(m - mx);
      w = expf(s - mx);
      l = l * corr + warp_sum(w);
      m = mx;
#pragma unroll
      for (int d = 0; d < kRgMaxDim / 32; ++d) acc[d] *= corr;
    }
    const int cnt = min(32, nkeys - base);
    for (int k = 0; k < cnt; ++k) {
      const float wk = __shfl_sync(0xffffffffu, w, k);
      const int vr_row = __shfl_sync(0xffffffffu, row, k);
      if (vr_row < 0) continue;
      const T* vr = v_pool + vr_row * vrow;
#pragma unroll
      for (int d = 0; d < kRgMaxDim / 32; ++d) {
        const int c = d * 32 + lane;
        if (c < DV) acc[d] += wk * ldf<T>(vr + c);
      }
    }
  }
  float inv = l > 0.f ? 1.f / l : 0.f;
  if (p.gate) inv *= sigmoid_f(ldf<T>(reinterpret_cast<const T*>(p.gate) + t * p.gate_stride + h));
#pragma unroll
  for (int d = 0; d < kRgMaxDim / 32; ++d) {
    const int c = d * 32 + lane;
    if (c < DV) stf<T>(out + c, acc[d] * inv);
  }
}

}  // namespace blitz

extern "C" {
using namespace blitz;

// q: [tokens, q_stride], rotated; k_pool, v_pool: [max_pages][page_rows][kv_heads][dim or vdim] (see rope_store.cu) with
// every key up to a token's own position already stored; out: [tokens, out_stride].  Rows are the sequences of the step: tokens
// tok_indptr[r] .. tok_indptr[r + 1] (null: one token per row), pages page_indices[page_indptr[r] ..].  A row without
// pages gives zeros.  window 0 = unlimited; softcap 0 = none; sink may be null ([q_heads], activation type).  v_row: elements
// from a value head to the next one in a pool row (vdim, or dim where values are the first columns of the keys).  bias:
// [q_heads][bias_len] in the activation type, by distance, or null.
int blitz_attn_ragged(const void* q, int64_t q_stride, const void* k_pool, const void* v_pool, void* out, int64_t out_stride,
                      const int32_t* pos, const int32_t* tok_indptr, const int32_t* page_indptr,
                      const int32_t* page_indices, const void* sink, const void* bias, int bias_len, int v_row, const void* gate, int64_t gate_stride, int num_tokens,
                      int rows, int q_heads, int kv_heads, int dim, int vdim, int page_size, int page_rows, int max_pages,
                      int window, int keep_first, int chunked, int sigmoid, float scale, float softcap, int* status, int dtype, cudaStream_t stream) {
  if (num_tokens <= 0 || rows <= 0) return 0;
  if (dim <= 0 || vdim <= 0 || vdim > kRgMaxDim || dim > kRgMaxQueryDim || kv_heads <= 0 || q_heads % kv_heads != 0 || window < 0 ||
      keep_first < 0 || v_row < vdim || (chunked && (window < 1 || keep_first)) || (sigmoid && sink) || (bias && bias_len < 1))
    return -1;
  RaggedAttnParams p{q, k_pool, v_pool, gate, out, q_stride, out_stride, gate_stride, pos, tok_indptr, page_indptr, page_indices,
                     sink, bias, bias_len, v_row, num_tokens, rows, q_heads, kv_heads, dim, vdim, page_size, page_rows, max_pages, window, keep_first, chunked, sigmoid,
                     scale, softcap, status};
  const int64_t items = static_cast<int64_t>(num_tokens) * q_heads;
  const dim3 grid((unsigned)((items + kRgWarps - 1) / kRgWarps));
  cudaError_t e = cudaSuccess;
  BLITZ_DISPATCH_DTYPE3(dtype, (e = launch_pdl(attn_ragged_kernel<T>, grid, dim3(kRgWarps * 32),
                                               (size_t)kRgWarps * dim * sizeof(float), stream, p)));
  return (int)e;
}

}  // extern "C"
