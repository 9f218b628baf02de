// Per-head RMSNorm of queries and keys with the paged KV write, for attention without a rotation:
//
//   q <- q / rms(q) * w_q * temperature(pos)     in place       temperature(p) = 1 + coef * ln(floor((p + 1) / every) + 1)
//   k    k / rms(k) * w_k                        to the cache
//   v                                            to the cache
//
// A block per token.  Wide form: as many lanes per head as it has groups of eight dimensions (rounded up to a power of two);
// else a warp per head, one element at a time.
#include "launch.cuh"
#include "ptx.cuh"
#include "scalar.cuh"

namespace blitz {

struct NormStoreParams {
  void* q;            // [tokens][q_heads * dim], in place
  const void *k, *v;  // [tokens][kv_heads * dim or vdim]
  int64_t row;        // row pitch of q, k and v
  const void *q_w, *k_w;  // [dim]
  const int32_t *pos, *slot;
  void *k_pool, *v_pool;  // row of token `off` of page n: n * page_rows + off
  float eps, temp_coef;
  int temp_every;         // 0: no temperature
  int q_heads, kv_heads, dim, vdim, page_size, page_rows, max_pages;
  int* status;
};

template <typename T, bool WIDE>
__global__ void __launch_bounds__(256) norm_store_kernel(const NormStoreParams p) {
  ptx::griddep_launch_dependents();
  ptx::griddep_wait();
  const int t = blockIdx.x;
  int s = p.slot[t];
  if (s >= p.max_pages * p.page_size) {
    if (threadIdx.x == 0 && p.status) atomicCAS(p.status, 0, kStatusBadIndex);
    s = -1;
  }
  const int page = s >= 0 ? s / p.page_size : 0, off = s >= 0 ? s % p.page_size : 0;
  const int64_t at_row = static_cast<int64_t>(page) * p.page_rows + off;
  const int64_t vrow = static_cast<int64_t>(p.kv_heads) * p.vdim;
  T* kdst = reinterpret_cast<T*>(p.k_pool) + at_row * p.kv_heads * p.dim;
  T* vdst = reinterpret_cast<T*>(p.v_pool) + at_row * vrow;
  T* q = reinterpret_cast<T*>(p.q) + t * p.row;
  const T* k = reinterpret_cast<const T*>(p.k) + t * p.row;
  const T* v = reinterpret_cast<const T*>(p.v) + t * p.row;
  const T *qw = reinterpret_cast<const T*>(p.q_w), *kw = reinterpret_cast<const T*>(p.k_w);
  const float temp = p.temp_every > 0 ? 1.f + p.temp_coef * logf(static_cast<float>((p.pos[t] + 1) / p.temp_every + 1)) : 1.f;
  const float inv_dim = 1.f / static_cast<float>(p.dim);
  const int heads = p.q_heads + (s >= 0 ? p.kv_heads : 0);
  if (WIDE) {
    const int vec = p.dim >> 3;
    int lanes = 1;  // per head
    while (lanes < vec) lanes <<= 1;
    const int per = blockDim.x / lanes, c = threadIdx.x & (lanes - 1);
    for (int h0 = 0; h0 < heads; h0 += per) {  // the same number of turns for every lane of a warp
      const int head = h0 + threadIdx.x / lanes;
      const bool is_q = head < p.q_heads, on = head < heads && c < vec;
      const int64_t at = static_cast<int64_t>(is_q ? head : head - p.q_heads) * p.dim + c * 8;
      float x[8] = {}, ss = 0.f;
      if (on) ldf8<T>((is_q ? q : k) + at, x);
#pragma unroll
      for (int j = 0; j < 8; ++j) ss += x[j] * x[j];
      for (int o = lanes >> 1; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
      if (on) {
        const float f = rsqrtf(ss * inv_dim + p.eps) * (is_q ? temp : 1.f);
        float w[8];
        ldf8<T>((is_q ? qw : kw) + c * 8, w);
#pragma unroll
        for (int j = 0; j < 8; ++j) x[j] = x[j] * f * w[j];
        stf8<T>((is_q ? q : kdst) + at, x);
      }
    }
    if (s >= 0)
      for (int i = threadIdx.x * 8; i < vrow; i += blockDim.x * 8) {
        float x[8];
        ldf8<T>(v + i, x);
        stf8<T>(vdst + i, x);
      }
    return;
  }
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
  for (int head = warp; head < heads; head += warps) {
    const bool is_q = head < p.q_heads;
    const int64_t base = static_cast<int64_t>(is_q ? head : head - p.q_heads) * p.dim;
    const T* src = (is_q ? q : k) + base;
    T* dst = (is_q ? q : kdst) + base;
    const T* w = is_q ? qw : kw;
    float ss = 0.f;
    for (int d = lane; d < p.dim; d += 32) {
      const float x = ldf<T>(src + d);
      ss += x * x;
    }
    const float f = rsqrtf(warp_sum(ss) * inv_dim + p.eps) * (is_q ? temp : 1.f);
    for (int d = lane; d < p.dim; d += 32) stf<T>(dst + d, ldf<T>(src + d) * f * ldf<T>(w + d));
  }
  if (s >= 0)
    for (int i = threadIdx.x; i < vrow; i += blockDim.x) stf<T>(vdst + i, ldf<T>(v + i));
}

}  // namespace blitz

extern "C" {
using namespace blitz;

// Pools as for blitz_rope_store.  temp_every 0: queries are not scaled by their position.
int blitz_norm_store(void* q, const void* k, const void* v, int64_t row, const void* q_w, const void* k_w, float eps, float temp_coef,
                     int temp_every, const int32_t* pos, const int32_t* slot, void* k_pool, void* v_pool, int num_tokens, int q_heads,
                     int kv_heads, int dim, int vdim, int page_size, int page_rows, int max_pages, int* status, int dtype,
                     cudaStream_t stream) {
  if (num_tokens <= 0) return 0;
  if (dim <= 0 || vdim <= 0 || q_heads <= 0 || kv_heads <= 0 || temp_every < 0 || !q || !k || !v || !q_w || !k_w) return -1;
  NormStoreParams p{q, k, v, row, q_w, k_w, pos, slot, k_pool, v_pool, eps, temp_coef, temp_every,
                    q_heads, kv_heads, dim, vdim, page_size, page_rows, max_pages, status};
  const uintptr_t al = dtype == 2 ? 32 : 16;
  bool wide = ((dim | vdim | row) & 7) == 0 && dim <= 256;
  for (const void* x : {(const void*)q, k, v, q_w, k_w, (const void*)k_pool, (const void*)v_pool})
    wide = wide && (reinterpret_cast<uintptr_t>(x) % al) == 0;
  const dim3 grid(num_tokens), block((q_heads + kv_heads) * dim <= 2048 ? 128 : 256);
  auto go = [&](auto type) {
    using T = decltype(type);
    return wide ? launch_pdl(norm_store_kernel<T, true>, grid, block, 0, stream, p)
                : launch_pdl(norm_store_kernel<T, false>, grid, block, 0, stream, p);
  };
  cudaError_t e = cudaSuccess;
  BLITZ_DISPATCH_DTYPE3(dtype, (e = go(T{})));
  return (int)e;
}

}  // extern "C"
