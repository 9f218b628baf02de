// Latent attention: what happens between its projections.  Keys and values of all heads come from one latent vector per
// token, and a rotated key part is shared by all heads; only these two are cached ([pages][page][rank + rot]).
//
//   latent_store    queries' latent: RMSNorm in place; keys' latent: RMSNorm, to the cache; rotated key part, to the cache
//   latent_rotate   the last `rot` dimensions of every query head, in place or to where the absorbed queries are
//   latent_gather   whole pages, back to back (prompts: the operand of the product that expands keys and values)
//
// Rotation pairs are (i, i + rot / 2), or (2 i, 2 i + 1); frequencies are unevaluated sums of two fp32 numbers as in rope_store.cu.
#include "launch.cuh"
#include "ptx.cuh"
#include "scalar.cuh"

namespace blitz {

__device__ __forceinline__ float2 latent_angle(float pos, float2 f) {  // (cos, sin) of pos * (f.x + f.y)
  const float a = pos * f.x;
  const float err = fmaf(pos, f.x, -a) + pos * f.y;
  float sn, cs;
  sincosf(a, &sn, &cs);
  const float c_err = 1.f - 0.5f * err * err;
  return make_float2(cs * c_err - err * sn, sn * c_err + err * cs);
}

struct LatentStoreParams {
  void* cq;         // [tokens][row pitch], q_rank columns, in place (null: no latent of queries)
  const void* ckv;  // [tokens][row pitch], rank + rot columns
  int64_t row;
  const void *cq_w, *ckv_w;
  const int32_t *pos, *slot;
  void* pool;       // [max_pages][page_size][rank + rot]
  const float2* freq;
  float eps;
  int q_rank, rank, rot, interleaved, page_size, max_pages;
  int* status;
};

template <typename T, bool WIDE>
__global__ void __launch_bounds__(256) latent_store_kernel(const LatentStoreParams p) {
  ptx::griddep_launch_dependents();
  ptx::griddep_wait();
  __shared__ float red[2][33];
  const int t = blockIdx.x;
  int s = p.slot[t];
  if (s >= p.max_pages * p.page_size) {
    if (threadIdx.x == 0 && p.status) atomicCAS(p.status, 0, kStatusBadIndex);
    s = -1;
  }
  constexpr int V = WIDE ? 8 : 1;
  T* cq = reinterpret_cast<T*>(p.cq) + t * p.row;
  const T* ckv = reinterpret_cast<const T*>(p.ckv) + t * p.row;
  T* dst = reinterpret_cast<T*>(p.pool) + static_cast<int64_t>(s < 0 ? 0 : s) * (p.rank + p.rot);
  auto squares = [&](const T* x, int n) {
    float ss = 0.f;
    for (int i = threadIdx.x * V; i < n; i += blockDim.x * V) {
      if (WIDE) {
        float v[8];
        ldf8<T>(x + i, v);
#pragma unroll
        for (int j = 0; j < 8; ++j) ss += v[j] * v[j];
      } else {
        const float v = ldf<T>(x + i);
        ss += v * v;
      }
    }
    return ss;
  };
  const int q_rank = p.cq ? p.q_rank : 0;
  const float sq = block_sum(squares(cq, q_rank), red[0]), sk = block_sum(squares(ckv, p.rank), red[1]);
  auto scaled = [&](const T* x, const void* w_, T* out, int n, float ss) {
    const float f = rsqrtf(ss / static_cast<float>(n) + p.eps);
    const T* w = reinterpret_cast<const T*>(w_);
    for (int i = threadIdx.x * V; i < n; i += blockDim.x * V) {
      if (WIDE) {
        float v[8], g[8];
        ldf8<T>(x + i, v);
        ldf8<T>(w + i, g);
#pragma unroll
        for (int j = 0; j < 8; ++j) v[j] = v[j] * f * g[j];
        stf8<T>(out + i, v);
      } else {
        stf<T>(out + i, ldf<T>(x + i) * f * ldf<T>(w + i));
      }
    }
  };
  if (q_rank > 0) scaled(cq, p.cq_w, cq, q_rank, sq);
  if (s < 0) return;
  scaled(ckv, p.ckv_w, dst, p.rank, sk);
  const int half = p.rot >> 1;
  const float pos = static_cast<float>(p.pos[t]);
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    const float2 a = latent_angle(pos, p.freq[i]);
    const int iu = p.rank + (p.interleaved ? 2 * i : i), iv = p.interleaved ? iu + 1 : iu + half;
    const float u = ldf<T>(ckv + iu), v = ldf<T>(ckv + iv);
    stf<T>(dst + iu, u * a.x - v * a.y);
    stf<T>(dst + iv, v * a.x + u * a.y);
  }
}

struct LatentRotateParams {
  const void* q;  // [tokens][row]: heads of dim + rot columns
  void* out;      // head h's rotated part at h * out_step of a row
  int64_t row, out_row;
  const int32_t* pos;
  const float2* freq;
  int heads, dim, rot, out_step;
};

template <typename T, int V, bool PAIRS>
__global__ void __launch_bounds__(256) latent_rotate_kernel(const LatentRotateParams p) {
  ptx::griddep_launch_dependents();
  ptx::griddep_wait();
  extern __shared__ float s_ang[];  // [rot / 2] cos, [rot / 2] sin
  const int t = blockIdx.x, half = p.rot >> 1, vec = half / V;
  const float pos = static_cast<float>(p.pos[t]);
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    const float2 a = latent_angle(pos, p.freq[i]);
    s_ang[i] = a.x;
    s_ang[half + i] = a.y;
  }
  __syncthreads();
  for (int it = threadIdx.x; it < p.heads * vec; it += blockDim.x) {
    const int h = it / vec, i = (it - h * vec) * V;
    const T* src = reinterpret_cast<const T*>(p.q) + t * p.row + static_cast<int64_t>(h) * (p.dim + p.rot) + p.dim + (PAIRS ? 2 * i : i);
    T* dst = reinterpret_cast<T*>(p.out) + t * p.out_row + static_cast<int64_t>(h) * p.out_step + (PAIRS ? 2 * i : i);
    if constexpr (PAIRS) {
      float x[2 * V];
      if constexpr (V == 4) {
        ldf8<T>(src, x);
      } else {
        x[0] = ldf<T>(src);
        x[1] = ldf<T>(src + 1);
      }
#pragma unroll
      for (int j = 0; j < V; ++j) {
        const float cs = s_ang[i + j], sn = s_ang[half + i + j], u = x[2 * j], v = x[2 * j + 1];
        x[2 * j] = u * cs - v * sn;
        x[2 * j + 1] = v * cs + u * sn;
      }
      if constexpr (V == 4) {
        stf8<T>(dst, x);
      } else {
        stf<T>(dst, x[0]);
        stf<T>(dst + 1, x[1]);
      }
      continue;
    }
    float u[V], v[V];
    if constexpr (V == 8) {
      ldf8<T>(src, u);
      ldf8<T>(src + half, v);
    } else {
      u[0] = ldf<T>(src);
      v[0] = ldf<T>(src + half);
    }
#pragma unroll
    for (int j = 0; j < V; ++j) {
      const float cs = s_ang[i + j], sn = s_ang[half + i + j], x = u[j];
      u[j] = x * cs - v[j] * sn;
      v[j] = v[j] * cs + x * sn;
    }
    if constexpr (V == 8) {
      stf8<T>(dst, u);
      stf8<T>(dst + half, v);
    } else {
      stf<T>(dst, u[0]);
      stf<T>(dst + half, v[0]);
    }
  }
}

__global__ void __launch_bounds__(256) latent_gather_kernel(const uint4* pool, const int32_t* pages, uint4* out, int per_page, int max_pages,
                                                            int* status) {
  ptx::griddep_launch_dependents();
  ptx::griddep_wait();
  int page = pages[blockIdx.x];
  if (page < 0 || page >= max_pages) {
    if (threadIdx.x == 0 && status) atomicCAS(status, 0, kStatusBadIndex);
    page = 0;
  }
  const uint4* src = pool + static_cast<int64_t>(page) * per_page;
  uint4* dst = out + static_cast<int64_t>(blockIdx.x) * per_page;
  for (int i = blockIdx.y * blockDim.x + threadIdx.x; i < per_page; i += gridDim.y * blockDim.x) dst[i] = src[i];
}

}  // namespace blitz

extern "C" {
using namespace blitz;

// cq (q_rank columns, may be null) and ckv (rank + rot columns): column ranges of one projection with row pitch `row`.
int blitz_latent_store(void* cq, const void* ckv, int64_t row, const void* cq_w, const void* ckv_w, const int32_t* pos, const int32_t* slot,
                       void* pool, const void* freq, float eps, int num_tokens, int q_rank, int rank, int rot, int interleaved, int page_size,
                       int max_pages, int* status, int dtype, cudaStream_t stream) {
  if (num_tokens <= 0) return 0;
  if (rank <= 0 || rot < 0 || (rot & 1) || (rot > 0 && freq == nullptr) || (cq && (q_rank <= 0 || cq_w == nullptr))) return -1;
  LatentStoreParams p{cq, ckv, row, cq_w, ckv_w, pos, slot, pool, reinterpret_cast<const float2*>(freq), eps,
                      q_rank, rank, rot, interleaved, page_size, max_pages, status};
  const uintptr_t al = dtype == 2 ? 32 : 16;
  bool wide = ((q_rank | rank | rot | row) & 7) == 0;
  for (const void* x : {(const void*)cq, ckv, cq_w, ckv_w, (const void*)pool}) wide = wide && (reinterpret_cast<uintptr_t>(x) % al) == 0;
  const int n = (q_rank > rank ? q_rank : rank) / (wide ? 8 : 1);
  const dim3 grid(num_tokens), block(n <= 64 ? 64 : n <= 128 ? 128 : 256);
  auto go = [&](auto type) {
    using T = decltype(type);
    return wide ? launch_pdl(latent_store_kernel<T, true>, grid, block, 0, stream, p)
                : launch_pdl(latent_store_kernel<T, false>, grid, block, 0, stream, p);
  };
  cudaError_t e = cudaSuccess;
  BLITZ_DISPATCH_DTYPE3(dtype, (e = go(T{})));
  return (int)e;
}

// q: heads of dim + rot columns; head h's rotated part goes to out + h * out_step (its first rotated column).
int blitz_latent_rotate(const void* q, int64_t row, void* out, int64_t out_row, int out_step, const int32_t* pos, const void* freq,
                        int num_tokens, int heads, int dim, int rot, int interleaved, int dtype, cudaStream_t stream) {
  if (num_tokens <= 0 || rot == 0) return 0;
  if (heads <= 0 || dim < 0 || rot < 0 || (rot & 1) || rot > 4096 || freq == nullptr) return -1;
  LatentRotateParams p{q, out, row, out_row, pos, reinterpret_cast<const float2*>(freq), heads, dim, rot, out_step};
  const uintptr_t al = dtype == 2 ? 32 : 16;
  const bool wide = (rot & (interleaved ? 7 : 15)) == 0 && ((dim | row | out_row | out_step) & 7) == 0 && reinterpret_cast<uintptr_t>(q) % al == 0 &&
                    reinterpret_cast<uintptr_t>(out) % al == 0;
  const int items = heads * (rot / 2) / (wide ? (interleaved ? 4 : 8) : 1);
  const dim3 grid(num_tokens), block(items <= 64 ? 64 : items <= 128 ? 128 : 256);
  const size_t smem = (size_t)rot * sizeof(float);
  auto go = [&](auto type) {
    using T = decltype(type);
    if (interleaved)
      return wide ? launch_pdl(latent_rotate_kernel<T, 4, true>, grid, block, smem, stream, p)
                  : launch_pdl(latent_rotate_kernel<T, 1, true>, grid, block, smem, stream, p);
    return wide ? launch_pdl(latent_rotate_kernel<T, 8, false>, grid, block, smem, stream, p)
                : launch_pdl(latent_rotate_kernel<T, 1, false>, grid, block, smem, stream, p);
  };
  cudaError_t e = cudaSuccess;
  BLITZ_DISPATCH_DTYPE3(dtype, (e = go(T{})));
  return (int)e;
}

// out [num_pages][page bytes] = the named pages of the pool; page_bytes: a multiple of 16.
int blitz_latent_gather(const void* pool, const int32_t* pages, void* out, int num_pages, int64_t page_bytes, int max_pages, int* status,
                        cudaStream_t stream) {
  if (num_pages <= 0) return 0;
  if (page_bytes & 15) return -1;
  const int per = (int)(page_bytes / 16);
  const int y = per > 2048 ? 4 : 1;
  return (int)launch_pdl(latent_gather_kernel, dim3(num_pages, y), dim3(256), 0, stream, reinterpret_cast<const uint4*>(pool), pages,
                         reinterpret_cast<uint4*>(out), per, max_pages, status);
}

}  // extern "C"
