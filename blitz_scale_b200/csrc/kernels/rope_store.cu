// Rotary embedding of q and k with the paged KV write, general form: rotation of the first `rot_dims` dimensions of a
// head (0 = none), interleaved (dimensions 2i, 2i + 1 are a pair) or half-split pairs, any head size, fp32 or 16-bit
// activations, and a choice of what the value plane of the cache receives: the value columns of the projection, or
// the keys as projected, before rotation (models without a value projection).
//
// (elementwise.cu's rope_kv_store is the special case of a fully rotated half-split head with a value projection.)
//
// The angle of pair i at position p is p * f_i.  The caller passes f_i as an unevaluated sum of two fp32 numbers;
// the product's rounding error and the low part are put back through the addition theorem, so the angle is good to
// fp32 rounding of its sine and cosine at any position instead of losing a digit per factor 10 of p.
#include "launch.cuh"
#include "ptx.cuh"
#include "scalar.cuh"

namespace blitz {

struct RopeStoreParams {
  void* q;           // [tokens][q_heads * dim], rotated in place
  const void* k;     // [tokens][kv_heads * dim]
  const void* v;     // [tokens][kv_heads * dim] or null: the value plane receives the keys before rotation
  int64_t row;       // row pitch of q, k and v
  const int32_t* pos;
  const int32_t* slot;
  void* kv;
  const float2* freq;  // [rot_dims / 2] (high, low)
  int q_heads, kv_heads, dim, rot_dims, interleaved, page_size, max_pages, wide;
  int* status;
};

template <typename T>
__global__ void rope_store_kernel(const RopeStoreParams p) {
  ptx::griddep_launch_dependents();
  ptx::griddep_wait();
  extern __shared__ float s_ang[];  // [rot_dims / 2] cos, [rot_dims / 2] sin
  const int t = blockIdx.x;
  const int half = p.rot_dims >> 1;
  const float pos = static_cast<float>(p.pos[t]);
  for (int i = threadIdx.x; i < half; i += blockDim.x) {
    const float2 f = p.freq[i];
    const float a = pos * f.x;
    const float err = fmaf(pos, f.x, -a) + pos * f.y;
    float sn, cs;
    sincosf(a, &sn, &cs);
    const float c_err = 1.f - 0.5f * err * err;  // cos and sin of the small angle `err`, to second order
    s_ang[i] = cs * c_err - err * sn;
    s_ang[half + i] = sn * c_err + err * cs;
  }
  __syncthreads();
  int s = p.slot[t];
  if (s >= p.max_pages * p.page_size) {
    if (threadIdx.x == 0 && p.status) atomicCAS(p.status, 0, kStatusBadIndex);
    s = -1;
  }
  const int page = s >= 0 ? s / p.page_size : 0, off = s >= 0 ? s % p.page_size : 0;
  const int64_t kvrow = static_cast<int64_t>(p.kv_heads) * p.dim;
  const int64_t plane = p.page_size * kvrow;
  T* kdst = reinterpret_cast<T*>(p.kv) + static_cast<int64_t>(page) * 2 * plane + off * kvrow;
  T* vdst = kdst + plane;
  T* q = reinterpret_cast<T*>(p.q) + t * p.row;
  const T* k = reinterpret_cast<const T*>(p.k) + t * p.row;
  if (p.wide) {
    // interleaved heads: eight elements (four pairs) per access; dimensions that pass unchanged ride along
    const int vec = p.dim >> 3;
    for (int it = threadIdx.x; it < (p.q_heads + p.kv_heads) * vec; it += blockDim.x) {
      const int head = it / vec, d0 = (it - head * vec) * 8;
      const bool is_q = head < p.q_heads;
      if ((!is_q && s < 0) || (is_q && d0 >= p.rot_dims)) continue;
      const int64_t at = static_cast<int64_t>(is_q ? head : head - p.q_heads) * p.dim + d0;
      float x[8], y[8];
      ldf8<T>((is_q ? q : k) + at, x);
#pragma unroll
      for (int j = 0; j < 8; j += 2) {
        const int i = (d0 + j) >> 1;
        const bool rot = d0 + j < p.rot_dims;
        const float cs = rot ? s_ang[i] : 1.f, sn = rot ? s_ang[half + i] : 0.f;
        y[j] = x[j] * cs - x[j + 1] * sn;
        y[j + 1] = x[j + 1] * cs + x[j] * sn;
      }
      stf8<T>((is_q ? q : kdst) + at, y);
      if (!is_q && p.v == nullptr) stf8<T>(vdst + at, x);
    }
    if (p.v != nullptr && s >= 0) {
      const T* v = reinterpret_cast<const T*>(p.v) + t * p.row;
      for (int i = threadIdx.x * 8; i < kvrow; i += blockDim.x * 8) {
        float x[8];
        ldf8<T>(v + i, x);
        stf8<T>(vdst + i, x);
      }
    }
    return;
  }
  // Rotated pairs of q and k.  With two-element accesses only where pairs are neighbours and rows even.
  const bool vec = p.interleaved && ((p.dim | p.row) & 1) == 0;
  const int items = (p.q_heads + p.kv_heads) * half;
  for (int it = threadIdx.x; it < items; it += blockDim.x) {
    const int head = it / half, i = it - head * half;
    const float cs = s_ang[i], sn = s_ang[half + i];
    const int iu = p.interleaved ? 2 * i : i, iv = p.interleaved ? 2 * i + 1 : i + half;
    const bool is_q = head < p.q_heads;
    const int64_t base = static_cast<int64_t>(is_q ? head : head - p.q_heads) * p.dim;
    if (!is_q && s < 0) continue;
    const T* src = (is_q ? q : k) + base;
    T* dst = (is_q ? q : kdst) + base;
    float u, v;
    if (vec) {
      const float2 f = ldf2<T>(src + iu);
      u = f.x; v = f.y;
    } else {
      u = ldf<T>(src + iu); v = ldf<T>(src + iv);
    }
    const float ru = u * cs - v * sn, rv = v * cs + u * sn;
    if (vec) {
      stf2<T>(dst + iu, ru, rv);
    } else {
      stf<T>(dst + iu, ru);
      stf<T>(dst + iv, rv);
    }
    if (!is_q && p.v == nullptr) {
      if (vec) {
        stf2<T>(vdst + base + iu, u, v);
      } else {
        stf<T>(vdst + base + iu, u);
        stf<T>(vdst + base + iv, v);
      }
    }
  }
  if (s < 0) return;
  const int rest = p.dim - p.rot_dims;  // dimensions that pass unchanged: keys, and values taken from them
  for (int it = threadIdx.x; it < p.kv_heads * rest; it += blockDim.x) {
    const int64_t at = static_cast<int64_t>(it / rest) * p.dim + p.rot_dims + it % rest;
    const T x = k[at];
    kdst[at] = x;
    if (p.v == nullptr) vdst[at] = x;
  }
  if (p.v != nullptr) {
    const T* v = reinterpret_cast<const T*>(p.v) + t * p.row;
    for (int i = threadIdx.x; i < kvrow; i += blockDim.x) vdst[i] = v[i];
  }
}

}  // namespace blitz

extern "C" {
using namespace blitz;

int blitz_rope_store(void* q, const void* k, const void* v, int64_t row, const int32_t* pos, const int32_t* slot,
                     void* kv_layer, const void* freq, int num_tokens, int q_heads, int kv_heads, int dim, int rot_dims,
                     int interleaved, int page_size, int max_pages, int* status, int dtype, cudaStream_t stream) {
  if (num_tokens <= 0) return 0;
  if (rot_dims < 0 || (rot_dims & 1) || rot_dims > dim || rot_dims > 4096 || (rot_dims > 0 && freq == nullptr)) return -1;
  RopeStoreParams p{q, k, v, row, pos, slot, kv_layer, reinterpret_cast<const float2*>(freq), q_heads, kv_heads, dim,
                    rot_dims, interleaved, page_size, max_pages, 0, status};
  const uintptr_t al = dtype == 2 ? 32 : 16;
  p.wide = interleaved && ((dim | row) & 7) == 0;
  for (const void* x : {(const void*)q, k, v, (const void*)kv_layer}) p.wide = p.wide && (reinterpret_cast<uintptr_t>(x) % al) == 0;
  cudaError_t e = cudaSuccess;
  BLITZ_DISPATCH_DTYPE3(dtype, (e = launch_pdl(rope_store_kernel<T>, dim3(num_tokens), dim3(p.wide && (q_heads + kv_heads) * dim <= 2048 ? 128 : 256),
                                               (size_t)rot_dims * sizeof(float), stream, p)));
  return (int)e;
}

}  // extern "C"
