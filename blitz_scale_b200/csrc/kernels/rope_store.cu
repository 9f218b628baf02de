// Rotary embedding of q and k with the paged KV write, general form: rotation of the first `rot_dims` dimensions of a
// head (0 = none), interleaved (dimensions 2i, 2i + 1 are a pair) or half-split pairs (i, i + rot_dims / 2), any head size,
// values of another size than the keys, fp32 or 16-bit activations, and a choice of what the value plane of the cache
// receives: the value columns of the projection, or the keys as projected, before rotation (models without a value
// projection).  Biases of the projections are added here, in fp32, before the rotation; `gain` multiplies the rotated
// dimensions (scaled rotations).  Layers that read another layer's cache pass no keys: only q is rotated.  NORM: before the
// rotation the whole row of queries, and that of keys, is divided by its root mean square and multiplied by a weight per column.
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
  const void* k;     // [tokens][kv_heads * dim] or null: no keys and values to store
  const void* v;     // [tokens][kv_heads * vdim] or null: the value plane receives the keys before rotation
  const void *q_b, *k_b, *v_b;  // biases, or null
  int64_t row;       // row pitch of q, k and v
  const int32_t* pos;
  const int32_t* slot;
  void *k_pool, *v_pool;  // row of token `off` of page n: n * page_rows + off
  const float2* freq;  // [rot_dims / 2] (high, low)
  float gain;
  const void *q_w, *k_w;  // NORM: [q_heads * dim], [kv_heads * dim]
  float eps;
  int q_heads, kv_heads, dim, vdim, rot_dims, interleaved, page_size, page_rows, max_pages;
  int* status;
};

enum RopeMode : int { kRopeAny = 0, kRopeWidePairs = 1, kRopeWideHalves = 2 };  // wide: eight elements per access

template <typename T, int MODE, bool NORM>
__global__ void __launch_bounds__(NORM && MODE == kRopeWideHalves ? 1024 : 256, NORM && MODE == kRopeWideHalves ? 1 : MODE == kRopeAny ? 5 : 4) rope_store_kernel(const RopeStoreParams p) {
  ptx::griddep_launch_dependents();
  ptx::griddep_wait();
  extern __shared__ float s_ang[];  // [rot_dims / 2] cos, [rot_dims / 2] sin
  const int t = blockIdx.x;
  const int half = p.rot_dims >> 1;
  int s = p.k ? p.slot[t] : -1;
  if (s >= p.max_pages * p.page_size) {
    if (threadIdx.x == 0 && p.status) atomicCAS(p.status, 0, kStatusBadIndex);
    s = -1;
  }
  const int page = s >= 0 ? s / p.page_size : 0, off = s >= 0 ? s % p.page_size : 0;
  const int64_t krow = static_cast<int64_t>(p.kv_heads) * p.dim, vrow = static_cast<int64_t>(p.kv_heads) * p.vdim;
  const int64_t at_row = static_cast<int64_t>(page) * p.page_rows + off;
  T* kdst = reinterpret_cast<T*>(p.k_pool) + at_row * krow;
  T* vdst = reinterpret_cast<T*>(p.v_pool) + at_row * vrow;
  T* q = reinterpret_cast<T*>(p.q) + t * p.row;
  const T* k = reinterpret_cast<const T*>(p.k) + t * p.row;
  const T *q_b = reinterpret_cast<const T*>(p.q_b), *k_b = reinterpret_cast<const T*>(p.k_b), *v_b = reinterpret_cast<const T*>(p.v_b);
  const int heads = p.q_heads + (s >= 0 ? p.kv_heads : 0);
  const T *q_w = reinterpret_cast<const T*>(p.q_w), *k_w = reinterpret_cast<const T*>(p.k_w);
  float q_f = 1.f, k_f = 1.f;
  __shared__ float2 red[32];
  if (NORM && MODE != kRopeWideHalves) {
    auto squares = [&](const T* x, int n) {
      float ss = 0.f;
      if (MODE != kRopeAny) {
        for (int i = threadIdx.x * 8; i < n; i += blockDim.x * 8) {
          float v[8];
          ldf8<T>(x + i, v);
#pragma unroll
          for (int j = 0; j < 8; ++j) ss += v[j] * v[j];
        }
      } else {
        for (int i = threadIdx.x; i < n; i += blockDim.x) {
          const float v = ldf<T>(x + i);
          ss += v * v;
        }
      }
      return ss;
    };
    const int nq = p.q_heads * p.dim, nk = p.k ? p.kv_heads * p.dim : 0;
    const float2 ss = block_sum2(squares(q, nq), squares(k, nk), red);
    q_f = rsqrtf(ss.x / static_cast<float>(nq) + p.eps);
    if (p.k) k_f = rsqrtf(ss.y / static_cast<float>(nk) + p.eps);
  }
  auto angles = [&]() {
    const float pos = static_cast<float>(p.pos[t]);
    for (int i = threadIdx.x; i < half; i += blockDim.x) {
      const float2 f = p.freq[i];
      const float a = pos * f.x;
      const float err = fmaf(pos, f.x, -a) + pos * f.y;
      float sn, cs;
      sincosf(a, &sn, &cs);
      const float c_err = 1.f - 0.5f * err * err;  // cos and sin of the small angle `err`, to second order
      s_ang[i] = (cs * c_err - err * sn) * p.gain;
      s_ang[half + i] = (sn * c_err + err * cs) * p.gain;
    }
    __syncthreads();
  };
  if (MODE != kRopeWideHalves) angles();
  if (MODE != kRopeAny) {
    auto load8 = [&](const T* src, const T* bias, int64_t at, float (&x)[8]) {
      ldf8<T>(src + at, x);
      if (bias) {
        float b[8];
        ldf8<T>(bias + at, b);
#pragma unroll
        for (int j = 0; j < 8; ++j) x[j] += b[j];
      }
      if (NORM && MODE != kRopeWideHalves) {
        const bool is_q = src == q;
        float w[8];
        ldf8<T>((is_q ? q_w : k_w) + at, w);
        const float f = is_q ? q_f : k_f;
#pragma unroll
        for (int j = 0; j < 8; ++j) x[j] *= f * w[j];
      }
    };
    if (MODE == kRopeWidePairs) {
      // eight elements (four pairs) per access; dimensions that pass unchanged ride along
      const int vec = p.dim >> 3;
      for (int it = threadIdx.x; it < heads * vec; it += blockDim.x) {
        const int head = it / vec, d0 = (it - head * vec) * 8;
        const bool is_q = head < p.q_heads;
        if (is_q && d0 >= p.rot_dims && !q_b && !NORM) continue;
        const int64_t at = static_cast<int64_t>(is_q ? head : head - p.q_heads) * p.dim + d0;
        float x[8], y[8];
        load8(is_q ? q : k, is_q ? q_b : k_b, at, x);
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
    } else {
      // half-split heads: eight pairs per item, or eight dimensions that pass unchanged.  A thread's first item is requested
      // before the angles are computed.
      const int turns = half >> 3, vec = turns + ((p.dim - p.rot_dims) >> 3);
      const int items = (p.q_heads + (p.k ? p.kv_heads : 0)) * vec;  // (known before the slot is)
      struct Item {
        int64_t base;
        int c;
        bool is_q, on;
      };
      auto item = [&](int it) {
        Item m;
        const int head = it / vec;
        m.c = it - head * vec;
        m.is_q = head < p.q_heads;
        m.base = static_cast<int64_t>(m.is_q ? head : head - p.q_heads) * p.dim;
        m.on = it < items && !(m.is_q && m.c >= turns && !q_b && !NORM);
        return m;
      };
      auto first = [&](const Item& m) { return m.base + (m.c < turns ? m.c * 8 : p.rot_dims + (m.c - turns) * 8); };
      Item m = item(threadIdx.x);
      float u[8], v[8];
      auto request = [&]() {
        if (!m.on) return;
        load8(m.is_q ? q : k, m.is_q ? q_b : k_b, first(m), u);
        if (m.c < turns) load8(m.is_q ? q : k, m.is_q ? q_b : k_b, first(m) + half, v);
      };
      request();
      auto copy_values = [&]() {
        if (p.v == nullptr || s < 0) return;
        const T* v = reinterpret_cast<const T*>(p.v) + t * p.row;
        for (int i = threadIdx.x * 8; i < vrow; i += blockDim.x * 8) {
          float x[8];
          ldf8<T>(v + i, x);
          if (v_b) {
            float b[8];
            ldf8<T>(v_b + i, b);
#pragma unroll
            for (int j = 0; j < 8; ++j) x[j] += b[j];
          }
          stf8<T>(vdst + i, x);
        }
      };
      float wu[8], wv[8];
      if (NORM) {  // while the values are on their way
        if (m.on) {
          const T* w = (m.is_q ? q_w : k_w) + first(m);
          ldf8<T>(w, wu);
          if (m.c < turns) ldf8<T>(w + half, wv);
        }
        copy_values();
        angles();
      }
      if (NORM) {  // every thread has one item at most (see the launch): its values are what the norms are taken over
        float ss = 0.f;
        if (m.on) {
#pragma unroll
          for (int j = 0; j < 8; ++j) ss += u[j] * u[j] + (m.c < turns ? v[j] * v[j] : 0.f);
        }
        const float2 sum = block_sum2(m.is_q ? ss : 0.f, m.is_q ? 0.f : ss, red);
        q_f = rsqrtf(sum.x / static_cast<float>(p.q_heads * p.dim) + p.eps);
        if (p.k) k_f = rsqrtf(sum.y / static_cast<float>(p.kv_heads * p.dim) + p.eps);
        if (m.on) {
          const float f = m.is_q ? q_f : k_f;
#pragma unroll
          for (int j = 0; j < 8; ++j) {
            u[j] *= f * wu[j];
            if (m.c < turns) v[j] *= f * wv[j];
          }
        }
      }
      if (!NORM) angles();
      for (int it = threadIdx.x; it < items; it += blockDim.x) {
        if (it != static_cast<int>(threadIdx.x)) {
          m = item(it);
          request();
        }
        if (!m.on || (!m.is_q && s < 0)) continue;
        T* dst = m.is_q ? q : kdst;
        const int64_t at = first(m);
        const bool both = !m.is_q && p.v == nullptr;  // values are the keys before rotation
        if (both) stf8<T>(vdst + at, u);
        if (m.c < turns) {
          if (both) stf8<T>(vdst + at + half, v);
#pragma unroll
          for (int j = 0; j < 8; ++j) {
            const float cs = s_ang[m.c * 8 + j], sn = s_ang[half + m.c * 8 + j], x = u[j];
            u[j] = x * cs - v[j] * sn;
            v[j] = v[j] * cs + x * sn;
          }
          stf8<T>(dst + at + half, v);
        }
        stf8<T>(dst + at, u);
      }
      if (NORM) return;
    }
    if (p.v != nullptr && s >= 0) {
      const T* v = reinterpret_cast<const T*>(p.v) + t * p.row;
      for (int i = threadIdx.x * 8; i < vrow; i += blockDim.x * 8) {
        float x[8];
        ldf8<T>(v + i, x);
        if (v_b) {
          float b[8];
          ldf8<T>(v_b + i, b);
#pragma unroll
          for (int j = 0; j < 8; ++j) x[j] += b[j];
        }
        stf8<T>(vdst + i, x);
      }
    }
    return;
  }
  // Rotated pairs of q and k.  With two-element accesses only where pairs are neighbours and rows even.
  const bool vec = p.interleaved && ((p.dim | p.row) & 1) == 0;
  for (int it = threadIdx.x; it < heads * half; it += blockDim.x) {
    const int head = it / half, i = it - head * half;
    const float cs = s_ang[i], sn = s_ang[half + i];
    const int iu = p.interleaved ? 2 * i : i, iv = p.interleaved ? 2 * i + 1 : i + half;
    const bool is_q = head < p.q_heads;
    const int64_t base = static_cast<int64_t>(is_q ? head : head - p.q_heads) * p.dim;
    const T* src = (is_q ? q : k) + base;
    const T* bias = is_q ? q_b : k_b;
    T* dst = (is_q ? q : kdst) + base;
    float u, v;
    if (vec) {
      const float2 f = ldf2<T>(src + iu);
      u = f.x; v = f.y;
    } else {
      u = ldf<T>(src + iu); v = ldf<T>(src + iv);
    }
    if (bias) {
      u += ldf<T>(bias + base + iu);
      v += ldf<T>(bias + base + iv);
    }
    if (NORM) {
      const T* w = (is_q ? q_w : k_w) + base;
      const float f = is_q ? q_f : k_f;
      u *= f * ldf<T>(w + iu);
      v *= f * ldf<T>(w + iv);
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
  const int rest = p.dim - p.rot_dims;  // dimensions that pass unchanged: keys, values taken from them, queries with a bias
  for (int it = threadIdx.x; it < heads * rest; it += blockDim.x) {
    const int head = it / rest;
    const bool is_q = head < p.q_heads;
    if (is_q && !q_b && !NORM) continue;
    const int64_t at = static_cast<int64_t>(is_q ? head : head - p.q_heads) * p.dim + p.rot_dims + it % rest;
    const T* bias = is_q ? q_b : k_b;
    float x = ldf<T>((is_q ? q : k) + at) + (bias ? ldf<T>(bias + at) : 0.f);
    if (NORM) x *= (is_q ? q_f : k_f) * ldf<T>((is_q ? q_w : k_w) + at);
    stf<T>((is_q ? q : kdst) + at, x);
    if (!is_q && p.v == nullptr) stf<T>(vdst + at, x);
  }
  if (p.v != nullptr && s >= 0) {
    const T* v = reinterpret_cast<const T*>(p.v) + t * p.row;
    for (int i = threadIdx.x; i < vrow; i += blockDim.x) stf<T>(vdst + i, ldf<T>(v + i) + (v_b ? ldf<T>(v_b + i) : 0.f));
  }
}

}  // namespace blitz

extern "C" {
using namespace blitz;

// Pools: [max_pages][page_rows][heads][size]; a page's `page_size` token rows are its first ones (with one tensor for keys
// and values page_rows is 2 page_size and v_pool points at the first value plane).  q_w, k_w: weights of the norms over whole rows, or null.
int blitz_rope_store(void* q, const void* k, const void* v, const void* q_b, const void* k_b, const void* v_b, int64_t row,
                     const void* q_w, const void* k_w, float eps,
                     const int32_t* pos, const int32_t* slot, void* k_pool, void* v_pool, const void* freq, float gain,
                     int num_tokens, int q_heads, int kv_heads, int dim, int vdim, int rot_dims, int interleaved, int page_size,
                     int page_rows, int max_pages, int* status, int dtype, cudaStream_t stream) {
  if (num_tokens <= 0) return 0;
  if (rot_dims < 0 || (rot_dims & 1) || rot_dims > dim || rot_dims > 4096 || (rot_dims > 0 && freq == nullptr)) return -1;
  if (k != nullptr && v == nullptr && vdim != dim) return -1;
  if (q_w != nullptr && (q_b || k_b || (k && (k_w == nullptr || v == nullptr)))) return -1;
  RopeStoreParams p{q, k, v, q_b, k_b, v_b, row, pos, slot, k_pool, v_pool, reinterpret_cast<const float2*>(freq), gain, q_w, k_w, eps, q_heads,
                    kv_heads, dim, vdim, rot_dims, interleaved, page_size, page_rows, max_pages, status};
  const uintptr_t al = dtype == 2 ? 32 : 16;
  bool wide = ((dim | vdim | row) & 7) == 0 && (interleaved || (rot_dims & 15) == 0);
  for (const void* x : {(const void*)q, k, v, q_b, k_b, v_b, q_w, k_w, (const void*)k_pool, (const void*)v_pool})
    wide = wide && (reinterpret_cast<uintptr_t>(x) % al) == 0;
  const int items = (q_heads + (k ? kv_heads : 0)) * (rot_dims / 16 + (dim - rot_dims) / 8);  // of the wide half-split form
  if (q_w && !interleaved && items > 1024) wide = false;
  const int one_each = q_w && wide && !interleaved ? (items + 31) / 32 * 32 : 0;
  const dim3 grid(num_tokens), block(one_each ? one_each : wide && (q_heads + kv_heads) * dim <= 2048 ? 128 : 256);
  const size_t smem = (size_t)rot_dims * sizeof(float);
  auto go = [&](auto type, auto norm) {
    using T = decltype(type);
    constexpr bool N = decltype(norm)::value;
    if (!wide) return launch_pdl(rope_store_kernel<T, kRopeAny, N>, grid, block, smem, stream, p);
    return interleaved ? launch_pdl(rope_store_kernel<T, kRopeWidePairs, N>, grid, block, smem, stream, p)
                       : launch_pdl(rope_store_kernel<T, kRopeWideHalves, N>, grid, block, smem, stream, p);
  };
  cudaError_t e = cudaSuccess;
  BLITZ_DISPATCH_DTYPE3(dtype, (e = q_w ? go(T{}, std::true_type{}) : go(T{}, std::false_type{})));
  return (int)e;
}

}  // extern "C"
