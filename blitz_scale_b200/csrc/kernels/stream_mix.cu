// Hyper-connections with the dynamic-tanh norm: a model whose residual is several fp32 streams per token.  Between two
// sublayers the streams take up the output y of the last one and are collapsed into the input of the next one:
//
//   x_t <- sum_s mix[s][t] x_s + out[t] y          (all streams at once, from the old ones)
//   u    = sum_s in[s] x_s                          in null: the sum of the streams
//   h    = tanh(alpha u) w + b
//
// One kernel per sublayer does all three: one read and one write of the streams.  At the start every stream is the token's
// embedding; the first kernels read the embedding table instead of the streams, which are written when the first y arrives.
// y is a row per token, or the rows that a mixture of experts has left for the token (add_row, -1: none), plus the weight of
// its identity experts times what the sublayer read.
//
// No reduction over the columns: a thread owns four columns and walks tokens, with the coefficients of its layer and its
// columns' weights in registers.  The rows of the next token's experts are looked up a token ahead.
#include "launch.cuh"
#include "ptx.cuh"
#include "scalar.cuh"
#include "tmap.cuh"

namespace blitz {

constexpr int kSmMaxStreams = 8;

struct StreamMixParams {
  const int32_t* ids;       // from_embed
  const void* embed;
  float* x;                 // [tokens][streams][hidden]
  const void* y;            // last sublayer's output, or null
  const int32_t* add_row;   // [tokens][n_add] rows of y, or null: row t
  const float* ident;       // [tokens] weight of `prev`, or null
  const void* prev;         // [tokens][hidden]
  const void *mix, *out_w;  // [streams][streams], [streams]
  const void* in_w;         // [streams], or null
  const void *alpha, *w, *b;
  const int32_t* rows;      // result t comes from token rows[t] + row_offset (null: t)
  void* h;                  // [tokens][hidden], or null
  float* u;                 // [tokens][hidden], or null
  int tokens, hidden, vocab, n_add, row_offset, from_embed, write;
  int* status;
};

template <int VEC>
struct Cols {
  float v[VEC];
};

template <typename T, int VEC>
__device__ __forceinline__ Cols<VEC> cols_load(const T* p) {
  Cols<VEC> c;
  if constexpr (VEC == 4) {
    const float4 a = ldf4<T>(p);
    c.v[0] = a.x; c.v[1] = a.y; c.v[2] = a.z; c.v[3] = a.w;
  } else {
    c.v[0] = ldf<T>(p);
  }
  return c;
}
template <typename T, int VEC>
__device__ __forceinline__ void cols_store(T* p, const Cols<VEC>& c) {
  if constexpr (VEC == 4) stf4<T>(p, make_float4(c.v[0], c.v[1], c.v[2], c.v[3]));
  else stf<T>(p, c.v[0]);
}

// As they lie in memory.
template <typename T, int VEC>
struct alignas(VEC * sizeof(T)) RawCols {
  T e[VEC];
};

enum SmPending : int { kSmNone = 0, kSmDense = 1, kSmRows = 2 };

template <typename T, int VEC, int S, int PEND, int AT_ONCE>
__global__ void __launch_bounds__(256) stream_mix_kernel(const StreamMixParams p) {
  ptx::griddep_launch_dependents();
  const int64_t H = p.hidden;
  const int c = (blockIdx.y * blockDim.x + threadIdx.x) * VEC;
  const bool on = c < p.hidden;
  float mix[S][S], ow[S], iw[S], alpha = 0.f;
  Cols<VEC> w, b;
  if (on) {  // weights are not written by kernels still running
#pragma unroll
    for (int s = 0; s < S; ++s) {
      iw[s] = p.in_w ? ldf<T>(reinterpret_cast<const T*>(p.in_w) + s) : 1.f;
      if (PEND != kSmNone) {
        ow[s] = ldf<T>(reinterpret_cast<const T*>(p.out_w) + s);
#pragma unroll
        for (int t = 0; t < S; ++t) mix[s][t] = ldf<T>(reinterpret_cast<const T*>(p.mix) + s * S + t);
      }
    }
    if (p.h) {
      alpha = ldf<T>(reinterpret_cast<const T*>(p.alpha));
      w = cols_load<T, VEC>(reinterpret_cast<const T*>(p.w) + c);
      b = cols_load<T, VEC>(reinterpret_cast<const T*>(p.b) + c);
    }
  }
  ptx::griddep_wait();
  if (!on) return;
  auto source = [&](int t) { return p.rows ? p.rows[t] + p.row_offset : t; };
  int place[AT_ONCE];  // the first rows of a token
  auto look_up = [&](int src) {
    const int32_t* rows = p.add_row + static_cast<int64_t>(src) * p.n_add;
#pragma unroll
    for (int k = 0; k < AT_ONCE; ++k) place[k] = k < p.n_add ? rows[k] : -1;
  };
  if (PEND == kSmRows && static_cast<int>(blockIdx.x) < p.tokens) look_up(source(blockIdx.x));
  for (int t = blockIdx.x; t < p.tokens; t += gridDim.x) {
    const int src = source(t);
    Cols<VEC> x[S];
    float* xr = p.x + static_cast<int64_t>(src) * S * H + c;
    if (p.from_embed) {
      const int id = p.ids[src];
      Cols<VEC> e = {};
      if (id >= 0 && id < p.vocab) e = cols_load<T, VEC>(reinterpret_cast<const T*>(p.embed) + id * H + c);
      else if (p.status && c == 0) atomicCAS(p.status, 0, kStatusBadIndex);
#pragma unroll
      for (int s = 0; s < S; ++s) x[s] = e;
    } else {
#pragma unroll
      for (int s = 0; s < S; ++s) x[s] = cols_load<float, VEC>(xr + s * H);
    }
    if (PEND != kSmNone) {
      Cols<VEC> y = {};
      const T* yp = reinterpret_cast<const T*>(p.y) + c;
      if (PEND == kSmDense) {
        y = cols_load<T, VEC>(yp + src * H);
      } else {
        using Raw = RawCols<T, VEC>;
        auto get = [&](const T* q) { return *reinterpret_cast<const Raw*>(q); };
        auto sum = [&](float f, const Raw& r) {
#pragma unroll
          for (int i = 0; i < VEC; ++i) y.v[i] += f * ldf<T>(&r.e[i]);
        };
        Raw v[AT_ONCE], same;
        float f = 0.f, use[AT_ONCE];
#pragma unroll
        for (int k = 0; k < AT_ONCE; ++k) {  // all requested before the first is used
          use[k] = place[k] >= 0 ? 1.f : 0.f;
          v[k] = get(yp + max(place[k], 0) * H);
        }
        if (p.ident) {
          f = p.ident[src];
          same = get(reinterpret_cast<const T*>(p.prev) + src * H + c);
        }
        if (t + static_cast<int>(gridDim.x) < p.tokens) look_up(source(t + gridDim.x));
#pragma unroll
        for (int k = 0; k < AT_ONCE; ++k)
          if (use[k] != 0.f) sum(1.f, v[k]);
        for (int k = AT_ONCE; k < p.n_add; ++k) {
          const int r = p.add_row[static_cast<int64_t>(src) * p.n_add + k];
          if (r >= 0) sum(1.f, get(yp + r * H));
        }
        if (f != 0.f) sum(f, same);
      }
#pragma unroll
      for (int i = 0; i < VEC; ++i) {
        float n[S];
#pragma unroll
        for (int t2 = 0; t2 < S; ++t2) {
          n[t2] = ow[t2] * y.v[i];
#pragma unroll
          for (int s = 0; s < S; ++s) n[t2] = fmaf(mix[s][t2], x[s].v[i], n[t2]);
        }
#pragma unroll
        for (int s = 0; s < S; ++s) x[s].v[i] = n[s];
      }
      if (p.write) {
#pragma unroll
        for (int s = 0; s < S; ++s) cols_store<float, VEC>(xr + s * H, x[s]);
      }
    }
    if (p.h == nullptr && p.u == nullptr) continue;
    Cols<VEC> u;
#pragma unroll
    for (int i = 0; i < VEC; ++i) {
      float a = 0.f;
#pragma unroll
      for (int s = 0; s < S; ++s) a = fmaf(iw[s], x[s].v[i], a);
      u.v[i] = a;
    }
    if (p.u) cols_store<float, VEC>(p.u + t * H + c, u);
    if (p.h) {
#pragma unroll
      for (int i = 0; i < VEC; ++i) u.v[i] = fmaf(tanhf(alpha * u.v[i]), w.v[i], b.v[i]);
      cols_store<T, VEC>(reinterpret_cast<T*>(p.h) + t * H + c, u);
    }
  }
}

template <typename T, int VEC, int S>
static cudaError_t launch_stream_mix(const StreamMixParams& p, cudaStream_t stream) {
  const int n = p.hidden / VEC;
  int threads = 32;
  while (threads < n && threads < 256) threads <<= 1;
  const int chunks = (n + threads - 1) / threads;
  // a block that walks several tokens reads the coefficients once
  const int most = (device_sm_count() * (2048 / threads) + chunks - 1) / chunks;
  const dim3 grid(p.tokens < most ? p.tokens : most, chunks), block(threads);
  if (p.y == nullptr) return launch_pdl(stream_mix_kernel<T, VEC, S, kSmNone, 1>, grid, block, 0, stream, p);
  if (p.add_row == nullptr) return launch_pdl(stream_mix_kernel<T, VEC, S, kSmDense, 1>, grid, block, 0, stream, p);
  if (p.n_add <= 4) return launch_pdl(stream_mix_kernel<T, VEC, S, kSmRows, 4>, grid, block, 0, stream, p);
  return launch_pdl(stream_mix_kernel<T, VEC, S, kSmRows, 8>, grid, block, 0, stream, p);
}

}  // namespace blitz

extern "C" {
using namespace blitz;

// See the top of the file.  x fp32 [tokens][streams][hidden]; embed, y, prev, h and all weights in the activation type (dtype
// 0 fp16, 1 bf16, 2 fp32).  y null: the streams stay as they are (`write` must be 0 then); from_embed: the streams are the
// embeddings of `ids` and x is not read.  h: the normalised input of the next sublayer; u: the input before the norm, fp32.
// With `rows`, h must not be `prev`.
int blitz_stream_mix(const int32_t* ids, const void* embed, int vocab, int from_embed, float* x, const void* y, const int32_t* add_row,
                     int n_add, const float* ident, const void* prev, const void* mix, const void* out_w, const void* in_w,
                     const void* alpha, const void* w, const void* b, const int32_t* rows, int row_offset, void* h, float* u, int write,
                     int tokens, int hidden, int streams, int* status, int dtype, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (hidden <= 0 || streams < 1 || streams > kSmMaxStreams || x == nullptr || n_add < 0) return -1;
  if (from_embed && (ids == nullptr || embed == nullptr)) return -1;
  if (y == nullptr ? write != 0 : (mix == nullptr || out_w == nullptr)) return -1;
  if (h && (alpha == nullptr || w == nullptr || b == nullptr)) return -1;
  if (ident && (prev == nullptr || add_row == nullptr)) return -1;
  if (rows && (write || (h && h == prev))) return -1;
  StreamMixParams p{ids, embed, x, y, add_row, ident, prev, mix, out_w, in_w, alpha, w, b, rows, h, u,
                    tokens, hidden, vocab, n_add, row_offset, from_embed, write, status};
  auto go = [&](auto type, auto vec) -> cudaError_t {
    using T = decltype(type);
    constexpr int V = decltype(vec)::value;
    switch (streams) {
      case 1: return launch_stream_mix<T, V, 1>(p, stream);
      case 2: return launch_stream_mix<T, V, 2>(p, stream);
      case 3: return launch_stream_mix<T, V, 3>(p, stream);
      case 4: return launch_stream_mix<T, V, 4>(p, stream);
      case 5: return launch_stream_mix<T, V, 5>(p, stream);
      case 6: return launch_stream_mix<T, V, 6>(p, stream);
      case 7: return launch_stream_mix<T, V, 7>(p, stream);
      default: return launch_stream_mix<T, V, 8>(p, stream);
    }
  };
  cudaError_t e = cudaSuccess;
  BLITZ_DISPATCH_DTYPE3(dtype, (e = (hidden & 3) ? go(T{}, std::integral_constant<int, 1>{}) : go(T{}, std::integral_constant<int, 4>{})));
  return (int)e;
}

}  // extern "C"
