// Hyper-connections with an RMS norm (stream_mix.cu has them with a norm that needs no sums over the columns), and for decode
// steps what lies between the norm and the mixer's projections: a causal convolution on every channel and the mixes with the
// previous token's row.
//
//   y    = y0 + bias                                                  the last sublayer's output, or
//   y    = (y0 / rms(y0) w0 + y1 / rms(y1) w1) / 2                    those of two sublayers side by side
//   x_t <- sum_s mix[s][t] x_s + out[t] y                             all streams at once, from the old ones
//   u    = sum_s in[s] x_s                                            in null: the sum of the streams
//   h    = u / sqrt(mean(u^2) + eps) (w_offset + w)                   w: one number, or one per column
//   h   <- h + sum_j conv[j] h_(j - taps + 1 tokens back)             CONV: the earlier ones from the sequence's history
//   m_i  = h + (h_previous - h) mu_i                                  CONV with mixes: one row per mix
//
// A block per token.  A thread keeps its columns of u in registers between the two passes; every other value of a column is
// only used by the thread that owns the column, the histories (by slot, fp32) included: what the norm gives is not rounded before
// the convolution and the mixes are done.  At the start every stream is the token's
// embedding; the first kernels read the embedding table instead of the streams.
#include "launch.cuh"
#include "ptx.cuh"
#include "scalar.cuh"
#include "tmap.cuh"

namespace blitz {

constexpr int kSrMaxStreams = 8;
constexpr int kSrKeep = 4;  // groups of columns of u that a thread keeps in registers; further ones are kept in shared memory
constexpr int kSrThreads = 512;

struct StreamRmsParams {
  const int32_t* ids;       // from_embed
  const void* embed;
  float* x;                 // [tokens][streams][hidden]
  const void *y, *y1;       // last outputs [tokens][y_row]; y null: none, y1 null: one
  int64_t y_row;
  const void *bias;         // [hidden], or null
  const void *w0, *w1;      // [hidden], with y1
  const void *mix, *out_w;  // [streams][streams], [streams]
  const void* in_w;         // [streams], or null
  const void* w;            // [1] or [hidden]
  const int32_t* rows;      // result t comes from token rows[t] + row_offset (null: t)
  void* h;                  // [tokens][hidden] (mixes: [tokens][mixes][hidden]), or null
  int h32;                  // h is fp32 (no convolution)
  float* u;                 // [tokens][hidden], or null
  const void* conv;         // [taps][hidden], or null
  float* hist;              // [slots][taps - 1][hidden]
  const void* mu;           // [mixes][hidden]
  float* shift;             // [slots][hidden]
  const int32_t *pos, *seq_slot;
  float eps, w_offset;
  int hidden, vocab, row_offset, from_embed, write, w_step, taps, mixes, num_slots;
  int* status;
};

template <typename T, int VEC>
struct SrCols {
  float v[VEC];
  __device__ __forceinline__ void load(const T* p) {
    if constexpr (VEC == 4) {
      const float4 a = ldf4<T>(p);
      v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
    } else {
      v[0] = ldf<T>(p);
    }
  }
  __device__ __forceinline__ void store(T* p) const {
    if constexpr (VEC == 4) stf4<T>(p, make_float4(v[0], v[1], v[2], v[3]));
    else stf<T>(p, v[0]);
  }
};

// Columns as they lie in memory.
template <typename T, int VEC>
struct alignas(VEC * sizeof(T)) SrRaw {
  T e[VEC];
};

// What the convolution reads beside the token's row, requested before the norm is known: up to kSrTaps taps and kSrMixes mixes.
constexpr int kSrTaps = 4, kSrMixes = 5;
template <typename T, int VEC>
struct SrEarly {
  SrRaw<T, VEC> conv[kSrTaps], mu[kSrMixes];
  SrCols<float, VEC> hist[kSrTaps - 1], prev;  // taps and history end at the last place
};

template <typename T, int VEC, int S, bool CONV>
__global__ void __launch_bounds__(kSrThreads, CONV || S > 4 ? 1 : 2) stream_rms_kernel(const StreamRmsParams p) {
  using C = SrCols<T, VEC>;
  using F = SrCols<float, VEC>;
  __shared__ float s_mix[S * S], s_out[S], s_in[S];
  __shared__ float2 red[32], red2[32];
  extern __shared__ __align__(16) float s_keep[];
  ptx::griddep_launch_dependents();
  const T *w = reinterpret_cast<const T*>(p.w), *bias = reinterpret_cast<const T*>(p.bias);
  constexpr int kKeep = CONV ? 2 : kSrKeep;
  const bool ahead = CONV && p.taps <= kSrTaps && p.mixes <= kSrMixes;
  using Raw = SrRaw<T, VEC>;
  SrEarly<T, VEC> early[CONV ? kKeep : 1];
  auto raw = [](const void* base, int64_t at) { return *reinterpret_cast<const Raw*>(reinterpret_cast<const T*>(base) + at); };
  if (CONV && ahead) {
#pragma unroll
    for (int g = 0; g < kKeep; ++g) {
      const int c = (threadIdx.x + g * blockDim.x) * VEC;
      SrEarly<T, VEC>& e = early[CONV ? g : 0];
      if (c >= p.hidden) continue;
#pragma unroll
      for (int j = 0; j < kSrTaps; ++j)
        if (j >= kSrTaps - p.taps) e.conv[j] = raw(p.conv, static_cast<int64_t>(j - (kSrTaps - p.taps)) * p.hidden + c);
#pragma unroll
      for (int m = 0; m < kSrMixes; ++m)
        if (m < p.mixes) e.mu[m] = raw(p.mu, static_cast<int64_t>(m) * p.hidden + c);
    }
  }
  for (int i = threadIdx.x; i < S * S; i += blockDim.x) {  // weights are not written by kernels still running
    if (p.mix) s_mix[i] = ldf<T>(reinterpret_cast<const T*>(p.mix) + i);
    if (i < S) {
      s_in[i] = p.in_w ? ldf<T>(reinterpret_cast<const T*>(p.in_w) + i) : 1.f;
      if (p.out_w) s_out[i] = ldf<T>(reinterpret_cast<const T*>(p.out_w) + i);
    }
  }
  ptx::griddep_wait();
  __syncthreads();
  const int t = blockIdx.x, src = p.rows ? p.rows[t] + p.row_offset : t;
  const int n = p.hidden / VEC;
  float* xr = p.x + static_cast<int64_t>(src) * S * p.hidden;
  const T* er = nullptr;
  if (p.from_embed) {
    const int id = p.ids[src];
    if (id >= 0 && id < p.vocab) er = reinterpret_cast<const T*>(p.embed) + static_cast<int64_t>(id) * p.hidden;
    else if (p.status && threadIdx.x == 0) atomicCAS(p.status, 0, kStatusBadIndex);
  }
  int slot = -1, at = 0;
  if (CONV) {
    slot = p.seq_slot[t];
    at = p.pos[t];
    if (slot >= p.num_slots) {
      if (p.status && threadIdx.x == 0) atomicCAS(p.status, 0, kStatusBadIndex);
      slot = -1;
    }
  }
  if (CONV && ahead && slot >= 0) {
#pragma unroll
    for (int g = 0; g < kKeep; ++g) {
      const int c = (threadIdx.x + g * blockDim.x) * VEC;
      SrEarly<T, VEC>& e = early[CONV ? g : 0];
      if (c >= p.hidden) continue;
#pragma unroll
      for (int j = 0; j + 1 < kSrTaps; ++j)
        if (j >= kSrTaps - p.taps)
          e.hist[j].load(p.hist + (static_cast<int64_t>(slot) * (p.taps - 1) + j - (kSrTaps - p.taps)) * p.hidden + c);
      if (p.mixes > 0 && at > 0) e.prev.load(p.shift + static_cast<int64_t>(slot) * p.hidden + c);
    }
  }
  const T* y0 = p.y ? reinterpret_cast<const T*>(p.y) + src * p.y_row : nullptr;
  const T* y1 = p.y1 ? reinterpret_cast<const T*>(p.y1) + src * p.y_row : nullptr;
  float f0 = 1.f, f1 = 0.f;
  if (y1) {  // the two outputs' norms
    float a = 0.f, b = 0.f;
    for (int i = threadIdx.x; i < n; i += blockDim.x) {
      C c, d;
      c.load(y0 + i * VEC);
      d.load(y1 + i * VEC);
#pragma unroll
      for (int k = 0; k < VEC; ++k) {
        a += c.v[k] * c.v[k];
        b += d.v[k] * d.v[k];
      }
    }
    const float2 sum = block_sum2(a, b, red2);
    f0 = 0.5f * rsqrtf(sum.x / static_cast<float>(p.hidden) + p.eps);
    f1 = 0.5f * rsqrtf(sum.y / static_cast<float>(p.hidden) + p.eps);
  }
  F keep[kKeep];
  float ss = 0.f;
  auto collect = [&](int i) {
    const int c = i * VEC;
    F x[S];
    if (p.from_embed) {
      C e = {};
      if (er) e.load(er + c);
#pragma unroll
      for (int s = 0; s < S; ++s)
#pragma unroll
        for (int k = 0; k < VEC; ++k) x[s].v[k] = e.v[k];
    } else {
#pragma unroll
      for (int s = 0; s < S; ++s) x[s].load(xr + static_cast<int64_t>(s) * p.hidden + c);
    }
    if (y0) {
      C y;
      y.load(y0 + c);
      if (y1) {
        C z, a, b;
        z.load(y1 + c);
        a.load(reinterpret_cast<const T*>(p.w0) + c);
        b.load(reinterpret_cast<const T*>(p.w1) + c);
#pragma unroll
        for (int k = 0; k < VEC; ++k) y.v[k] = y.v[k] * f0 * a.v[k] + z.v[k] * f1 * b.v[k];
      } else if (bias) {
        C b;
        b.load(bias + c);
#pragma unroll
        for (int k = 0; k < VEC; ++k) y.v[k] += b.v[k];
      }
#pragma unroll
      for (int k = 0; k < VEC; ++k) {
        float r[S];
#pragma unroll
        for (int o = 0; o < S; ++o) {
          r[o] = s_out[o] * y.v[k];
#pragma unroll
          for (int s = 0; s < S; ++s) r[o] = fmaf(s_mix[s * S + o], x[s].v[k], r[o]);
        }
#pragma unroll
        for (int s = 0; s < S; ++s) x[s].v[k] = r[s];
      }
      if (p.write)
#pragma unroll
        for (int s = 0; s < S; ++s) x[s].store(xr + static_cast<int64_t>(s) * p.hidden + c);
    }
    F u = {};
#pragma unroll
    for (int s = 0; s < S; ++s)
#pragma unroll
      for (int k = 0; k < VEC; ++k) u.v[k] = fmaf(s_in[s], x[s].v[k], u.v[k]);
#pragma unroll
    for (int k = 0; k < VEC; ++k) ss += u.v[k] * u.v[k];
    if (p.u) u.store(p.u + static_cast<int64_t>(t) * p.hidden + c);
    return u;
  };
  const int behind = kKeep * blockDim.x;
#pragma unroll
  for (int g = 0; g < kKeep; ++g) {
    const int i = threadIdx.x + g * blockDim.x;
    if (i < n) keep[g] = collect(i);
  }
  for (int i = threadIdx.x + behind; i < n; i += blockDim.x) collect(i).store(s_keep + (i - behind) * VEC);
  if (p.h == nullptr) return;
  const float scale = rsqrtf(block_sum2(ss, 0.f, red).x / static_cast<float>(p.hidden) + p.eps);
  const float gain = p.w_step ? 0.f : p.w_offset + ldf<T>(w);
  const int per = CONV && p.mixes > 0 ? p.mixes : 1;
  T* out = reinterpret_cast<T*>(p.h) + static_cast<int64_t>(t) * per * p.hidden;
  auto convolved = [&](int c, C h, const SrEarly<T, VEC>& e) {
    F now;
#pragma unroll
    for (int k = 0; k < VEC; ++k) now.v[k] = h.v[k];
    auto add = [&](const Raw& a, const F& b) {
#pragma unroll
      for (int k = 0; k < VEC; ++k) h.v[k] += ldf<T>(&a.e[k]) * b.v[k];
    };
#pragma unroll
    for (int k = 0; k < VEC; ++k) h.v[k] += ldf<T>(&e.conv[kSrTaps - 1].e[k]) * now.v[k];
    if (slot >= 0) {
      float* hist = p.hist + static_cast<int64_t>(slot) * (p.taps - 1) * p.hidden + c;
#pragma unroll
      for (int j = 0; j + 1 < kSrTaps; ++j) {
        const int first = kSrTaps - p.taps;
        if (j < first) continue;
        if (kSrTaps - 1 - j <= at) add(e.conv[j], e.hist[j]);
        if (j > first) e.hist[j].store(hist + static_cast<int64_t>(j - first - 1) * p.hidden);
      }
      if (p.taps > 1) now.store(hist + static_cast<int64_t>(p.taps - 2) * p.hidden);
    }
    if (p.mixes == 0) {
      h.store(out + c);
      return;
    }
    float d[VEC];
#pragma unroll
    for (int k = 0; k < VEC; ++k) {
      d[k] = (slot >= 0 && at > 0 ? e.prev.v[k] : 0.f) - h.v[k];
      now.v[k] = h.v[k];
    }
    if (slot >= 0) now.store(p.shift + static_cast<int64_t>(slot) * p.hidden + c);
#pragma unroll
    for (int m = 0; m < kSrMixes; ++m) {
      if (m >= p.mixes) continue;
      C b;
#pragma unroll
      for (int k = 0; k < VEC; ++k) b.v[k] = h.v[k] + d[k] * ldf<T>(&e.mu[m].e[k]);
      b.store(out + static_cast<int64_t>(m) * p.hidden + c);
    }
  };
  auto normed = [&](int c, const F& u) {
    C h;
    if (p.w_step) {
      C a;
      a.load(w + c);
#pragma unroll
      for (int k = 0; k < VEC; ++k) h.v[k] = u.v[k] * scale * (p.w_offset + a.v[k]);
    } else {
#pragma unroll
      for (int k = 0; k < VEC; ++k) h.v[k] = u.v[k] * scale * gain;
    }
    return h;
  };
  auto finish = [&](int c, C h) {
    if (CONV) {
      const T* conv = reinterpret_cast<const T*>(p.conv) + c;
      float* hist = p.hist + static_cast<int64_t>(slot < 0 ? 0 : slot) * (p.taps - 1) * p.hidden + c;
      C a;
      F now;
#pragma unroll
      for (int k = 0; k < VEC; ++k) now.v[k] = h.v[k];
      a.load(conv + static_cast<int64_t>(p.taps - 1) * p.hidden);
#pragma unroll
      for (int k = 0; k < VEC; ++k) h.v[k] += a.v[k] * now.v[k];
      if (slot >= 0) {
        for (int j = 0; j + 1 < p.taps; ++j) {  // the oldest first; what a place holds moves to the one before it
          F b;
          b.load(hist + static_cast<int64_t>(j) * p.hidden);
          if (j > 0) b.store(hist + static_cast<int64_t>(j - 1) * p.hidden);
          if (p.taps - 1 - j <= at) {
            a.load(conv + static_cast<int64_t>(j) * p.hidden);
#pragma unroll
            for (int k = 0; k < VEC; ++k) h.v[k] += a.v[k] * b.v[k];
          }
        }
        if (p.taps > 1) now.store(hist + static_cast<int64_t>(p.taps - 2) * p.hidden);
      }
      if (p.mixes > 0) {
        F prev = {};
        if (slot >= 0) {
          float* shift = p.shift + static_cast<int64_t>(slot) * p.hidden + c;
          if (at > 0) prev.load(shift);
#pragma unroll
          for (int k = 0; k < VEC; ++k) now.v[k] = h.v[k];
          now.store(shift);
        }
        for (int m = 0; m < p.mixes; ++m) {
          C b;
          b.load(reinterpret_cast<const T*>(p.mu) + static_cast<int64_t>(m) * p.hidden + c);
#pragma unroll
          for (int k = 0; k < VEC; ++k) b.v[k] = h.v[k] + (prev.v[k] - h.v[k]) * b.v[k];
          b.store(out + static_cast<int64_t>(m) * p.hidden + c);
        }
        return;
      }
    }
    if (!CONV && p.h32) {
      F wide;
#pragma unroll
      for (int k = 0; k < VEC; ++k) wide.v[k] = h.v[k];
      wide.store(reinterpret_cast<float*>(p.h) + static_cast<int64_t>(t) * p.hidden + c);
      return;
    }
    h.store(out + c);
  };
#pragma unroll
  for (int g = 0; g < kKeep; ++g) {
    const int i = threadIdx.x + g * blockDim.x;
    if (i >= n) continue;
    const C h = normed(i * VEC, keep[g]);
    if (CONV && ahead) convolved(i * VEC, h, early[CONV ? g : 0]);
    else finish(i * VEC, h);
  }
  for (int i = threadIdx.x + behind; i < n; i += blockDim.x) {
    F u;
    u.load(s_keep + (i - behind) * VEC);
    finish(i * VEC, normed(i * VEC, u));
  }
}

}  // namespace blitz

extern "C" {
using namespace blitz;

// See the top of the file.  x fp32 [tokens][streams][hidden]; embed, y, y1, h and all weights in the activation type (dtype 0 fp16,
// 1 bf16, 2 fp32); h32: h is fp32.  y null: the streams stay as they are (`write` must be 0 then).  w_step: 0 one norm weight, 1 a
// weight per column.  conv null: no convolution; else every row is one token of a sequence with a state slot (negative: none).
int blitz_stream_rms(const int32_t* ids, const void* embed, int vocab, int from_embed, float* x, const void* y, const void* y1,
                     int64_t y_row, const void* bias, const void* w0, const void* w1, const void* mix, const void* out_w,
                     const void* in_w, const void* w, int w_step, float w_offset, float eps, const int32_t* rows, int row_offset, void* h,
                     int h32, float* u, int write, const void* conv, int taps, float* hist, const void* mu, int mixes, float* shift,
                     const int32_t* pos, const int32_t* seq_slot, int num_slots, int tokens, int hidden, int streams, int* status,
                     int dtype, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (hidden <= 0 || streams < 1 || streams > kSrMaxStreams || x == nullptr) return -1;
  if (from_embed && (ids == nullptr || embed == nullptr)) return -1;
  if (y == nullptr ? (write != 0 || y1 != nullptr) : (mix == nullptr || out_w == nullptr)) return -1;
  if (y1 && (w0 == nullptr || w1 == nullptr || bias != nullptr)) return -1;
  if (h && w == nullptr) return -1;
  if ((rows && write) || (h32 && conv)) return -1;
  if (conv && (rows || !h || taps < 1 || !pos || !seq_slot || (taps > 1 && !hist) || (mixes > 0 && (!mu || !shift)))) return -1;
  StreamRmsParams p{ids, embed, x, y, y1, y_row, bias, w0, w1, mix, out_w, in_w, w, rows, h, h32, u, conv, hist, mu, shift, pos, seq_slot,
                    eps, w_offset, hidden, vocab, row_offset, from_embed, write, w_step, taps, mixes, num_slots, status};
  const int vec = (hidden & 3) || (y_row & 3) ? 1 : 4, n = hidden / vec;
  int threads = 32;
  // few tokens: as many threads as there are groups
  while (threads < n && threads < (tokens <= device_sm_count() ? kSrThreads : 256)) threads <<= 1;
  const int keep = conv ? 2 : kSrKeep;
  while (threads * keep < n && threads < kSrThreads) threads <<= 1;
  const size_t smem = threads * keep < n ? (size_t)(n - threads * keep) * vec * sizeof(float) : 0;
  if (smem > 40 * 1024) return -1;
  auto go = [&](auto type, auto v, auto s) -> cudaError_t {
    using T = decltype(type);
    constexpr int V = decltype(v)::value, S = decltype(s)::value;
    return conv ? launch_pdl(stream_rms_kernel<T, V, S, true>, dim3(tokens), dim3(threads), smem, stream, p)
                : launch_pdl(stream_rms_kernel<T, V, S, false>, dim3(tokens), dim3(threads), smem, stream, p);
  };
  auto wide = [&](auto type, auto s) -> cudaError_t {
    return vec == 4 ? go(type, std::integral_constant<int, 4>{}, s) : go(type, std::integral_constant<int, 1>{}, s);
  };
  auto sized = [&](auto type) -> cudaError_t {
    switch (streams) {
      case 1: return wide(type, std::integral_constant<int, 1>{});
      case 2: return wide(type, std::integral_constant<int, 2>{});
      case 3: return wide(type, std::integral_constant<int, 3>{});
      case 4: return wide(type, std::integral_constant<int, 4>{});
      case 5: return wide(type, std::integral_constant<int, 5>{});
      case 6: return wide(type, std::integral_constant<int, 6>{});
      case 7: return wide(type, std::integral_constant<int, 7>{});
      default: return wide(type, std::integral_constant<int, 8>{});
    }
  };
  cudaError_t e = cudaSuccess;
  BLITZ_DISPATCH_DTYPE3(dtype, (e = sized(T{})));
  return (int)e;
}

}  // extern "C"
