// Causal short convolutions over the rows of a step (prompts, portions of prompts and single tokens in one launch), and the mixes
// of a token's row with the one before it:
//
//   c[t]  = conv_b + sum_j conv[j] * x[t - taps + 1 + j]          inputs before the start of the sequence: zero
//   out[t] = act(c[t])                                            act: none or silu
//   out[t] = x[t] + c[t]                                          RES
//   out[t][i] = h[t] + (h[t - 1] - h[t]) mu[i],  h = x + c        mixes, one row each; h before the start of the sequence: zero
//
// State of a sequence by slot: the last taps - 1 inputs, and with mixes the last h.  The convolution only reads them, because a
// row's first tokens and its last ones belong to different threads; conv_keep, which runs after it, writes both (the last h comes
// through `last`).  With one token per row the convolution writes its history itself.  A row whose first token has position 0
// starts from nothing and reads neither.
//
// Inputs and histories may be fp32 where outputs and weights are shorter (template parameter X): what a norm gives is then rounded
// once, behind the convolution and the mixes.
//
// A thread walks `span` tokens of VEC channels with the last taps - 1 inputs in registers.
#include "launch.cuh"
#include "ptx.cuh"
#include "scalar.cuh"

namespace blitz {

constexpr int kTcvMaxTaps = 16;
constexpr int kTcvThreads = 128;
constexpr int kTcvAhead = 4;  // tokens requested at once
constexpr int kTcvMaxMixes = 8;

struct TokenConvParams {
  const void* x;  // [tokens][row]
  int64_t row;
  const void *conv, *conv_b;  // [taps][width], [width] or null
  void* hist;                 // [slots][taps - 1][width]
  void* out;                  // [tokens][out_row]; mixes: [tokens][mixes][width]
  int64_t out_row;
  const void* mu;             // [mixes][width]
  const void* shift;          // [slots][width]
  void* last;                 // [rows][width]: h of every row's last token
  const int32_t *pos, *tok_indptr, *seq_slot;
  int num_tokens, rows, width, taps, num_slots, span, silu, residual, mixes;
  int* status;
};

template <typename T, int VEC>
struct TcvCols {
  float v[VEC];
  __device__ __forceinline__ void load(const T* p) {
    if constexpr (VEC == 8) {
      ldf8<T>(p, v);
    } else if constexpr (VEC == 4) {
      const float4 a = ldf4<T>(p);
      v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
    } else {
      v[0] = ldf<T>(p);
    }
  }
  __device__ __forceinline__ void store(T* p) const {
    if constexpr (VEC == 8) stf8<T>(p, v);
    else if constexpr (VEC == 4) stf4<T>(p, make_float4(v[0], v[1], v[2], v[3]));
    else stf<T>(p, v[0]);
  }
};

template <typename T, typename X, int VEC, int TAPS>
__global__ void __launch_bounds__(kTcvThreads) token_conv_kernel(const TokenConvParams p) {
  using C = TcvCols<T, VEC>;
  using I = TcvCols<X, VEC>;
  ptx::griddep_launch_dependents();
  const int c = (blockIdx.x * kTcvThreads + threadIdx.x) * VEC;
  const int64_t W = p.width;
  const bool on = c < p.width;
  C w[TAPS], wb = {};
  if (on) {  // weights are not written by kernels still running
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {  // fewer taps than TAPS: the missing ones come first and are zero
      w[j] = {};
      if (j >= TAPS - p.taps) w[j].load(reinterpret_cast<const T*>(p.conv) + (j - (TAPS - p.taps)) * W + c);
    }
    if (p.conv_b) wb.load(reinterpret_cast<const T*>(p.conv_b) + c);
  }
  ptx::griddep_wait();
  if (!on) return;
  const X* x = reinterpret_cast<const X*>(p.x) + c;
  X* hist = reinterpret_cast<X*>(p.hist) + c;
  T* out = reinterpret_cast<T*>(p.out) + c;
  const bool single = p.tok_indptr == nullptr;
  const int t0 = single ? blockIdx.y : blockIdx.y * p.span, t1 = single ? t0 + 1 : min(p.num_tokens, t0 + p.span);
  I in[TAPS];  // inputs, oldest first; in[TAPS - 1] is the current token's
  auto slot_of = [&](int b) {
    const int slot = p.seq_slot[b];
    if (slot >= p.num_slots) {
      if (p.status && c == 0) atomicCAS(p.status, 0, kStatusBadIndex);
      return -1;
    }
    return slot;
  };
  auto fill = [&](int b, int t, int first) {  // the inputs before token t of row b, whose portion begins at token `first`
    const int slot = slot_of(b), at = p.pos[first] + t - first, i = t - first;
#pragma unroll
    for (int j = 1; j < TAPS; ++j) {
      const int back = TAPS - j;
      in[j] = {};  // (shifted down by one when the token itself comes in)
      if (back < p.taps && at >= back) {
        if (back <= i) in[j].load(x + (t - back) * p.row);
        else if (slot >= 0) in[j].load(hist + (static_cast<int64_t>(slot) * (p.taps - 1) + (p.taps - 1 - (back - i))) * W);
      }
    }
  };
  auto convolve = [&](const I& raw) {
#pragma unroll
    for (int j = 0; j + 1 < TAPS; ++j) in[j] = in[j + 1];
    in[TAPS - 1] = raw;
    C a = wb;
#pragma unroll
    for (int j = 0; j < TAPS; ++j)
#pragma unroll
      for (int k = 0; k < VEC; ++k) a.v[k] = fmaf(w[j].v[k], in[j].v[k], a.v[k]);
    if (p.silu)
#pragma unroll
      for (int k = 0; k < VEC; ++k) a.v[k] = __fdividef(a.v[k], 1.f + __expf(fminf(-a.v[k], 80.f)));
    if (p.residual)
#pragma unroll
      for (int k = 0; k < VEC; ++k) a.v[k] += raw.v[k];
    return a;
  };
  if (single) {
    I raw;
    raw.load(x + t0 * p.row);
    fill(t0, t0, t0);
    const int slot = slot_of(t0);
    convolve(raw).store(out + t0 * p.out_row);
    if (slot >= 0)
#pragma unroll
      for (int j = 1; j < TAPS; ++j)
        if (j >= TAPS - p.taps + 1) in[j].store(hist + (static_cast<int64_t>(slot) * (p.taps - 1) + j - (TAPS - p.taps + 1)) * W);
    return;
  }
  auto as_input = [](const C& a) {
    I b;
#pragma unroll
    for (int k = 0; k < VEC; ++k) b.v[k] = a.v[k];
    return b;
  };
  I prev = {};
  int b = row_of_token(p.tok_indptr, p.rows, t0);
  int first = p.tok_indptr[b], end = p.tok_indptr[b + 1];
  auto begin = [&](int t) {  // token t is the first one here of row b
    if (p.mixes > 0) {
      prev = {};
      if (t > first) {
        I raw;
        raw.load(x + (t - 1) * p.row);
        fill(b, t - 1, first);
        prev = as_input(convolve(raw));
        return;  // (its inputs are the ones before token t)
      }
      const int slot = slot_of(b);
      if (slot >= 0 && p.pos[first] > 0) prev.load(reinterpret_cast<const X*>(p.shift) + slot * W + c);
    }
    fill(b, t, first);
  };
  begin(t0);
  for (int base = t0; base < t1; base += kTcvAhead) {
    I raw[kTcvAhead];
#pragma unroll
    for (int k = 0; k < kTcvAhead; ++k) {
      raw[k] = {};
      if (base + k < t1) raw[k].load(x + (base + k) * p.row);
    }
#pragma unroll
    for (int k = 0; k < kTcvAhead; ++k) {
      const int t = base + k;
      if (t >= t1) continue;
      if (t >= end) {
        do {
          ++b;
          first = end;
          end = p.tok_indptr[b + 1];
        } while (t >= end);
        begin(t);
      }
      const C a = convolve(raw[k]);
      if (p.mixes == 0) {
        a.store(out + t * p.out_row);
        continue;
      }
      const I h = as_input(a);
      for (int m = 0; m < p.mixes; ++m) {
        C mu;
        mu.load(reinterpret_cast<const T*>(p.mu) + m * W + c);
#pragma unroll
        for (int i = 0; i < VEC; ++i) mu.v[i] = fmaf(prev.v[i] - h.v[i], mu.v[i], h.v[i]);
        mu.store(out + t * p.out_row + m * W);
      }
      if (t + 1 == end) h.store(reinterpret_cast<X*>(p.last) + b * W + c);
      prev = h;
    }
  }
}

// Histories after the step: place j of a row's history is its input number n - (taps - 1) + j of this portion, or what was n
// places further on; the last h comes from `last`.
template <typename T>
__global__ void __launch_bounds__(256) conv_keep_kernel(const TokenConvParams p) {
  ptx::griddep_launch_dependents();
  ptx::griddep_wait();
  const int r = blockIdx.y, c = blockIdx.x * 256 + threadIdx.x;
  const int beg = p.tok_indptr[r], n = p.tok_indptr[r + 1] - beg, slot = p.seq_slot[r];
  if (c >= p.width || n <= 0 || slot < 0 || slot >= p.num_slots) return;
  const int64_t W = p.width;
  const int keep = p.taps - 1;
  T* hist = reinterpret_cast<T*>(p.hist) + static_cast<int64_t>(slot) * keep * W + c;
  const T* x = reinterpret_cast<const T*>(p.x) + c;
  for (int j = 0; j < keep; ++j) {  // ascending: what is read has not been overwritten yet
    const int i = n - keep + j;
    hist[j * W] = i >= 0 ? x[(beg + i) * p.row] : hist[(j + n) * W];
  }
  if (p.mixes > 0) const_cast<T*>(reinterpret_cast<const T*>(p.shift))[slot * W + c] = reinterpret_cast<const T*>(p.last)[r * W + c];
}

template <typename T, typename X, int VEC>
static cudaError_t launch_token_conv(const TokenConvParams& p, cudaStream_t stream) {
  const int units = (p.width + VEC - 1) / VEC;
  const int spans = p.tok_indptr ? (p.num_tokens + p.span - 1) / p.span : p.num_tokens;
  const dim3 grid((units + kTcvThreads - 1) / kTcvThreads, spans), block(kTcvThreads);
  return p.taps <= 4 ? launch_pdl(token_conv_kernel<T, X, VEC, 4>, grid, block, 0, stream, p)
                     : launch_pdl(token_conv_kernel<T, X, (VEC > 4 ? 4 : VEC), kTcvMaxTaps>, dim3((p.width / (VEC > 4 ? 4 : VEC) + kTcvThreads) / kTcvThreads, spans),
                                  block, 0, stream, p);
}

}  // namespace blitz

extern "C" {
using namespace blitz;

// See the top of the file; everything in the activation type (dtype 0 fp16, 1 bf16, 2 fp32), but with x32 x, hist, shift and last in
// fp32.  tok_indptr null: one token per row
// (no mixes then).  With tok_indptr the histories are brought up to date by a second launch.
int blitz_token_conv(const void* x, int64_t row, const void* conv, const void* conv_b, void* hist, void* out, int64_t out_row,
                     int silu, int residual, int x32, const void* mu, int mixes, void* shift, void* last, const int32_t* pos,
                     const int32_t* tok_indptr, const int32_t* seq_slot, int num_tokens, int rows, int width, int taps, int num_slots,
                     int* status, int dtype, cudaStream_t stream) {
  if (num_tokens <= 0 || rows <= 0) return 0;
  if (taps < 1 || taps > kTcvMaxTaps || width < 1 || mixes < 0 || mixes > kTcvMaxMixes || (taps > 1 && hist == nullptr)) return -1;
  if (mixes > 0 && (tok_indptr == nullptr || mu == nullptr || shift == nullptr || last == nullptr || out_row < (int64_t)mixes * width)) return -1;
  TokenConvParams p{x, row, conv, conv_b, hist, out, out_row, mu, shift, last, pos, tok_indptr, seq_slot,
                    num_tokens, rows, width, taps, num_slots, num_tokens >= 2048 ? 32 : 8, silu, residual, mixes, status};
  if ((tok_indptr ? num_tokens / p.span : num_tokens) >= 65535 || rows > 65535) return -1;
  const int es = dtype == 2 ? 4 : 2, xs = x32 ? 4 : es;
  auto all = [&](int v) {
    bool ok = ((width | row | out_row) & (v - 1)) == 0;
    for (const void* q : {conv, conv_b, (const void*)out, mu}) ok = ok && (reinterpret_cast<uintptr_t>(q) % (v * es)) == 0;
    for (const void* q : {x, (const void*)hist, (const void*)shift, (const void*)last}) ok = ok && (reinterpret_cast<uintptr_t>(q) % (v * xs)) == 0;
    return ok;
  };
  const int vec = all(8) && (int64_t)num_tokens * width >= (1 << 20) ? 8 : all(4) ? 4 : 1;
  cudaError_t e = cudaSuccess;
  auto go = [&](auto type, auto input) -> cudaError_t {
    using T = decltype(type);
    using X = decltype(input);
    return vec == 8 ? launch_token_conv<T, X, 8>(p, stream) : vec == 4 ? launch_token_conv<T, X, 4>(p, stream) : launch_token_conv<T, X, 1>(p, stream);
  };
  BLITZ_DISPATCH_DTYPE3(dtype, (e = x32 ? go(T{}, float{}) : go(T{}, T{})));
  if (e != cudaSuccess || tok_indptr == nullptr || (taps < 2 && mixes == 0)) return (int)e;
  const dim3 grid((width + 255) / 256, rows);
  BLITZ_DISPATCH_DTYPE3(x32 ? 2 : dtype, (e = launch_pdl(conv_keep_kernel<T>, grid, dim3(256), 0, stream, p)));
  return (int)e;
}

}  // extern "C"
