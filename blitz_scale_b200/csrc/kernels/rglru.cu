// Recurrent block with a real-gated linear recurrent unit: the causal short convolution in front of it and the gated
// scan over time, both for ragged batches (prompts, portions of prompts and single tokens in one launch).
//
//   u[t]  = conv_b + sum_j conv[j] * (x[t - taps + 1 + j] + x_b)       inputs before the start of the sequence: zero
//   r, i  = sigmoid(gates[t] + gate_b)                                 gates: block-diagonal product of u, done outside
//   la    = -8 r softplus(lam),   S <- e^la S + sqrt(1 - e^(2 la)) i u
//   out   = S * gelu_tanh(y + y_b)
//
// State of a sequence (by slot): S [width] in fp32 and the last taps - 1 inputs x [taps - 1][width] as projected.
// The convolution kernel only reads that history; the scan kernel, which runs after it, writes both.  A row whose
// first token has position 0 starts from nothing and reads neither.
//
// Scan: a block owns 32 channels of one row and walks its tokens in tiles; inside a tile each warp scans a few tokens,
// the warps' (product of a, end state) pairs are chained through shared memory, and every warp repeats its tokens
// with the right start value.  sqrt(1 - a^2) is taken from expm1, which keeps its digits when a is close to 1.
#include "launch.cuh"
#include "ptx.cuh"
#include "scalar.cuh"

namespace blitz {

constexpr int kMaxTaps = 16;

struct ConvParams {
  const void* x;  // [tokens][row]
  int64_t row;
  const void* x_b;
  const void* conv;    // [taps][width]
  const void* conv_b;
  const void* hist;    // [slots][taps - 1][width]
  void* u;             // [tokens][u_stride]
  int64_t u_stride;
  const int32_t* pos;
  const int32_t* tok_indptr;
  const int32_t* seq_slot;
  int num_tokens, rows, width, taps, num_slots;
  int span;  // tokens per thread
  int* status;
};

constexpr int kConvTok = 8;  // tokens a thread loads at once
constexpr int kConvThreads = 128;

// A thread computes VEC channels of `span` consecutive tokens (one token per row in decode).  The last TAPS - 1 inputs
// stay in registers; they are filled where a row's portion begins, from the history or from the sequence's start.
template <typename T, int VEC, int TAPS>
__global__ void __launch_bounds__(kConvThreads) conv_causal_kernel(const ConvParams p) {
  ptx::griddep_launch_dependents();
  ptx::griddep_wait();
  const int c = (blockIdx.x * kConvThreads + threadIdx.x) * VEC;
  if (c >= p.width) return;
  auto load = [](const T* q) { return VEC == 2 ? ldf2<T>(q) : make_float2(ldf<T>(q), 0.f); };
  const T* x = reinterpret_cast<const T*>(p.x) + c;
  const T* hist = reinterpret_cast<const T*>(p.hist) + c;
  T* u = reinterpret_cast<T*>(p.u) + c;
  float2 w[TAPS];
#pragma unroll
  for (int j = 0; j < TAPS; ++j)  // fewer taps than TAPS: the missing ones come first and are zero
    w[j] = j >= TAPS - p.taps ? load(reinterpret_cast<const T*>(p.conv) + (j - (TAPS - p.taps)) * p.width + c) : make_float2(0.f, 0.f);
  const float2 xb = load(reinterpret_cast<const T*>(p.x_b) + c), ub = load(reinterpret_cast<const T*>(p.conv_b) + c);
  const bool single = p.tok_indptr == nullptr;
  const int t0 = single ? blockIdx.y : blockIdx.y * p.span, t1 = single ? t0 + 1 : min(p.num_tokens, t0 + p.span);
  float2 in[TAPS];  // inputs with bias, oldest first; in[TAPS - 1] is the current token's
  auto fill = [&](int b, int t, int first) {  // the inputs before token t of row b, whose portion begins at token `first`
    const int slot = p.seq_slot[b], at = p.pos[t], i = t - first;
    const bool ok = slot < p.num_slots;
    if (!ok && p.status) atomicCAS(p.status, 0, kStatusBadIndex);
#pragma unroll
    for (int j = 1; j < TAPS; ++j) {
      const int back = TAPS - j;
      float2 v = make_float2(0.f, 0.f);
      if (back < p.taps && at >= back && slot >= 0 && ok) {
        const float2 raw = back <= i ? load(x + static_cast<int64_t>(t - back) * p.row)
                                     : load(hist + (static_cast<int64_t>(slot) * (p.taps - 1) + (p.taps - 1 - (back - i))) * p.width);
        v = make_float2(raw.x + xb.x, raw.y + xb.y);
      }
      in[j] = v;  // shifted down by one when the token itself comes in
    }
  };
  auto emit = [&](int t, const float2& raw) {
#pragma unroll
    for (int j = 0; j + 1 < TAPS; ++j) in[j] = in[j + 1];
    in[TAPS - 1] = make_float2(raw.x + xb.x, raw.y + xb.y);
    float2 acc = ub;
#pragma unroll
    for (int j = 0; j < TAPS; ++j) {
      acc.x += w[j].x * in[j].x;
      acc.y += w[j].y * in[j].y;
    }
    if (VEC == 2) stf2<T>(u + static_cast<int64_t>(t) * p.u_stride, acc.x, acc.y);
    else stf<T>(u + static_cast<int64_t>(t) * p.u_stride, acc.x);
  };
  if (single) {
    fill(t0, t0, t0);
    emit(t0, load(x + static_cast<int64_t>(t0) * p.row));
    return;
  }
  float2 raw[kConvTok], next[kConvTok];
  auto request = [&](int t, float2 (&dst)[kConvTok]) {
#pragma unroll
    for (int k = 0; k < kConvTok; ++k)
      dst[k] = t + k < t1 ? load(x + static_cast<int64_t>(t + k) * p.row) : make_float2(0.f, 0.f);
  };
  request(t0, raw);
  int b = row_of_token(p.tok_indptr, p.rows, t0);
  int first = p.tok_indptr[b], end = p.tok_indptr[b + 1];
  fill(b, t0, first);
  for (int base = t0; base < t1; base += kConvTok) {
    request(base + kConvTok, next);
#pragma unroll
    for (int k = 0; k < kConvTok; ++k) {
      const int t = base + k;
      if (t < t1) {
        if (t >= end) {
          do {
            ++b;
            first = end;
            end = p.tok_indptr[b + 1];
          } while (t >= end);
          fill(b, t, first);
        }
        emit(t, raw[k]);
      }
    }
#pragma unroll
    for (int k = 0; k < kConvTok; ++k) raw[k] = next[k];
  }
}

struct ScanParams {
  const void* u;
  int64_t u_stride;
  const float* gates;  // [tokens][2 * width]: per block of `block` channels, its r columns, then its i columns
  const void* gate_b;  // the same order
  const void* lam;
  const void* y;       // [tokens][row]
  const void* x;       // [tokens][row], the convolution's inputs: the last ones become the history
  int64_t row;
  const void* y_b;
  float* state;        // [slots][width]
  void* hist;          // [slots][taps - 1][width]
  void* out;           // [tokens][out_stride]
  int64_t out_stride;
  const int32_t* pos;
  const int32_t* tok_indptr;
  const int32_t* seq_slot;
  int rows, width, block, taps, num_slots;
  int* status;
};

// decay and input of one token: S <- a S + b
__device__ __forceinline__ void rglru_gates(float rate, float r, float i, float u, float& a, float& b) {
  const float la = rate * __fdividef(1.f, 1.f + __expf(-r));
  a = __expf(la);
  const float x = 2.f * la;  // 1 - a^2 = 1 - e^x, by its series where the difference would lose digits
  const float rest = x > -0.03f ? -x * (1.f + x * (0.5f + x * (0.16666667f + x * 0.041666667f))) : 1.f - a * a;
  b = ptx::sqrt_approx(rest) * __fdividef(1.f, 1.f + __expf(-i)) * u;
}
__device__ __forceinline__ float gelu_tanh_ex2(float z) {
  return 0.5f * z * (1.f + ptx::tanh_ex2(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}

// Decode: one token per row, a thread per channel.
constexpr int kStepThreads = 256;
template <typename T>
__global__ void __launch_bounds__(kStepThreads) rglru_step_kernel(const ScanParams p) {
  ptx::griddep_launch_dependents();
  ptx::griddep_wait();
  const int r = blockIdx.y, c = blockIdx.x * kStepThreads + threadIdx.x;
  const int slot = p.seq_slot[r];
  if (slot < 0 || c >= p.width) return;
  if (slot >= p.num_slots) {
    if (p.status) atomicCAS(p.status, 0, kStatusBadIndex);
    return;
  }
  const int keep = p.taps - 1;
  const int rcol = (c / p.block) * 2 * p.block + c % p.block, icol = rcol + p.block;
  float* state = p.state + static_cast<int64_t>(slot) * p.width + c;
  const float* gt = p.gates + static_cast<int64_t>(r) * 2 * p.width;
  T* hist = reinterpret_cast<T*>(p.hist) + static_cast<int64_t>(slot) * keep * p.width + c;
  const T x = reinterpret_cast<const T*>(p.x)[static_cast<int64_t>(r) * p.row + c];
  const float y = ldf<T>(reinterpret_cast<const T*>(p.y) + static_cast<int64_t>(r) * p.row + c) + ldf<T>(reinterpret_cast<const T*>(p.y_b) + c);
  float a, b;
  rglru_gates(-8.f * softplus_f(ldf<T>(reinterpret_cast<const T*>(p.lam) + c)),
              gt[rcol] + ldf<T>(reinterpret_cast<const T*>(p.gate_b) + rcol), gt[icol] + ldf<T>(reinterpret_cast<const T*>(p.gate_b) + icol),
              ldf<T>(reinterpret_cast<const T*>(p.u) + static_cast<int64_t>(r) * p.u_stride + c), a, b);
  const float S = (p.pos[r] == 0 ? 0.f : a * *state) + b;
  *state = S;
  stf<T>(reinterpret_cast<T*>(p.out) + static_cast<int64_t>(r) * p.out_stride + c, S * gelu_tanh_ex2(y));
  for (int j = 0; j + 1 < keep; ++j) hist[static_cast<int64_t>(j) * p.width] = hist[static_cast<int64_t>(j + 1) * p.width];
  if (keep > 0) hist[static_cast<int64_t>(keep - 1) * p.width] = x;
}

template <typename T, int NW, int TS>
__global__ void __launch_bounds__(NW * 32, 1) rglru_scan_kernel(const ScanParams p) {
  ptx::griddep_launch_dependents();
  ptx::griddep_wait();
  __shared__ float sA[NW][32], sB[NW][32], s_carry[2][32];
  const int r = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int c = blockIdx.x * 32 + lane;
  const bool live = c < p.width;
  const int slot = p.seq_slot[r];
  const int t_beg = p.tok_indptr[r], t_end = p.tok_indptr[r + 1];
  if (slot < 0 || t_end <= t_beg) return;
  if (slot >= p.num_slots) {
    if (threadIdx.x == 0 && p.status) atomicCAS(p.status, 0, kStatusBadIndex);
    return;
  }
  const bool fresh = p.pos[t_beg] == 0;
  const int cc = live ? c : 0;
  const int rcol = (cc / p.block) * 2 * p.block + cc % p.block, icol = rcol + p.block;
  const float rb = ldf<T>(reinterpret_cast<const T*>(p.gate_b) + rcol), ib = ldf<T>(reinterpret_cast<const T*>(p.gate_b) + icol);
  const float yb = ldf<T>(reinterpret_cast<const T*>(p.y_b) + cc);
  const float rate = -8.f * softplus_f(ldf<T>(reinterpret_cast<const T*>(p.lam) + cc));
  float* state = p.state + static_cast<int64_t>(slot) * p.width + cc;
  if (warp == 0) s_carry[0][lane] = (fresh || !live) ? 0.f : *state;
  const T* u = reinterpret_cast<const T*>(p.u) + cc;
  const T* y = reinterpret_cast<const T*>(p.y) + cc;
  T* out = reinterpret_cast<T*>(p.out) + cc;
  int cur = 0;
  float gr[TS], gi[TS], nr[TS], ni[TS];
  T uu[TS], yy[TS], nu[TS], ny[TS];
  auto request = [&](int t0, float (&r_)[TS], float (&i_)[TS], T (&u_)[TS], T (&y_)[TS]) {
#pragma unroll
    for (int s = 0; s < TS; ++s) {
      const int t = min(t0 + s, t_end - 1);
      const float* gt = p.gates + static_cast<int64_t>(t) * 2 * p.width;
      r_[s] = gt[rcol];
      i_[s] = gt[icol];
      u_[s] = u[static_cast<int64_t>(t) * p.u_stride];
      y_[s] = y[static_cast<int64_t>(t) * p.row];
    }
  };
  request(t_beg + warp * TS, gr, gi, uu, yy);
  for (int base = t_beg; base < t_end; base += NW * TS, cur ^= 1) {
    const int t0 = base + warp * TS;
    if (base + NW * TS < t_end) request(t0 + NW * TS, nr, ni, nu, ny);  // the next tile's, while this one is computed
    float A = 1.f, B = 0.f;
#pragma unroll
    for (int s = 0; s < TS; ++s) {
      float a = 1.f, b = 0.f;
      if (t0 + s < t_end) rglru_gates(rate, gr[s] + rb, gi[s] + ib, ldf<T>(&uu[s]), a, b);
      gr[s] = a;
      gi[s] = b;
      B = a * B + b;
      A *= a;
    }
    sA[warp][lane] = A;
    sB[warp][lane] = B;
    __syncthreads();
    float S = s_carry[cur][lane];
    for (int w = 0; w < warp; ++w) S = sA[w][lane] * S + sB[w][lane];
    if (warp == NW - 1) s_carry[cur ^ 1][lane] = A * S + B;
#pragma unroll
    for (int s = 0; s < TS; ++s) {
      S = gr[s] * S + gi[s];
      if (t0 + s < t_end && live) stf<T>(out + static_cast<int64_t>(t0 + s) * p.out_stride, S * gelu_tanh_ex2(ldf<T>(&yy[s]) + yb));
    }
#pragma unroll
    for (int s = 0; s < TS; ++s) {
      gr[s] = nr[s];
      gi[s] = ni[s];
      uu[s] = nu[s];
      yy[s] = ny[s];
    }
    __syncthreads();
  }
  if (warp == 0 && live) {
    *state = s_carry[cur][lane];
    // history: place j of the new one is input number n - (taps - 1) + j of the portion, or what was j + n places
    // further on in the old one (ascending order: it has not been overwritten yet)
    const int n = t_end - t_beg, keep = p.taps - 1;
    T* hist = reinterpret_cast<T*>(p.hist) + static_cast<int64_t>(slot) * keep * p.width + c;
    const T* x = reinterpret_cast<const T*>(p.x) + c;
    for (int j = 0; j < keep; ++j) {
      const int i = n - keep + j;
      hist[static_cast<int64_t>(j) * p.width] = i >= 0 ? x[static_cast<int64_t>(t_beg + i) * p.row] : hist[static_cast<int64_t>(j + n) * p.width];
    }
  }
}

template <typename T, int VEC>
static cudaError_t launch_conv(const ConvParams& p, cudaStream_t stream) {
  const int units = (p.width + VEC - 1) / VEC;
  const int spans = p.tok_indptr ? (p.num_tokens + p.span - 1) / p.span : p.num_tokens;
  const dim3 grid((units + kConvThreads - 1) / kConvThreads, spans), block(kConvThreads);
  return p.taps <= 4 ? launch_pdl(conv_causal_kernel<T, VEC, 4>, grid, block, 0, stream, p)
                     : launch_pdl(conv_causal_kernel<T, VEC, kMaxTaps>, grid, block, 0, stream, p);
}

}  // namespace blitz

extern "C" {
using namespace blitz;

int blitz_conv_causal(const void* x, int64_t row, const void* x_b, const void* conv, const void* conv_b, const void* hist,
                      void* u, int64_t u_stride, const int32_t* pos, const int32_t* tok_indptr, const int32_t* seq_slot,
                      int num_tokens, int rows, int width, int taps, int num_slots, int* status, int dtype,
                      cudaStream_t stream) {
  if (num_tokens <= 0 || rows <= 0) return 0;
  if (taps < 1 || taps > kMaxTaps) return -1;
  ConvParams p{x, row, x_b, conv, conv_b, hist, u, u_stride, pos, tok_indptr, seq_slot, num_tokens, rows, width, taps,
               num_slots, num_tokens >= 2048 ? 64 : 16, status};
  if ((tok_indptr ? num_tokens / p.span : num_tokens) >= 65535) return -1;
  cudaError_t e = cudaSuccess;
  // two channels at a time where every row starts on an even element
  const uintptr_t pair = 2 * (dtype == 2 ? 4 : 2);
  bool vec = ((width | row | u_stride) & 1) == 0;
  for (const void* q : {x, x_b, conv, conv_b, hist, (const void*)u}) vec = vec && (reinterpret_cast<uintptr_t>(q) % pair) == 0;
  if (vec) {
    BLITZ_DISPATCH_DTYPE3(dtype, (e = launch_conv<T, 2>(p, stream)));
  } else {
    BLITZ_DISPATCH_DTYPE3(dtype, (e = launch_conv<T, 1>(p, stream)));
  }
  return (int)e;
}

// single: every row has one token (decode).
int blitz_rglru_scan(const void* u, int64_t u_stride, const float* gates, const void* gate_b, const void* lam,
                     const void* y, const void* x, int64_t row, const void* y_b, float* state, void* hist, void* out,
                     int64_t out_stride, const int32_t* pos, const int32_t* tok_indptr, const int32_t* seq_slot, int rows,
                     int width, int block, int taps, int num_slots, int single, int* status, int dtype,
                     cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (block <= 0 || width % block != 0 || rows > 65535 || taps < 1 || taps > kMaxTaps) return -1;
  ScanParams p{u, u_stride, gates, gate_b, lam, y, x, row, y_b, state, hist, out, out_stride, pos, tok_indptr, seq_slot,
               rows, width, block, taps, num_slots, status};
  cudaError_t e = cudaSuccess;
  if (single) {
    const dim3 grid((width + kStepThreads - 1) / kStepThreads, rows);
    BLITZ_DISPATCH_DTYPE3(dtype, (e = launch_pdl(rglru_step_kernel<T>, grid, dim3(kStepThreads), 0, stream, p)));
  } else {
    const dim3 grid((width + 31) / 32, rows);
    BLITZ_DISPATCH_DTYPE3(dtype, (e = launch_pdl(rglru_scan_kernel<T, 32, 4>, grid, dim3(1024), 0, stream, p)));
  }
  return (int)e;
}

}  // extern "C"
