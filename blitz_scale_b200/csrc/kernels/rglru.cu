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
  int* status;
};

constexpr int kConvTok = 8;  // tokens per thread

template <typename T>
__global__ void __launch_bounds__(128) conv_causal_kernel(const ConvParams p) {
  ptx::griddep_launch_dependents();
  ptx::griddep_wait();
  const int c = blockIdx.x * blockDim.x + threadIdx.x;
  if (c >= p.width) return;
  const int t0 = blockIdx.y * kConvTok, t1 = min(p.num_tokens, t0 + kConvTok);
  const T* x = reinterpret_cast<const T*>(p.x) + c;
  const T* hist = reinterpret_cast<const T*>(p.hist) + c;
  float w[kMaxTaps];
#pragma unroll
  for (int j = 0; j < kMaxTaps; ++j) w[j] = j < p.taps ? ldf<T>(reinterpret_cast<const T*>(p.conv) + j * p.width + c) : 0.f;
  const float xb = ldf<T>(reinterpret_cast<const T*>(p.x_b) + c), ub = ldf<T>(reinterpret_cast<const T*>(p.conv_b) + c);
  int b = p.tok_indptr ? row_of_token(p.tok_indptr, p.rows, t0) : t0;
  for (int t = t0; t < t1; ++t) {
    if (p.tok_indptr) {
      while (b + 1 < p.rows && p.tok_indptr[b + 1] <= t) ++b;
    } else {
      b = t;
    }
    const int i = p.tok_indptr ? t - p.tok_indptr[b] : 0;  // place in the row's portion
    const int slot = p.seq_slot[b], at = p.pos[t];
    float acc = ub;
    if (slot >= 0) {
      if (slot >= p.num_slots) {
        if (p.status) atomicCAS(p.status, 0, kStatusBadIndex);
        continue;
      }
#pragma unroll
      for (int j = 0; j < kMaxTaps; ++j) {
        if (j >= p.taps) break;
        const int back = p.taps - 1 - j;
        if (at < back) continue;  // before the start of the sequence
        const float v = back <= i ? ldf<T>(x + (t - back) * p.row)
                                  : ldf<T>(hist + (static_cast<int64_t>(slot) * (p.taps - 1) + (p.taps - 1 - (back - i))) * p.width);
        acc += w[j] * (v + xb);
      }
    }
    stf<T>(reinterpret_cast<T*>(p.u) + t * p.u_stride + c, acc);
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

template <typename T, int NW, int TS>
__global__ void __launch_bounds__(NW * 32) rglru_scan_kernel(const ScanParams p) {
  ptx::griddep_launch_dependents();
  ptx::griddep_wait();
  __shared__ float sA[NW][32], sB[NW][32], s_carry[2][32];
  const int r = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
  const int c = blockIdx.x * 32 + lane;
  const bool live = c < p.width;
  const int slot = p.seq_slot[r];
  const int t_beg = p.tok_indptr ? p.tok_indptr[r] : r, t_end = p.tok_indptr ? p.tok_indptr[r + 1] : r + 1;
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
  for (int base = t_beg; base < t_end; base += NW * TS, cur ^= 1) {
    float a[TS], b[TS];
    float A = 1.f, B = 0.f;
#pragma unroll
    for (int s = 0; s < TS; ++s) {
      const int t = base + warp * TS + s;
      a[s] = 1.f;
      b[s] = 0.f;
      if (t < t_end && live) {
        const float* gt = p.gates + static_cast<int64_t>(t) * 2 * p.width;
        const float la = rate * sigmoid_f(gt[rcol] + rb);
        a[s] = expf(la);
        b[s] = sqrtf(-expm1f(2.f * la)) * sigmoid_f(gt[icol] + ib) * ldf<T>(u + t * p.u_stride);
      }
      B = a[s] * B + b[s];
      A *= a[s];
    }
    sA[warp][lane] = A;
    sB[warp][lane] = B;
    __syncthreads();
    float S = s_carry[cur][lane];
    for (int w = 0; w < warp; ++w) S = sA[w][lane] * S + sB[w][lane];
    if (warp == NW - 1) s_carry[cur ^ 1][lane] = A * S + B;
#pragma unroll
    for (int s = 0; s < TS; ++s) {
      const int t = base + warp * TS + s;
      S = a[s] * S + b[s];
      if (t < t_end && live) stf<T>(out + t * p.out_stride, S * gelu_tanh_f(ldf<T>(y + t * p.row) + yb));
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
      hist[static_cast<int64_t>(j) * p.width] = i >= 0 ? x[(t_beg + i) * p.row] : hist[static_cast<int64_t>(j + n) * p.width];
    }
  }
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
               num_slots, status};
  const dim3 grid((width + 127) / 128, (num_tokens + kConvTok - 1) / kConvTok);
  cudaError_t e = cudaSuccess;
  BLITZ_DISPATCH_DTYPE3(dtype, (e = launch_pdl(conv_causal_kernel<T>, grid, dim3(128), 0, stream, p)));
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
  const dim3 grid((width + 31) / 32, rows);
  cudaError_t e = cudaSuccess;
  if (single) {
    BLITZ_DISPATCH_DTYPE3(dtype, (e = launch_pdl(rglru_scan_kernel<T, 1, 1>, grid, dim3(32), 0, stream, p)));
  } else {
    BLITZ_DISPATCH_DTYPE3(dtype, (e = launch_pdl(rglru_scan_kernel<T, 16, 4>, grid, dim3(512), 0, stream, p)));
  }
  return (int)e;
}

}  // extern "C"
