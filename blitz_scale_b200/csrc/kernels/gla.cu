// Gated linear attention, token by token (decode, fp32 mode, sizes the chunked kernel does not take).
//
// Per head a state S [dim][vdim] in fp32 that decays per key channel:
//
//   alpha = sigmoid(low A2 + b)^(1/tau)         low: the rank-r projection of the token
//   S    <- diag(alpha) S + k v^T,   o = S^T q * q_scale
//   out   = o / rms(o) * w * silu(g)
//
// Second form (WKV): the output sees the state before the token, plus the token itself with a bonus of its own per key channel,
// and the decay comes from a doubly exponential map (the recurrence of RWKV-6):
//
//   alpha = exp(-exp(tanh(low) A2 + b))         low: fp32
//   o     = (S + diag(u) k v^T)^T q * q_scale,  S <- diag(alpha) S + k v^T
//
// A block owns one (sequence row, head): decay projection, recurrence, output norm and gate are one kernel, so a
// decoded token costs one read and one write of the state and nothing else of that size.  The state slot of the row
// comes from seq_slot (negative: padding row, nothing happens); a row whose first token has position 0 starts from
// zero and does not read its slot, so a slot needs no clearing when it changes hands.
//
// In decode the state stays in global memory (read once, written once, straight through registers); for longer rows
// it is kept in shared memory from the first token to the last when it fits.
#include "launch.cuh"
#include "ptx.cuh"
#include "scalar.cuh"

namespace blitz {

constexpr int kGlaThreads = 256;

struct GlaParams {
  const void* q;   // [tokens][row]: heads x dim
  const void* k;
  const void* v;   // heads x vdim
  const void* g;   // heads x vdim
  const void* low; // rank (WKV: fp32)
  int64_t row, low_row;  // row pitch of the first four, and of low
  const void* a2;  // [rank][heads * dim]
  const void* a2_b;
  const void* norm;  // [vdim], head h's from h * norm_step on
  const void* bonus; // [heads * dim], WKV only
  float* state;    // [slots][heads][dim][vdim]
  void* out;       // [tokens][out_stride]: heads x vdim
  int64_t out_stride;
  const int32_t* pos;
  const int32_t* tok_indptr;  // null: row r is token r
  const int32_t* seq_slot;
  int rows, heads, dim, vdim, rank, num_slots, in_shared, norm_step;
  float q_scale, inv_tau, eps;
  int* status;
};

// VEC: value columns a thread handles at once.
template <typename T, int VEC, bool WKV>
__global__ void __launch_bounds__(kGlaThreads) gla_recurrent_kernel(const GlaParams p) {
  ptx::griddep_launch_dependents();
  ptx::griddep_wait();
  extern __shared__ __align__(16) float sm[];
  const int K = p.dim, V = p.vdim;
  const int Kp = (K + 3) & ~3;   // everything behind the three vectors stays 16-byte aligned
  float* s_alpha = sm;           // [Kp]
  float* s_k = s_alpha + Kp;     // [Kp]
  float* s_q = s_k + Kp;         // [Kp]
  float* s_bonus = s_q + Kp;     // [Kp] WKV: u * k
  float* s_low = s_bonus + (WKV ? Kp : 0);  // [rank] WKV: tanh(low)
  float* s_red = s_low + (WKV ? (p.rank + 3) & ~3 : 0);  // [40]
  float* s_o = s_red + 40;       // [kGlaThreads * VEC]
  float* s_state = s_o + kGlaThreads * VEC;
  const int r = blockIdx.x, h = blockIdx.y, tid = threadIdx.x;
  const int slot = p.seq_slot[r];
  if (slot < 0) return;
  if (slot >= p.num_slots) {
    if (tid == 0 && p.status) atomicCAS(p.status, 0, kStatusBadIndex);
    return;
  }
  const int t_beg = p.tok_indptr ? p.tok_indptr[r] : r, t_end = p.tok_indptr ? p.tok_indptr[r + 1] : r + 1;
  if (t_end <= t_beg) return;
  float* gstate = p.state + (static_cast<int64_t>(slot) * p.heads + h) * K * V;
  bool fresh = p.pos[t_beg] == 0;
  const bool keep = p.in_shared != 0;
  if (keep) {
    for (int i = tid; i < K * V; i += kGlaThreads) s_state[i] = fresh ? 0.f : gstate[i];
    fresh = false;
  }
  float* S = keep ? s_state : gstate;
  const int nv = (V + VEC - 1) / VEC;            // groups of value columns
  const int cols = nv < kGlaThreads ? nv : kGlaThreads;
  const int parts = kGlaThreads / cols;          // threads along the key dimension
  const int part = tid / cols, col = tid % cols;
  const T* a2 = reinterpret_cast<const T*>(p.a2) + h * K;
  const T* a2_b = reinterpret_cast<const T*>(p.a2_b) + h * K;
  const T* norm = reinterpret_cast<const T*>(p.norm) + static_cast<int64_t>(h) * p.norm_step;
  const T* bonus = reinterpret_cast<const T*>(p.bonus) + h * K;
  for (int t = t_beg; t < t_end; ++t) {
    const T* q = reinterpret_cast<const T*>(p.q) + t * p.row + h * K;
    const T* k = reinterpret_cast<const T*>(p.k) + t * p.row + h * K;
    const T* v = reinterpret_cast<const T*>(p.v) + t * p.row + static_cast<int64_t>(h) * V;
    const T* g = reinterpret_cast<const T*>(p.g) + t * p.row + static_cast<int64_t>(h) * V;
    const T* low = reinterpret_cast<const T*>(p.low) + t * p.low_row;
    if (WKV) {
      for (int i = tid; i < p.rank; i += kGlaThreads) s_low[i] = tanhf(reinterpret_cast<const float*>(p.low)[t * p.low_row + i]);
      __syncthreads();
    }
    for (int c = tid; c < K; c += kGlaThreads) {
      float z = ldf<T>(a2_b + c);
      for (int i = 0; i < p.rank; ++i) z += (WKV ? s_low[i] : ldf<T>(low + i)) * ldf<T>(a2 + static_cast<int64_t>(i) * p.heads * K + c);
      s_alpha[c] = WKV ? expf(-expf(z)) : expf(log_sigmoid(z) * p.inv_tau);
      s_k[c] = ldf<T>(k + c);
      s_q[c] = ldf<T>(q + c) * p.q_scale;
      if (WKV) s_bonus[c] = ldf<T>(bonus + c) * s_k[c];
    }
    __syncthreads();
    float ss = 0.f;
    for (int c0 = 0; c0 < nv; c0 += cols) {      // one round unless there are more groups than threads
      const int vg = (c0 + col) * VEC;
      float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
      if (part < parts && c0 + col < nv) {
        if (VEC == 4) {
          const float4 vv = ldf4<T>(v + vg);
#pragma unroll 4
          for (int c = part; c < K; c += parts) {
            float4* sp = reinterpret_cast<float4*>(S + static_cast<int64_t>(c) * V + vg);
            float4 s = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : *sp;
            const float a = s_alpha[c], kk = s_k[c], qq = s_q[c];
            if (WKV) {
              const float b = s_bonus[c];
              o.x += qq * (s.x + b * vv.x); o.y += qq * (s.y + b * vv.y); o.z += qq * (s.z + b * vv.z); o.w += qq * (s.w + b * vv.w);
            }
            s.x = a * s.x + kk * vv.x; s.y = a * s.y + kk * vv.y; s.z = a * s.z + kk * vv.z; s.w = a * s.w + kk * vv.w;
            *sp = s;
            if (!WKV) {
              o.x += qq * s.x; o.y += qq * s.y; o.z += qq * s.z; o.w += qq * s.w;
            }
          }
        } else {
          const float vv = ldf<T>(v + vg);
          for (int c = part; c < K; c += parts) {
            float* sp = S + static_cast<int64_t>(c) * V + vg;
            const float old = fresh ? 0.f : *sp, s = s_alpha[c] * old + s_k[c] * vv;
            *sp = s;
            o.x += s_q[c] * (WKV ? old + s_bonus[c] * vv : s);
          }
        }
      }
      if (VEC == 4) *reinterpret_cast<float4*>(s_o + tid * 4) = o;
      else s_o[tid] = o.x;
      __syncthreads();
      // sum over the parts; thread c of the first `cols` keeps its group's sums in the first part's place
      if (part == 0 && c0 + col < nv) {
        for (int i = 1; i < parts; ++i)
#pragma unroll
          for (int j = 0; j < VEC; ++j) s_o[tid * VEC + j] += s_o[(i * cols + col) * VEC + j];
#pragma unroll
        for (int j = 0; j < VEC; ++j) ss += s_o[tid * VEC + j] * s_o[tid * VEC + j];
      }
      if (nv > cols) {  // more than one round: park the sums in the output row until the norm is known
        if (part == 0 && c0 + col < nv)
          for (int j = 0; j < VEC; ++j) s_state[(keep ? K * V : 0) + vg + j] = s_o[tid * VEC + j];
        __syncthreads();
      }
    }
    const float scale = rsqrtf(block_sum(ss, s_red) / static_cast<float>(V) + p.eps);
    const float* o_row = nv > cols ? s_state + (keep ? K * V : 0) : s_o;
    T* out = reinterpret_cast<T*>(p.out) + t * p.out_stride + static_cast<int64_t>(h) * V;
    for (int c = tid; c < V; c += kGlaThreads)
      stf<T>(out + c, o_row[c] * scale * ldf<T>(norm + c) * silu_acc(ldf<T>(g + c)));
    fresh = false;
    __syncthreads();
  }
  if (keep)
    for (int i = tid; i < K * V; i += kGlaThreads) gstate[i] = s_state[i];
}

template <typename T, int VEC, bool WKV>
static cudaError_t launch_gla_recurrent(GlaParams p, bool multi, cudaStream_t stream) {
  const size_t base = ((WKV ? 4 : 3) * (size_t)((p.dim + 3) & ~3) + (WKV ? (size_t)((p.rank + 3) & ~3) : 0) + 40 + (size_t)kGlaThreads * VEC) * sizeof(float);
  const size_t park = (p.vdim + VEC - 1) / VEC > kGlaThreads ? (size_t)p.vdim * sizeof(float) : 0;
  const size_t whole = base + park + (size_t)p.dim * p.vdim * sizeof(float);
  constexpr size_t kLimit = 200 * 1024;
  p.in_shared = multi && whole <= kLimit;
  const size_t smem = p.in_shared ? whole : base + park;
  if (smem > kLimit) return cudaErrorInvalidValue;
  auto kern = gla_recurrent_kernel<T, VEC, WKV>;
  static PerDeviceOnce once;
  cudaError_t e = once.run([&] { return cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kLimit); });
  if (e != cudaSuccess) return e;
  return launch_pdl(kern, dim3(p.rows, p.heads), dim3(kGlaThreads), smem, stream, p);
}

template <bool WKV>
static int gla_recurrent_any(const GlaParams& p, int multi, int dtype, cudaStream_t stream) {
  cudaError_t e = cudaSuccess;
  // four value columns at a time where every row of v (and of the state) starts on a multiple of four elements
  const int es = dtype == 2 ? 4 : 2;
  const bool vec = (p.vdim & 3) == 0 && (p.row & 3) == 0 && (reinterpret_cast<uintptr_t>(p.v) % (4 * es)) == 0;
  if (vec) {
    BLITZ_DISPATCH_DTYPE3(dtype, (e = launch_gla_recurrent<T, 4, WKV>(p, multi != 0, stream)));
  } else {
    BLITZ_DISPATCH_DTYPE3(dtype, (e = launch_gla_recurrent<T, 1, WKV>(p, multi != 0, stream)));
  }
  return (int)e;
}

}  // namespace blitz

extern "C" {
using namespace blitz;

int blitz_gla_recurrent(const void* q, const void* k, const void* v, const void* g, const void* low, int64_t row,
                        const void* a2, const void* a2_b, const void* norm, float* state, void* out, int64_t out_stride,
                        const int32_t* pos, const int32_t* tok_indptr, const int32_t* seq_slot, int rows, int heads,
                        int dim, int vdim, int rank, int num_slots, float q_scale, float tau, float eps, int multi,
                        int* status, int dtype, cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (dim <= 0 || vdim <= 0 || heads <= 0 || heads > 65535 || !(tau > 0.f)) return -1;
  GlaParams p{q, k, v, g, low, row, row, a2, a2_b, norm, nullptr, state, out, out_stride, pos, tok_indptr, seq_slot, rows, heads, dim,
              vdim, rank, num_slots, 0, 0, q_scale, 1.f / tau, eps, status};
  return gla_recurrent_any<false>(p, multi, dtype, stream);
}

// The second form: low fp32 [tokens][low_row], a2 / a2_b of the decay's exponent, bonus [heads * dim], norm [heads * vdim].
int blitz_wkv_recurrent(const void* q, const void* k, const void* v, const void* g, int64_t row, const float* low, int64_t low_row,
                        const void* a2, const void* a2_b, const void* bonus, const void* norm, float* state, void* out,
                        int64_t out_stride, const int32_t* pos, const int32_t* tok_indptr, const int32_t* seq_slot, int rows,
                        int heads, int dim, int vdim, int rank, int num_slots, float eps, int multi, int* status, int dtype,
                        cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (dim <= 0 || vdim <= 0 || heads <= 0 || heads > 65535) return -1;
  GlaParams p{q, k, v, g, low, row, low_row, a2, a2_b, norm, bonus, state, out, out_stride, pos, tok_indptr, seq_slot, rows, heads, dim,
              vdim, rank, num_slots, 0, vdim, 1.f, 1.f, eps, status};
  return gla_recurrent_any<true>(p, multi, dtype, stream);
}

}  // extern "C"
