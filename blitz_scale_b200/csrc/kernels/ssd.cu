// State-space recurrence with a scalar decay per head (the recurrence of Mamba-2) and the gated group norm behind it.
//
// Per head a state S [state][vdim] in fp32; heads share B and C in groups (head h: group h / (heads / groups)):
//
//   dt  = softplus(dt_raw + dt_bias),   a = exp(-exp(A_log) dt)
//   S  <- a S + dt B x^T,               y = (S^T C + D x) silu(z)
//
// x, B and C come out of a short convolution (token_conv.cu).  y leaves the recurrence gated, in the activation type; the norm
// (ssd_norm) works on it in place, in equal parts of the row.
//
// ssd_recurrent: token by token (decode, fp32 mode, sizes the chunked form does not take); a block owns a (row, head).  In
// decode the state is read once and written once, straight through registers; for longer rows it stays in shared memory if it fits.
//
// ssd_chunk: prompts in bf16, in chunks of 64 tokens on the tensor cores (the chunkwise form of Dao and Gu, "Transformers are
// SSMs: Generalized Models and Efficient Algorithms Through Structured State Space Duality").  With b_t the running sum of the
// log decays within the chunk:
//
//   y_t   = e^(b_t) C_t^T S_0 + sum_{s <= t} (C_t . B_s) e^(b_t - b_s) dt_s x_s
//   S_end = e^(b_end) S_0 + sum_s B_s (e^(b_end - b_s) dt_s x_s)^T
//
// Every exponent is <= 0, so the decay is a factor per score and per row.  Decays, their sums, dt and the state are fp32;
// products with an fp32 operand split it into two bf16 numbers (x = hi + lo, relative error 2^-17); C . B is a product of
// 16-bit activations.  A block of 8 warps owns (row, head, up to 64 or 128 value columns) with the state in registers and
// fetches the next chunk's tiles while it works on this one.
#include "launch.cuh"
#include "mma.cuh"
#include "ptx.cuh"
#include "scalar.cuh"
#include "tmap.cuh"

namespace blitz {

constexpr int kSsdThreads = 256;

struct SsdParams {
  const void* x;    // [tokens][x_row]: heads x vdim
  const void* B;    // groups x state
  const void* C;    // groups x state
  int64_t x_row;    // row pitch of the three
  const void* z;    // [tokens][z_row]: heads x vdim
  const void* dt;   // heads
  int64_t z_row;    // row pitch of the two
  const void *dt_bias, *A_log, *D;  // [heads]
  float* state;     // [slots][heads][state][vdim]
  void* out;        // [tokens][out_stride]: heads x vdim
  int64_t out_stride;
  const int32_t *pos, *tok_indptr, *seq_slot;
  int rows, heads, groups, dim, vdim, num_slots, in_shared;
  int* status;
};

template <typename T, int VEC>
__global__ void __launch_bounds__(kSsdThreads) ssd_recurrent_kernel(const SsdParams p) {
  ptx::griddep_launch_dependents();
  ptx::griddep_wait();
  extern __shared__ __align__(16) float sm[];
  const int K = p.dim, V = p.vdim, Kp = (K + 3) & ~3;
  float* s_b = sm;           // [Kp] dt B
  float* s_c = s_b + Kp;     // [Kp]
  float* s_o = s_c + Kp;     // [kSsdThreads * VEC]
  float* s_state = s_o + kSsdThreads * VEC;
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
    for (int i = tid; i < K * V; i += kSsdThreads) s_state[i] = fresh ? 0.f : gstate[i];
    fresh = false;
  }
  float* S = keep ? s_state : gstate;
  const int nv = (V + VEC - 1) / VEC;  // groups of value columns
  const int cols = nv < kSsdThreads ? nv : kSsdThreads, parts = kSsdThreads / cols;
  const int part = tid / cols, col = tid % cols;
  const int grp = h / (p.heads / p.groups);
  const float rate = -expf(ldf<T>(reinterpret_cast<const T*>(p.A_log) + h)), bias = ldf<T>(reinterpret_cast<const T*>(p.dt_bias) + h),
              skip = ldf<T>(reinterpret_cast<const T*>(p.D) + h);
  for (int t = t_beg; t < t_end; ++t) {
    const T* x = reinterpret_cast<const T*>(p.x) + t * p.x_row + static_cast<int64_t>(h) * V;
    const T* B = reinterpret_cast<const T*>(p.B) + t * p.x_row + static_cast<int64_t>(grp) * K;
    const T* C = reinterpret_cast<const T*>(p.C) + t * p.x_row + static_cast<int64_t>(grp) * K;
    const T* z = reinterpret_cast<const T*>(p.z) + t * p.z_row + static_cast<int64_t>(h) * V;
    T* out = reinterpret_cast<T*>(p.out) + t * p.out_stride + static_cast<int64_t>(h) * V;
    const float dt = softplus_f(ldf<T>(reinterpret_cast<const T*>(p.dt) + t * p.z_row + h) + bias);
    const float a = expf(rate * dt);
    for (int c = tid; c < K; c += kSsdThreads) {
      s_b[c] = dt * ldf<T>(B + c);
      s_c[c] = ldf<T>(C + c);
    }
    __syncthreads();
    for (int c0 = 0; c0 < nv; c0 += cols) {
      const int vg = (c0 + col) * VEC;
      const bool on = part < parts && c0 + col < nv;
      float xx[VEC], o[VEC];
#pragma unroll
      for (int j = 0; j < VEC; ++j) o[j] = 0.f;
      if (on) {
        if constexpr (VEC == 4) {
          const float4 f = ldf4<T>(x + vg);
          xx[0] = f.x; xx[1] = f.y; xx[2] = f.z; xx[3] = f.w;
        } else {
          xx[0] = ldf<T>(x + vg);
        }
#pragma unroll 4
        for (int c = part; c < K; c += parts) {
          float* sp = S + static_cast<int64_t>(c) * V + vg;
          const float b = s_b[c], q = s_c[c];
          if constexpr (VEC == 4) {
            float4 s = fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<float4*>(sp);
            s.x = a * s.x + b * xx[0]; s.y = a * s.y + b * xx[1]; s.z = a * s.z + b * xx[2]; s.w = a * s.w + b * xx[3];
            *reinterpret_cast<float4*>(sp) = s;
            o[0] += q * s.x; o[1] += q * s.y; o[2] += q * s.z; o[3] += q * s.w;
          } else {
            const float s = a * (fresh ? 0.f : *sp) + b * xx[0];
            *sp = s;
            o[0] += q * s;
          }
        }
      }
#pragma unroll
      for (int j = 0; j < VEC; ++j) s_o[tid * VEC + j] = o[j];
      __syncthreads();
      for (int i = tid; i < cols * VEC; i += kSsdThreads) {
        const int v = c0 * VEC + i;
        if (v >= V) continue;
        float y = 0.f;
        for (int k = 0; k < parts; ++k) y += s_o[k * cols * VEC + i];
        stf<T>(out + v, (y + skip * ldf<T>(x + v)) * silu_acc(ldf<T>(z + v)));
      }
      __syncthreads();
    }
    fresh = false;
  }
  if (keep)
    for (int i = tid; i < K * V; i += kSsdThreads) gstate[i] = s_state[i];
}

template <typename T, int VEC>
static cudaError_t launch_ssd_recurrent(SsdParams p, cudaStream_t stream) {
  const size_t base = (2 * (size_t)((p.dim + 3) & ~3) + (size_t)kSsdThreads * VEC) * sizeof(float);
  const size_t whole = base + (size_t)p.dim * p.vdim * sizeof(float);
  constexpr size_t kLimit = 200 * 1024;
  p.in_shared = p.tok_indptr != nullptr && whole <= kLimit;
  const size_t smem = p.in_shared ? whole : base;
  if (smem > kLimit) return cudaErrorInvalidValue;
  auto kern = ssd_recurrent_kernel<T, VEC>;
  static PerDeviceOnce once;
  cudaError_t e = once.run([&] { return cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kLimit); });
  if (e != cudaSuccess) return e;
  return launch_pdl(kern, dim3(p.rows, p.heads), dim3(kSsdThreads), smem, stream, p);
}

// ------------------------------------------------------------------ chunks
constexpr int kScC = 64;  // tokens per chunk

// x = hi + lo in bf16, two neighbours at a time
__device__ __forceinline__ void ssd_split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pk2<__nv_bfloat16>(x, y);
  const float2 h = cvt2<__nv_bfloat16>(hi);
  lo = pk2<__nv_bfloat16>(x - h.x, y - h.y);
}
__device__ __forceinline__ void ssd_copy16(void* dst, const void* src, bool on) {  // zeros where off
  asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(ptx::smem_u32(dst)), "l"(src), "r"(on ? 16 : 0) : "memory");
}

template <int DK, int VB>
struct ScSmem {
  static constexpr int kQ = DK + 8;    // row pitches (bf16)
  static constexpr int kV = VB + 8;
  static constexpr int kA = kScC + 8;
  using bf = __nv_bfloat16;
  bf c[2][kScC * kQ], b[2][kScC * kQ], x[2][kScC * kV];
  bf xh[kScC * kV], xl[kScC * kV];     // x scaled for the state
  bf ah[kScC * kA], al[kScC * kA];
  bf sh[DK * kV], sl[DK * kV];
  float dt[kScC], cum[kScC + 1];       // cum[64]: of the chunk's last token
};

template <int DK, int VB>
__global__ void __launch_bounds__(kSsdThreads) ssd_chunk_kernel(const SsdParams p) {
  using bf = __nv_bfloat16;
  using SM = ScSmem<DK, VB>;
  constexpr int RB = DK / 16, CP = RB >= 8 ? 1 : 8 / RB;  // 16-row blocks of the state; warps that share one
  constexpr int NT = VB / CP / 8;                         // 8-column tiles of the state per warp
  constexpr int NO = VB / 2 / 8;                          // 8-column tiles of a chunk's output per warp
  static_assert(DK <= 128 && NT >= 2 && (NT & 1) == 0, "state of up to 128 rows");
  extern __shared__ __align__(16) uint8_t smem_raw[];
  SM& sm = *reinterpret_cast<SM*>(smem_raw);
  ptx::griddep_launch_dependents();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3, mi = lane >> 3, mr = lane & 7;
  const int v0 = blockIdx.x * VB, h = blockIdx.y, r = blockIdx.z, nv = min(VB, p.vdim - v0);
  const float rate = -expf(ldf(reinterpret_cast<const bf*>(p.A_log) + h)), bias = ldf(reinterpret_cast<const bf*>(p.dt_bias) + h),
              skip = ldf(reinterpret_cast<const bf*>(p.D) + h);
  ptx::griddep_wait();
  const int slot = p.seq_slot[r], t_beg = p.tok_indptr[r], len = p.tok_indptr[r + 1] - t_beg;
  if (slot < 0 || slot >= p.num_slots || len <= 0) {
    if (slot >= p.num_slots && tid == 0 && p.status) atomicCAS(p.status, 0, kStatusBadIndex);
    return;
  }
  const int grp = h / (p.heads / p.groups);
  const bf* X = reinterpret_cast<const bf*>(p.x) + static_cast<int64_t>(h) * p.vdim + v0;
  const bf* B = reinterpret_cast<const bf*>(p.B) + static_cast<int64_t>(grp) * p.dim;
  const bf* C = reinterpret_cast<const bf*>(p.C) + static_cast<int64_t>(grp) * p.dim;
  const bf* Z = reinterpret_cast<const bf*>(p.z) + static_cast<int64_t>(h) * p.vdim + v0;
  const bf* DT = reinterpret_cast<const bf*>(p.dt) + h;
  const int rbS = warp % RB, cS = (warp / RB) * (VB / CP), rowS = rbS * 16 + g;
  float* gstate = p.state + (static_cast<int64_t>(slot) * p.heads + h) * p.dim * p.vdim + v0;
  const bool fresh = p.pos[t_beg] == 0;
  float S[NT][4];
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int c = rowS + (e >> 1) * 8, col = cS + n * 8 + 2 * t4 + (e & 1);
      S[n][e] = (fresh || c >= p.dim || col >= nv) ? 0.f : gstate[static_cast<int64_t>(c) * p.vdim + col];
    }
  auto publish_state = [&] {
#pragma unroll
    for (int n = 0; n < NT; ++n) {
      const int at = rowS * SM::kV + cS + n * 8 + 2 * t4;
      uint32_t hi, lo;
      ssd_split2(S[n][0], S[n][1], hi, lo);
      *reinterpret_cast<uint32_t*>(sm.sh + at) = hi;
      *reinterpret_cast<uint32_t*>(sm.sl + at) = lo;
      ssd_split2(S[n][2], S[n][3], hi, lo);
      *reinterpret_cast<uint32_t*>(sm.sh + at + 8 * SM::kV) = hi;
      *reinterpret_cast<uint32_t*>(sm.sl + at + 8 * SM::kV) = lo;
    }
  };
  publish_state();
  const int nchunks = (len + kScC - 1) / kScC;
  auto fetch = [&](int ch) {  // tiles of a chunk; rows and columns behind the end arrive as zeros
    const int base = ch * kScC, n = min(kScC, len - base), buf = ch & 1;
    for (int e = tid; e < kScC * DK / 8; e += kSsdThreads) {
      const int t = e / (DK / 8), c = (e % (DK / 8)) * 8;
      const bool on = t < n && c < p.dim;
      const int64_t at = on ? (t_beg + base + t) * p.x_row + c : 0;
      ssd_copy16(sm.c[buf] + t * SM::kQ + c, C + at, on);
      ssd_copy16(sm.b[buf] + t * SM::kQ + c, B + at, on);
    }
    for (int e = tid; e < kScC * VB / 8; e += kSsdThreads) {
      const int t = e / (VB / 8), c = (e % (VB / 8)) * 8;
      const bool on = t < n && c < nv;
      ssd_copy16(sm.x[buf] + t * SM::kV + c, X + (on ? (t_beg + base + t) * p.x_row + c : 0), on);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
  };
  fetch(0);
  float raw0 = 0.f, raw1 = 0.f;  // warp 0: this lane's two tokens' dt, a chunk ahead
  auto fetch_dt = [&](int ch) {
    const int a = ch * kScC + 2 * lane;
    raw0 = a < len ? ldf(DT + (t_beg + a) * p.z_row) : 0.f;
    raw1 = a + 1 < len ? ldf(DT + (t_beg + a + 1) * p.z_row) : 0.f;
  };
  if (warp == 0) fetch_dt(0);
  const int rb = warp >> 1, cO = (warp & 1) * (VB / 2);  // this warp's part of the chunk's output

  for (int ch = 0; ch < nchunks; ++ch) {
    const int base = ch * kScC, n_tok = min(kScC, len - base), buf = ch & 1;
    const bf *sc = sm.c[buf], *sb = sm.b[buf], *sx = sm.x[buf];
    // ---- 1. steps and running sums of the log decays (no step behind the end: the sum stays)
    if (warp == 0) {
      const float d0 = 2 * lane < n_tok ? softplus_f(raw0 + bias) : 0.f, d1 = 2 * lane + 1 < n_tok ? softplus_f(raw1 + bias) : 0.f;
      const float l0 = rate * d0, l1 = rate * d1;
      float s = l0 + l1;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const float u = __shfl_up_sync(0xffffffffu, s, o);
        if (lane >= o) s += u;
      }
      sm.dt[2 * lane] = d0;
      sm.dt[2 * lane + 1] = d1;
      sm.cum[2 * lane] = s - l1;
      sm.cum[2 * lane + 1] = s;
      if (lane == 31) sm.cum[kScC] = s;
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    __syncthreads();  // (and everybody is through with the other buffer)
    if (ch + 1 < nchunks) {
      fetch(ch + 1);
      if (warp == 0) fetch_dt(ch + 1);
    }
    const float end = sm.cum[kScC];

    // ---- 2. scores within the chunk, 16 x 16 tiles on and below the diagonal, with decay and step; x scaled for the state
    for (int tile = warp; tile < 10; tile += 8) {
      const int i = tile >= 6 ? 3 : tile >= 3 ? 2 : tile >= 1 ? 1 : 0, j = tile - i * (i + 1) / 2;
      float acc[2][4] = {};
#pragma unroll
      for (int kk = 0; kk < DK / 16; ++kk) {
        uint32_t a0, a1, a2, a3, b0, b1, b2, b3;
        ldmatrix_x4(ptx::smem_u32(sc + (i * 16 + (mi & 1) * 8 + mr) * SM::kQ + kk * 16 + (mi >> 1) * 8), a0, a1, a2, a3);
        ldmatrix_x4(ptx::smem_u32(sb + (j * 16 + (mi >> 1) * 8 + mr) * SM::kQ + kk * 16 + (mi & 1) * 8), b0, b1, b2, b3);
        mma16816<bf>(acc[0], a0, a1, a2, a3, b0, b1);
        mma16816<bf>(acc[1], a0, a1, a2, a3, b2, b3);
      }
#pragma unroll
      for (int half = 0; half < 2; ++half) {
        const int t = i * 16 + g + half * 8;
        const float bt = sm.cum[t];
#pragma unroll
        for (int n = 0; n < 2; ++n) {
          const int s = j * 16 + n * 8 + 2 * t4;
          const float f0 = s <= t ? __expf(bt - sm.cum[s]) * sm.dt[s] : 0.f, f1 = s + 1 <= t ? __expf(bt - sm.cum[s + 1]) * sm.dt[s + 1] : 0.f;
          uint32_t hi, lo;
          ssd_split2(acc[n][2 * half] * f0, acc[n][2 * half + 1] * f1, hi, lo);
          *reinterpret_cast<uint32_t*>(sm.ah + t * SM::kA + s) = hi;
          *reinterpret_cast<uint32_t*>(sm.al + t * SM::kA + s) = lo;
        }
      }
    }
    for (int e = tid; e < kScC * VB / 8; e += kSsdThreads) {
      const int t = e / (VB / 8), c = (e % (VB / 8)) * 8;
      const float f = __expf(end - sm.cum[t]) * sm.dt[t];
      float v[8];
      ldf8(sx + t * SM::kV + c, v);
      uint4 hi, lo;
      ssd_split2(v[0] * f, v[1] * f, hi.x, lo.x);
      ssd_split2(v[2] * f, v[3] * f, hi.y, lo.y);
      ssd_split2(v[4] * f, v[5] * f, hi.z, lo.z);
      ssd_split2(v[6] * f, v[7] * f, hi.w, lo.w);
      *reinterpret_cast<uint4*>(sm.xh + t * SM::kV + c) = hi;
      *reinterpret_cast<uint4*>(sm.xl + t * SM::kV + c) = lo;
    }
    uint32_t gate[2][NO];  // on their way while the products run
#pragma unroll
    for (int half = 0; half < 2; ++half)
#pragma unroll
      for (int n = 0; n < NO; ++n) {
        const int t = rb * 16 + g + half * 8, col = cO + n * 8 + 2 * t4;
        gate[half][n] = 0u;
        if (t < n_tok && col < nv) gate[half][n] = *reinterpret_cast<const uint32_t*>(Z + (t_beg + base + t) * p.z_row + col);
      }
    __syncthreads();

    // ---- 3. output: state term, decayed, then the chunk's own values
    float O[NO][4] = {};
#pragma unroll
    for (int kk = 0; kk < DK / 16; ++kk) {
      uint32_t a0, a1, a2, a3;
      ldmatrix_x4(ptx::smem_u32(sc + (rb * 16 + (mi & 1) * 8 + mr) * SM::kQ + kk * 16 + (mi >> 1) * 8), a0, a1, a2, a3);
#pragma unroll
      for (int m = 0; m < NO / 2; ++m) {
        const int at = (kk * 16 + (mi & 1) * 8 + mr) * SM::kV + cO + m * 16 + (mi >> 1) * 8;
        uint32_t b0, b1, b2, b3, d0, d1, d2, d3;
        ldmatrix_x4_trans(ptx::smem_u32(sm.sh + at), b0, b1, b2, b3);
        ldmatrix_x4_trans(ptx::smem_u32(sm.sl + at), d0, d1, d2, d3);
        mma16816<bf>(O[2 * m], a0, a1, a2, a3, b0, b1);
        mma16816<bf>(O[2 * m + 1], a0, a1, a2, a3, b2, b3);
        mma16816<bf>(O[2 * m], a0, a1, a2, a3, d0, d1);
        mma16816<bf>(O[2 * m + 1], a0, a1, a2, a3, d2, d3);
      }
    }
    {
      const float e0 = __expf(sm.cum[rb * 16 + g]), e1 = __expf(sm.cum[rb * 16 + g + 8]);
#pragma unroll
      for (int n = 0; n < NO; ++n) {
        O[n][0] *= e0; O[n][1] *= e0;
        O[n][2] *= e1; O[n][3] *= e1;
      }
    }
    for (int j = 0; j <= rb; ++j) {
      uint32_t ah[4], al[4];
      const int off = (rb * 16 + (mi & 1) * 8 + mr) * SM::kA + j * 16 + (mi >> 1) * 8;
      ldmatrix_x4(ptx::smem_u32(sm.ah + off), ah[0], ah[1], ah[2], ah[3]);
      ldmatrix_x4(ptx::smem_u32(sm.al + off), al[0], al[1], al[2], al[3]);
#pragma unroll
      for (int m = 0; m < NO / 2; ++m) {
        uint32_t b0, b1, b2, b3;
        ldmatrix_x4_trans(ptx::smem_u32(sx + (j * 16 + (mi & 1) * 8 + mr) * SM::kV + cO + m * 16 + (mi >> 1) * 8), b0, b1, b2, b3);
        mma16816<bf>(O[2 * m], ah[0], ah[1], ah[2], ah[3], b0, b1);
        mma16816<bf>(O[2 * m + 1], ah[0], ah[1], ah[2], ah[3], b2, b3);
        mma16816<bf>(O[2 * m], al[0], al[1], al[2], al[3], b0, b1);
        mma16816<bf>(O[2 * m + 1], al[0], al[1], al[2], al[3], b2, b3);
      }
    }
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int t = rb * 16 + g + half * 8;
#pragma unroll
      for (int n = 0; n < NO; ++n) {
        const int col = cO + n * 8 + 2 * t4;
        if (t >= n_tok || col >= nv) continue;
        const float2 x = ldf2(sx + t * SM::kV + col), z = cvt2<bf>(gate[half][n]);
        stf2(reinterpret_cast<bf*>(p.out) + (t_beg + base + t) * p.out_stride + static_cast<int64_t>(h) * p.vdim + v0 + col,
             (O[n][2 * half] + skip * x.x) * __fdividef(z.x, 1.f + __expf(fminf(-z.x, 80.f))),
             (O[n][2 * half + 1] + skip * x.y) * __fdividef(z.y, 1.f + __expf(fminf(-z.y, 80.f))));
      }
    }
    __syncthreads();  // the state's old copy has been read

    // ---- 4. state
    {
      const float d = __expf(end);
#pragma unroll
      for (int n = 0; n < NT; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) S[n][e] *= d;
    }
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      uint32_t a0, a1, a2, a3;  // B^T: rows are state channels, columns tokens
      ldmatrix_x4_trans(ptx::smem_u32(sb + (j * 16 + (mi >> 1) * 8 + mr) * SM::kQ + rbS * 16 + (mi & 1) * 8), a0, a1, a2, a3);
#pragma unroll
      for (int m = 0; m < NT / 2; ++m) {
        const int at = (j * 16 + (mi & 1) * 8 + mr) * SM::kV + cS + m * 16 + (mi >> 1) * 8;
        uint32_t b0, b1, b2, b3, d0, d1, d2, d3;
        ldmatrix_x4_trans(ptx::smem_u32(sm.xh + at), b0, b1, b2, b3);
        ldmatrix_x4_trans(ptx::smem_u32(sm.xl + at), d0, d1, d2, d3);
        mma16816<bf>(S[2 * m], a0, a1, a2, a3, b0, b1);
        mma16816<bf>(S[2 * m + 1], a0, a1, a2, a3, b2, b3);
        mma16816<bf>(S[2 * m], a0, a1, a2, a3, d0, d1);
        mma16816<bf>(S[2 * m + 1], a0, a1, a2, a3, d2, d3);
      }
    }
    publish_state();
    // (the next chunk's first barrier comes before anybody reads the state or writes what this chunk has read)
    __syncthreads();
  }
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int c = rowS + (e >> 1) * 8, col = cS + n * 8 + 2 * t4 + (e & 1);
      if (c < p.dim && col < nv) gstate[static_cast<int64_t>(c) * p.vdim + col] = S[n][e];
    }
}

template <int DK, int VB>
static cudaError_t launch_ssd_chunk(const SsdParams& p, cudaStream_t stream) {
  auto kern = ssd_chunk_kernel<DK, VB>;
  constexpr int smem = (int)sizeof(ScSmem<DK, VB>);
  static_assert(smem <= 227 * 1024, "shared memory");
  static PerDeviceOnce once;
  cudaError_t e = once.run([&] { return cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem); });
  if (e != cudaSuccess) return e;
  return launch_pdl(kern, dim3((p.vdim + VB - 1) / VB, p.heads, p.rows), dim3(kSsdThreads), (size_t)smem, stream, p);
}

// Narrower blocks repeat the scores but give more of them: worth it while they do not fill the GPU.
template <int DK>
static cudaError_t launch_ssd_width(const SsdParams& p, cudaStream_t stream) {
  const int64_t items = (int64_t)p.heads * p.rows;
  const int sms = device_sm_count();
  if (DK < 128 || p.vdim <= 32 || items * ((p.vdim + 31) / 32) > 2 * sms) return launch_ssd_chunk<DK, 64>(p, stream);
  return launch_ssd_chunk<DK, DK < 128 ? 64 : 32>(p, stream);
}

// ------------------------------------------------------------------ norm
// A block per (part of the row, token): x <- x / rms(x) * w in place.
template <typename T, int VEC>
__global__ void __launch_bounds__(256) part_norm_kernel(T* x, int64_t row, const T* w, float eps, int part) {
  __shared__ float red[33];
  ptx::griddep_launch_dependents();
  ptx::griddep_wait();
  T* xr = x + blockIdx.y * row + static_cast<int64_t>(blockIdx.x) * part;
  const T* wr = w + static_cast<int64_t>(blockIdx.x) * part;
  constexpr int kKeep = 4;
  float keep[kKeep][VEC], ss = 0.f;
  auto load = [&](const T* q, float (&v)[VEC]) {
    if constexpr (VEC == 8) ldf8<T>(q, v);
    else v[0] = ldf<T>(q);
  };
  const int n = part / VEC;
#pragma unroll
  for (int k = 0; k < kKeep; ++k) {
    const int i = threadIdx.x + k * blockDim.x;
    if (i >= n) continue;
    load(xr + i * VEC, keep[k]);
#pragma unroll
    for (int j = 0; j < VEC; ++j) ss += keep[k][j] * keep[k][j];
  }
  for (int i = threadIdx.x + kKeep * blockDim.x; i < n; i += blockDim.x) {
    float v[VEC];
    load(xr + i * VEC, v);
#pragma unroll
    for (int j = 0; j < VEC; ++j) ss += v[j] * v[j];
  }
  const float f = rsqrtf(block_sum(ss, red) / static_cast<float>(part) + eps);
  auto put = [&](int i, float (&v)[VEC]) {
    float g[VEC];
    load(wr + i * VEC, g);
#pragma unroll
    for (int j = 0; j < VEC; ++j) v[j] *= f * g[j];
    if constexpr (VEC == 8) stf8<T>(xr + i * VEC, v);
    else stf<T>(xr + i, v[0]);
  };
#pragma unroll
  for (int k = 0; k < kKeep; ++k) {
    const int i = threadIdx.x + k * blockDim.x;
    if (i < n) put(i, keep[k]);
  }
  for (int i = threadIdx.x + kKeep * blockDim.x; i < n; i += blockDim.x) {
    float v[VEC];
    load(xr + i * VEC, v);
    put(i, v);
  }
}

// The same with a warp per part, for parts that a warp holds in registers: `kPartVecs` groups of eight per lane.
constexpr int kPartVecs = 4;
template <typename T>
__global__ void __launch_bounds__(256) part_norm_warp_kernel(T* x, int64_t row, const T* w, float eps, int parts, int part, int64_t items) {
  ptx::griddep_launch_dependents();
  ptx::griddep_wait();
  const int64_t item = static_cast<int64_t>(blockIdx.x) * 8 + (threadIdx.x >> 5);
  if (item >= items) return;
  const int lane = threadIdx.x & 31, n = part / 8, which = static_cast<int>(item % parts);
  T* xr = x + item / parts * row + static_cast<int64_t>(which) * part;
  const T* wr = w + static_cast<int64_t>(which) * part;
  float v[kPartVecs][8], ss = 0.f;
#pragma unroll
  for (int k = 0; k < kPartVecs; ++k)
    if (lane + k * 32 < n) ldf8<T>(xr + (lane + k * 32) * 8, v[k]);
#pragma unroll
  for (int k = 0; k < kPartVecs; ++k)
    if (lane + k * 32 < n)
#pragma unroll
      for (int j = 0; j < 8; ++j) ss += v[k][j] * v[k][j];
  const float f = rsqrtf(warp_sum(ss) / static_cast<float>(part) + eps);
#pragma unroll
  for (int k = 0; k < kPartVecs; ++k)
    if (lane + k * 32 < n) {
      float g[8];
      ldf8<T>(wr + (lane + k * 32) * 8, g);
#pragma unroll
      for (int j = 0; j < 8; ++j) v[k][j] *= f * g[j];
      stf8<T>(xr + (lane + k * 32) * 8, v[k]);
    }
}

}  // namespace blitz

extern "C" {
using namespace blitz;

// tok_indptr null: one token per row (decode).  dtype 0 fp16, 1 bf16, 2 fp32.
int blitz_ssd_recurrent(const void* x, const void* B, const void* C, int64_t x_row, const void* z, const void* dt, int64_t z_row,
                        const void* dt_bias, const void* A_log, const void* D, float* state, void* out, int64_t out_stride,
                        const int32_t* pos, const int32_t* tok_indptr, const int32_t* seq_slot, int rows, int heads, int groups, int dim,
                        int vdim, int num_slots, int* status, int dtype, cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (dim <= 0 || vdim <= 0 || heads <= 0 || heads > 65535 || groups <= 0 || heads % groups) return -1;
  SsdParams p{x, B, C, x_row, z, dt, z_row, dt_bias, A_log, D, state, out, out_stride, pos, tok_indptr, seq_slot,
              rows, heads, groups, dim, vdim, num_slots, 0, status};
  const int es = dtype == 2 ? 4 : 2;
  const bool vec = (vdim & 3) == 0 && (x_row & 3) == 0 && (reinterpret_cast<uintptr_t>(x) % (4 * es)) == 0;
  cudaError_t e = cudaSuccess;
  if (vec) {
    BLITZ_DISPATCH_DTYPE3(dtype, (e = launch_ssd_recurrent<T, 4>(p, stream)));
  } else {
    BLITZ_DISPATCH_DTYPE3(dtype, (e = launch_ssd_recurrent<T, 1>(p, stream)));
  }
  return (int)e;
}

// Whether the chunked kernel takes these sizes (bf16 only; vectors of 8 elements).
int blitz_ssd_chunk_supported(int dim, int vdim) {
  return dim > 0 && dim <= 128 && (dim & 7) == 0 && vdim > 0 && (vdim & 7) == 0;
}

// As blitz_ssd_recurrent for rows of any length in bf16.  Row pitches and the bases of x, B, C: multiples of 8 elements.
int blitz_ssd_chunk(const void* x, const void* B, const void* C, int64_t x_row, const void* z, const void* dt, int64_t z_row,
                    const void* dt_bias, const void* A_log, const void* D, float* state, void* out, int64_t out_stride,
                    const int32_t* pos, const int32_t* tok_indptr, const int32_t* seq_slot, int rows, int heads, int groups, int dim,
                    int vdim, int num_slots, int* status, cudaStream_t stream) {
  if (rows <= 0) return 0;
  if (!blitz_ssd_chunk_supported(dim, vdim) || heads <= 0 || heads > 65535 || rows > 65535 || groups <= 0 || heads % groups) return -1;
  if ((x_row & 7) || (z_row & 1) || (out_stride & 1) || tok_indptr == nullptr) return -1;
  for (const void* q : {x, B, C})
    if (reinterpret_cast<uintptr_t>(q) & 15) return -1;
  if ((reinterpret_cast<uintptr_t>(z) | reinterpret_cast<uintptr_t>(out)) & 3) return -1;
  SsdParams p{x, B, C, x_row, z, dt, z_row, dt_bias, A_log, D, state, out, out_stride, pos, tok_indptr, seq_slot,
              rows, heads, groups, dim, vdim, num_slots, 0, status};
  return (int)(dim <= 32 ? launch_ssd_width<32>(p, stream) : dim <= 64 ? launch_ssd_width<64>(p, stream) : launch_ssd_width<128>(p, stream));
}

// RMS norm of a row in `parts` equal parts, each by its own root mean square, in place; w [parts * part].
int blitz_part_norm(void* x, int64_t row, const void* w, float eps, int tokens, int parts, int part, int dtype, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  if (parts <= 0 || part <= 0 || tokens > 65535) return -1;
  const uintptr_t al = dtype == 2 ? 32 : 16;
  const bool wide = ((part | row) & 7) == 0 && reinterpret_cast<uintptr_t>(x) % al == 0 && reinterpret_cast<uintptr_t>(w) % al == 0;
  const int n = part / (wide ? 8 : 1);
  const dim3 grid(parts, tokens), block(n <= 64 ? 64 : n <= 256 ? 128 : 256);
  auto go = [&](auto type) {
    using T = decltype(type);
    const int64_t items = (int64_t)tokens * parts;
    if (wide && part <= 256 * kPartVecs && items / 8 >= device_sm_count())
      return launch_pdl(part_norm_warp_kernel<T>, dim3((unsigned)((items + 7) / 8)), dim3(256), 0, stream, (T*)x, row, (const T*)w, eps, parts, part, items);
    return wide ? launch_pdl(part_norm_kernel<T, 8>, grid, block, 0, stream, (T*)x, row, (const T*)w, eps, part)
                : launch_pdl(part_norm_kernel<T, 1>, grid, block, 0, stream, (T*)x, row, (const T*)w, eps, part);
  };
  cudaError_t e = cudaSuccess;
  BLITZ_DISPATCH_DTYPE3(dtype, (e = go(T{})));
  return (int)e;
}

}  // extern "C"
