// Gated linear attention of prompts, in chunks on the tensor cores (bf16 activations, fp32 state; gla.cu has the
// recurrence itself and serves single tokens and everything this kernel does not take).
//
// With b_t the running sum of the log decays within a chunk of 64 tokens (per key channel, b <= 0 and falling):
//
//   o_t   = (q_t e^(b_t))^T S_0 + sum_{s <= t} (sum_c q_tc k_sc e^(b_tc - b_sc)) v_s
//   S_end = diag(e^(b_end)) S_0 + sum_s (k_s e^(b_end - b_s)) v_s^T
//
// (the chunkwise form of Yang, Wang, Shen, Panda and Kim, "Gated Linear Attention Transformers with Hardware-Efficient
// Training").  e^(b_t - b_s) must be split between q and k to become a matrix product, and e^(-b_s) alone overflows for
// fast decays, so the chunk is cut into four blocks of 16 tokens with r_i = b at the end of block i - 1 (r_0 = 0):
//
//   q'_t = q_t e^(b_t - r_i),  t in block i          <= |q|
//   k~_s = k_s e^(r_(j+1) - b_s),  s in block j      <= |k|
//
// and every product takes the factor between two block borders from a table: block (i, j < i) scales k~ by
// e^(r_i - r_(j+1)) <= 1, the state term scales q' by e^(r_i), the state update scales k~ by e^(b_end - r_(j+1)).  Only
// within one block is the factor e^(r_i - r_(i+1)) >= 1; when a channel decays by more than e^-80 within 16 tokens, which
// that form cannot hold, the block's 136 scores are computed one by one from the unscaled inputs, a warp per row.
//
// 32-bit arithmetic where the design asks for it: decays, their sums and exponentials and the state are fp32, and the
// products that involve them split their fp32 operands into two bf16 numbers (x = hi + lo, relative error 2^-17) and
// drop only the lo * lo term.
//
// Second form (WKV, see gla.cu): o_t sees the decays up to the token before it, so q takes b_(t-1) where the first form takes b_t,
// the scores are those of s < t, and the token's own score is sum_c q_tc u_c k_tc without any decay.
//
// A block of 16 warps owns (row, head, 64 or 128 value columns) and walks the row's chunks with the state in registers; everything
// a chunk reads from global memory is requested one chunk (the gates: half a chunk) ahead.  The blocks of one head form a thread-block cluster, which exchanges the 64 partial sums of squares per chunk through
// distributed shared memory, so that the output norm and the gate are applied here and nothing but the result is
// written.  (gla_decay_kernel computes b beforehand: every value block of a head needs it.)
#include "launch.cuh"
#include "mma.cuh"
#include "ptx.cuh"
#include "scalar.cuh"
#include "tmap.cuh"

namespace blitz {

constexpr int kGcC = 64;        // tokens per chunk
constexpr int kGcB = 16;        // tokens per block
constexpr int kGcV = 64;        // value columns per CTA: this many, or twice as many when that still fills the GPU
constexpr int kGcThreads = 512;
constexpr int kGcMaxCluster = 8;
constexpr float kGcMaxDecay = 80.f;

struct GlaChunkParams {
  const __nv_bfloat16 *q, *k, *v, *g, *low;
  int64_t row;
  const float* low32;    // WKV: [tokens][low_row], instead of low
  int64_t low_row;
  const __nv_bfloat16 *a2, *a2_b, *norm, *bonus;  // norm: head h's from h * norm_step on; bonus [heads * dim]: WKV
  int norm_step;
  float* cum;      // [tokens][heads * dim]: running sums of the log decays within each chunk
  float* state;    // [slots][heads][dim][vdim]
  __nv_bfloat16* out;
  int64_t out_stride;
  const int32_t *pos, *tok_indptr, *seq_slot;
  int heads, dim, vdim, rank, num_slots;
  float q_scale, inv_tau, eps;
  int* status;
};

// log(sigmoid(z)) = min(z, 0) - log(1 + e^-|z|) on the special-function unit; the series keeps the digits of a slow decay
__device__ __forceinline__ float log_sigmoid_ex2(float z) {
  const float e = __expf(-fabsf(z));
  const float l = e < 0.03f ? e * (1.f - e * (0.5f - e * (0.33333333f - e * 0.25f))) : __logf(1.f + e);
  return fminf(z, 0.f) - l;
}

// Running sum of log(sigmoid(low a2 + b)) / tau (WKV: -exp(tanh(low) a2 + b)) over a chunk; a thread per channel.
constexpr int kGdThreads = 128, kGdPitch = kGcC + 4, kGdMaxRank = 128;
template <bool WKV>
__global__ void __launch_bounds__(kGdThreads) gla_decay_kernel(const GlaChunkParams p) {
  ptx::griddep_launch_dependents();
  ptx::griddep_wait();
  extern __shared__ __align__(16) float s_low[];  // [rank][kGdPitch] by token, and behind it the channels' coefficients [rank][kGdThreads]
  float* s_w = s_low + p.rank * kGdPitch;
  const int r = blockIdx.z, hk = p.heads * p.dim;
  const int t0 = p.tok_indptr[r] + blockIdx.y * kGcC, n = min(kGcC, p.tok_indptr[r + 1] - t0);
  if (n <= 0) return;
  const int c = blockIdx.x * kGdThreads + threadIdx.x;
  for (int i = 0; i < p.rank; ++i) s_w[i * kGdThreads + threadIdx.x] = c < hk ? ldf(p.a2 + static_cast<int64_t>(i) * hk + c) : 0.f;
  for (int i = threadIdx.x; i < n * p.rank; i += kGdThreads)
    s_low[i % p.rank * kGdPitch + i / p.rank] = WKV ? tanhf(p.low32[static_cast<int64_t>(t0 + i / p.rank) * p.low_row + i % p.rank])
                   : ldf(p.low + static_cast<int64_t>(t0 + i / p.rank) * p.row + i % p.rank);
  __syncthreads();
  if (c >= hk) return;
  const float bias = ldf(p.a2_b + c);
  float sum = 0.f;
  constexpr int kAtOnce = 16;  // tokens whose sums a thread forms together
  for (int first = 0; first < n; first += kAtOnce) {
    float zs[kAtOnce];
#pragma unroll
    for (int k = 0; k < kAtOnce; ++k) zs[k] = bias;
    for (int i = 0; i < p.rank; ++i) {
      const float w = s_w[i * kGdThreads + threadIdx.x];
#pragma unroll
      for (int k = 0; k < kAtOnce; k += 4) {  // (what lies behind the last token is not used)
        const float4 a = *reinterpret_cast<const float4*>(s_low + i * kGdPitch + first + k);
        zs[k] = fmaf(a.x, w, zs[k]);
        zs[k + 1] = fmaf(a.y, w, zs[k + 1]);
        zs[k + 2] = fmaf(a.z, w, zs[k + 2]);
        zs[k + 3] = fmaf(a.w, w, zs[k + 3]);
      }
    }
#pragma unroll
    for (int k = 0; k < kAtOnce; ++k) {
      const int t = first + k;
      if (t >= n) break;
      const float z = zs[k];
      // (e^-104 is zero in fp32; larger steps would only cost the sum its digits)
      sum += WKV ? -fminf(__expf(z), 104.f) : log_sigmoid_ex2(z) * p.inv_tau;
      p.cum[static_cast<int64_t>(t0 + t) * hk + c] = sum;
    }
  }
}

__device__ __forceinline__ float silu_ex2(float z) { return __fdividef(z, 1.f + __expf(-z)); }

// x = hi + lo in bf16, two neighbours at a time
__device__ __forceinline__ void split2(float x, float y, uint32_t& hi, uint32_t& lo) {
  hi = pk2<__nv_bfloat16>(x, y);
  const float2 h = cvt2<__nv_bfloat16>(hi);
  lo = pk2<__nv_bfloat16>(x - h.x, y - h.y);
}

template <int DK, int VB>
struct GcSmem {
  static constexpr int kQ = DK + 8;       // row pitch of q' (bf16)
  static constexpr int kK = DK + 8;       // row pitch of k~ (fp32)
  static constexpr int kV = VB + 8;       // row pitch of v and S (bf16)
  static constexpr int kA = kGcC + 8;     // row pitch of A (bf16)
  static constexpr int kParts = kGcMaxCluster;
  float k[kGcC * kK];
  float ref[2][5 * DK];                   // r_0 .. r_4 (r_4 = b_end), by parity of the chunk
  float fs[10 * DK];                      // e^(r_i - r_(j+1)) of the ten score tiles
  float fe[5 * DK];                       // e^(b_end - r_(j+1)), j = 0 .. 3, and e^(b_end)
  float ss[2][kParts][kGcC];              // partial sums of squares of every cluster rank, by parity of the chunk
  float part[4][kGcC];
  float norm[VB];
  float own[kGcC];                        // WKV: scores of the tokens with themselves
  int wide[4];                            // block whose decay the factored form cannot hold
  __nv_bfloat16 qh[kGcC * kQ], ql[kGcC * kQ];  // q'
  __nv_bfloat16 ih[kGcC * kQ], il[kGcC * kQ];  // q e^b
  __nv_bfloat16 v[kGcC * kV];
  __nv_bfloat16 ah[kGcC * kA], al[kGcC * kA];
  __nv_bfloat16 sh[DK * kV], sl[DK * kV];
};

// N neighbouring elements (the address is a multiple of N elements).
template <int N, typename T>
__device__ __forceinline__ void ldn(const T* p, float (&v)[N]) {
  if constexpr (N == 4) {
    const float4 f = ldf4(p);
    v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w;
  } else if constexpr (N == 2) {
    const float2 f = ldf2(p);
    v[0] = f.x; v[1] = f.y;
  } else {
    v[0] = ldf(p);
  }
}

// Tiles 0 .. 5: (1,0) (2,0) (2,1) (3,0) (3,1) (3,2); 6 .. 9: the diagonal.
__device__ __forceinline__ void gc_tile(int tile, int& i, int& j) {
  i = tile >= 6 ? tile - 6 : (tile >= 3 ? 3 : tile >= 1 ? 2 : 1);
  j = tile >= 6 ? i : (tile >= 3 ? tile - 3 : tile >= 1 ? tile - 1 : 0);
}

template <int DK, int VB, bool WKV>
__global__ void __launch_bounds__(kGcThreads, 1) gla_chunk_kernel(const GlaChunkParams p) {
  using bf = __nv_bfloat16;
  using SM = GcSmem<DK, VB>;
  constexpr int RB = DK / 16;             // 16-row blocks of the state
  constexpr int CP = RB >= 4 ? 16 / RB : 4;  // warps that share a row block of it (DK = 32: half the warps have no part)
  constexpr int NT = VB / CP / 8;       // 8-column tiles of the state per warp
  constexpr int NO = VB / 32;             // 8-column tiles of a chunk's output per warp
  constexpr int kVecs = kGcC * DK / 8;    // vectors of 8 q (k, b) elements of a chunk
  constexpr int NV = (kVecs + kGcThreads - 1) / kGcThreads;
  static_assert(RB * CP <= 16 && (NT & 1) == 0, "DK is 32, 64 or 128");
  extern __shared__ __align__(16) uint8_t smem_raw[];
  SM& sm = *reinterpret_cast<SM*>(smem_raw);
  ptx::griddep_launch_dependents();
  ptx::griddep_wait();
  const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
  const int mi = lane >> 3, mr = lane & 7;
  const int h = blockIdx.y, r = blockIdx.z, nrank = gridDim.x, rank = blockIdx.x;
  const int v0 = blockIdx.x * VB, nv = min(VB, p.vdim - v0);
  const int slot = p.seq_slot[r];
  const int t_beg = p.tok_indptr[r], len = p.tok_indptr[r + 1] - t_beg;
  const int hk = p.heads * p.dim;
  // the CTAs of a cluster have the same row: they take the same way out
  if (slot < 0 || slot >= p.num_slots || len <= 0) {
    if (slot >= p.num_slots && tid == 0 && p.status) atomicCAS(p.status, 0, kStatusBadIndex);
    return;
  }
  ptx::cluster_arrive_release();  // every CTA of the cluster runs: its shared memory may be written
  ptx::cluster_wait_acquire();
  const bool has_state = warp < RB * CP;
  const int rbS = warp % RB, cS = has_state ? (warp / RB) * (VB / CP) : 0;  // this warp's part of the state
  const int rowS = rbS * 16 + g;
  float* gstate = p.state + (static_cast<int64_t>(slot) * p.heads + h) * p.dim * p.vdim + v0;
  float S[NT][4];
  const bool fresh = p.pos[t_beg] == 0;
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int c = rowS + (e >> 1) * 8, col = cS + n * 8 + 2 * t4 + (e & 1);
      S[n][e] = (fresh || !has_state || c >= p.dim || col >= nv) ? 0.f : gstate[static_cast<int64_t>(c) * p.vdim + col];
    }
  auto publish_state = [&] {
    if (!has_state) return;
#pragma unroll
    for (int n = 0; n < NT; ++n) {
      const int at = rowS * SM::kV + cS + n * 8 + 2 * t4;
      uint32_t hi, lo;
      split2(S[n][0], S[n][1], hi, lo);
      *reinterpret_cast<uint32_t*>(sm.sh + at) = hi;
      *reinterpret_cast<uint32_t*>(sm.sl + at) = lo;
      split2(S[n][2], S[n][3], hi, lo);
      *reinterpret_cast<uint32_t*>(sm.sh + at + 8 * SM::kV) = hi;
      *reinterpret_cast<uint32_t*>(sm.sl + at + 8 * SM::kV) = lo;
    }
  };
  publish_state();
  const int rb = warp >> 2, cO = (warp & 3) * (VB / 4);  // this warp's part of the chunk's output
  const int nchunks = (len + kGcC - 1) / kGcC;

  // what a chunk reads, requested one chunk ahead: q, k and b by vectors, v, and the table of block borders (with wide
  // blocks the registers do not hold b as well: it is read, from L2, when the chunk starts)
  constexpr bool kAheadB = VB == kGcV;
  uint4 rq[NV], rk[NV], rv[VB / 64];
  float rb8[NV][8], rbq[WKV ? NV : 1][8], rref[2];  // rbq: b of the token before (what q takes)
  auto request_b = [&](int chunk) {
    const int base = chunk * kGcC, last = min(kGcC, len - base) - 1;
    const float* cum = p.cum + static_cast<int64_t>(t_beg + base) * hk + h * p.dim;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int e = tid + i * kGcThreads, t = e / (DK / 8), c = (e % (DK / 8)) * 8;
#pragma unroll
      for (int j = 0; j < 8; ++j) rb8[i][j] = 0.f;
      if (e < kVecs && c < p.dim) ldf8(cum + static_cast<int64_t>(min(t, last)) * hk + c, rb8[i]);  // no decay past the end
      if (WKV) {
#pragma unroll
        for (int j = 0; j < 8; ++j) rbq[WKV ? i : 0][j] = 0.f;
        if (e < kVecs && c < p.dim && t > 0) ldf8(cum + static_cast<int64_t>(min(t - 1, last)) * hk + c, rbq[WKV ? i : 0]);
      }
    }
  };
  auto request = [&](int chunk) {
    const int base = chunk * kGcC, last = min(kGcC, len - base) - 1;
    const float* cum = p.cum + static_cast<int64_t>(t_beg + base) * hk + h * p.dim;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int e = tid + i * kGcThreads, t = e / (DK / 8), c = (e % (DK / 8)) * 8;
      rq[i] = rk[i] = make_uint4(0, 0, 0, 0);
      if (e < kVecs && c < p.dim && t <= last) {
        const int64_t at = static_cast<int64_t>(t_beg + base + t) * p.row + h * p.dim + c;
        rq[i] = *reinterpret_cast<const uint4*>(p.q + at);
        rk[i] = *reinterpret_cast<const uint4*>(p.k + at);
      }
    }
    if (kAheadB) request_b(chunk);
#pragma unroll
    for (int i = 0; i < VB / 64; ++i) {
      const int t = tid / 8, c = (tid % 8) * 8 + i * 64;
      rv[i] = make_uint4(0, 0, 0, 0);
      if (t <= last && c < nv)
        rv[i] = *reinterpret_cast<const uint4*>(p.v + static_cast<int64_t>(t_beg + base + t) * p.row + h * p.vdim + v0 + c);
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
      const int e = tid + i * kGcThreads, blk = e / DK, c = e % DK;
      rref[i] = (e < 5 * DK && blk > 0 && c < p.dim) ? cum[static_cast<int64_t>(min(blk * kGcB - 1, last)) * hk + c] : 0.f;
    }
  };
  auto keep_borders = [&](int chunk) {
#pragma unroll
    for (int i = 0; i < 2; ++i)
      if (tid + i * kGcThreads < 5 * DK) sm.ref[chunk & 1][tid + i * kGcThreads] = rref[i];
  };
  request(0);
  keep_borders(0);
  if (tid < 4) sm.wide[tid] = 0;
  if (tid < nv) sm.norm[tid] = ldf(p.norm + static_cast<int64_t>(h) * p.norm_step + v0 + tid);
  __syncthreads();

  for (int ch = 0; ch < nchunks; ++ch) {
    const int base = ch * kGcC, n_tok = min(kGcC, len - base);
    const float* ref = sm.ref[ch & 1];
    if (!kAheadB) request_b(ch);
    // ---- 1. q', q e^b, k~, v and the factor tables into shared memory
#pragma unroll
    for (int i = 0; i < NV; ++i) {
      const int e = tid + i * kGcThreads, t = e / (DK / 8), c = (e % (DK / 8)) * 8, blk = t / kGcB;
      if (e < kVecs) {
        float q8[8], k8[8], i8[8], lo8[8], hi8[8];
        unpack8<bf>(rq[i], q8);
        unpack8<bf>(rk[i], k8);
        ldf8(ref + blk * DK + c, lo8);
        ldf8(ref + (blk + 1) * DK + c, hi8);
        if (WKV) {  // the lanes of a token are neighbours
          float u8[8] = {}, own = 0.f;
          if (c < p.dim) ldf8(p.bonus + h * p.dim + c, u8);
#pragma unroll
          for (int j = 0; j < 8; ++j) own += q8[j] * u8[j] * k8[j];
#pragma unroll
          for (int o = 1; o < DK / 8; o <<= 1) own += __shfl_xor_sync(0xffffffffu, own, o);
          if (c == 0) sm.own[t] = own;
        }
        const float(&b8)[8] = WKV ? rbq[WKV ? i : 0] : rb8[i];
#pragma unroll
        for (int j = 0; j < 8; ++j) {
          q8[j] *= p.q_scale;
          i8[j] = q8[j] * __expf(b8[j]);
          q8[j] *= __expf(b8[j] - lo8[j]);
          k8[j] *= __expf(hi8[j] - rb8[i][j]);
        }
        auto put = [&](const float (&x)[8], bf* dh, bf* dl) {
          uint4 hi, lo;
          split2(x[0], x[1], hi.x, lo.x);
          split2(x[2], x[3], hi.y, lo.y);
          split2(x[4], x[5], hi.z, lo.z);
          split2(x[6], x[7], hi.w, lo.w);
          *reinterpret_cast<uint4*>(dh + t * SM::kQ + c) = hi;
          *reinterpret_cast<uint4*>(dl + t * SM::kQ + c) = lo;
        };
        put(q8, sm.qh, sm.ql);
        put(i8, sm.ih, sm.il);
        stf8(sm.k + t * SM::kK + c, k8);
      }
    }
#pragma unroll
    for (int i = 0; i < VB / 64; ++i) *reinterpret_cast<uint4*>(sm.v + (tid / 8) * SM::kV + (tid % 8) * 8 + i * 64) = rv[i];
    for (int e = tid; e < 10 * DK; e += kGcThreads) {
      int i, j;
      gc_tile(e / DK, i, j);
      const float d = ref[i * DK + e % DK] - ref[(j + 1) * DK + e % DK];
      if (i == j && d > kGcMaxDecay) sm.wide[i] = 1;
      sm.fs[e] = __expf(d);
    }
    for (int e = tid; e < 5 * DK; e += kGcThreads)
      sm.fe[e] = __expf(ref[4 * DK + e % DK] - (e < 4 * DK ? ref[e + DK] : 0.f));
    __syncthreads();
    if (ch + 1 < nchunks) request(ch + 1);

    // ---- 2. scores within the chunk: ten 16 x 16 tiles on and below the diagonal
    if (warp < 10) {
      int i, j;
      gc_tile(warp, i, j);
      float acc[2][4];
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[n][e] = 0.f;
      if (!(i == j && sm.wide[i])) {
        const float* fs = sm.fs + warp * DK + 2 * t4;
#pragma unroll
        for (int kk = 0; kk < DK / 16; ++kk) {
          const uint32_t off = static_cast<uint32_t>((i * kGcB + (mi & 1) * 8 + mr) * SM::kQ + kk * 16 + (mi >> 1) * 8);
          uint32_t ah[4], al[4];
          ldmatrix_x4(ptx::smem_u32(sm.qh + off), ah[0], ah[1], ah[2], ah[3]);
          ldmatrix_x4(ptx::smem_u32(sm.ql + off), al[0], al[1], al[2], al[3]);
          // factors of channels 2 t4, + 1 and + 8, + 9
          const float2 f0 = *reinterpret_cast<const float2*>(fs + kk * 16), f1 = *reinterpret_cast<const float2*>(fs + kk * 16 + 8);
#pragma unroll
          for (int n = 0; n < 2; ++n) {
            const float* kr = sm.k + (j * kGcB + n * 8 + g) * SM::kK + kk * 16 + 2 * t4;
            const float2 x = *reinterpret_cast<const float2*>(kr), y = *reinterpret_cast<const float2*>(kr + 8);
            uint32_t bh0, bl0, bh1, bl1;
            split2(x.x * f0.x, x.y * f0.y, bh0, bl0);
            split2(y.x * f1.x, y.y * f1.y, bh1, bl1);
            mma16816<bf>(acc[n], ah[0], ah[1], ah[2], ah[3], bh0, bh1);
            mma16816<bf>(acc[n], ah[0], ah[1], ah[2], ah[3], bl0, bl1);
            mma16816<bf>(acc[n], al[0], al[1], al[2], al[3], bh0, bh1);
          }
        }
      }
#pragma unroll
      for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
          const int t = g + half * 8, s = n * 8 + 2 * t4;
          if (i == j && sm.wide[i]) continue;
          float x = acc[n][2 * half], y = acc[n][2 * half + 1];
          if (i == j) {  // above the diagonal (a factored score may be anything there)
            if (s > t) x = 0.f;
            if (s + 1 > t) y = 0.f;
            if (WKV && s == t) x = sm.own[i * kGcB + t];
            if (WKV && s + 1 == t) y = sm.own[i * kGcB + t];
          }
          uint32_t hi, lo;
          split2(x, y, hi, lo);
          const int at = (i * kGcB + t) * SM::kA + j * kGcB + s;
          *reinterpret_cast<uint32_t*>(sm.ah + at) = hi;
          *reinterpret_cast<uint32_t*>(sm.al + at) = lo;
        }
    }
    // blocks that the factored form cannot hold: a warp per row, the scores one by one from the unscaled inputs
    for (int i = 0; i < 4; ++i) {
      if (!sm.wide[i]) continue;
      constexpr int CH = DK / 32;  // channels of a lane
      const int t = warp, c = lane * CH;
      const bool on = i * kGcB + t < n_tok && c < p.dim;
      const int64_t tok = t_beg + base + i * kGcB;
      float q[CH], bt[CH], x[kGcB];
#pragma unroll
      for (int e = 0; e < CH; ++e) q[e] = bt[e] = 0.f;
      if (on) {
        ldn<CH>(p.q + (tok + t) * p.row + h * p.dim + c, q);
        if (!WKV || i * kGcB + t > 0) ldn<CH>(p.cum + (tok + t - (WKV ? 1 : 0)) * hk + h * p.dim + c, bt);
      }
#pragma unroll
      for (int s = 0; s < kGcB; ++s) {
        x[s] = 0.f;
        if (on && (WKV ? s < t : s <= t)) {
          float k[CH], bs[CH];
          ldn<CH>(p.k + (tok + s) * p.row + h * p.dim + c, k);
          ldn<CH>(p.cum + (tok + s) * hk + h * p.dim + c, bs);
#pragma unroll
          for (int e = 0; e < CH; ++e) x[s] += q[e] * k[e] * __expf(bt[e] - bs[e]);
          x[s] *= p.q_scale;
        }
      }
      // lane s receives the sum of x[s] over the lanes (both halves of the warp the same)
#pragma unroll
      for (int o = 8; o > 0; o >>= 1) {
        const bool up = lane & o;
#pragma unroll
        for (int s = 0; s < o; ++s) {
          const float give = up ? x[s] : x[s + o], keep = up ? x[s + o] : x[s];
          x[s] = keep + __shfl_xor_sync(0xffffffffu, give, o);
        }
      }
      x[0] += __shfl_xor_sync(0xffffffffu, x[0], 16);
      if (lane < kGcB) {
        const float y = WKV && lane == t ? sm.own[i * kGcB + t] : x[0];
        const bf hi = __float2bfloat16_rn(y);
        const int at = (i * kGcB + t) * SM::kA + i * kGcB + lane;
        sm.ah[at] = hi;
        sm.al[at] = __float2bfloat16_rn(y - __bfloat162float(hi));
      }
    }
    __syncthreads();

    // ---- 3. output: state term, then the chunk's own values
    float O[NO][4];
#pragma unroll
    for (int n = 0; n < NO; ++n)
#pragma unroll
      for (int e = 0; e < 4; ++e) O[n][e] = 0.f;
    uint32_t gate[2][NO];  // [half][n], two values each, on their way while the products run
#pragma unroll
    for (int half = 0; half < 2; ++half)
#pragma unroll
      for (int n = 0; n < NO; ++n) {
        const int t = rb * 16 + g + half * 8, col = cO + n * 8 + 2 * t4;
        gate[half][n] = 0u;
        if (t < n_tok && col < nv)
          gate[half][n] = *reinterpret_cast<const uint32_t*>(p.g + static_cast<int64_t>(t_beg + base + t) * p.row + h * p.vdim + v0 + col);
      }
#pragma unroll
    for (int kk = 0; kk < DK / 16; ++kk) {
      const uint32_t off = static_cast<uint32_t>((rb * kGcB + (mi & 1) * 8 + mr) * SM::kQ + kk * 16 + (mi >> 1) * 8);
      uint32_t ah[4], al[4];
      ldmatrix_x4(ptx::smem_u32(sm.ih + off), ah[0], ah[1], ah[2], ah[3]);
      ldmatrix_x4(ptx::smem_u32(sm.il + off), al[0], al[1], al[2], al[3]);
#pragma unroll
      for (int m = 0; m < NO / 2; ++m) {
        const uint32_t at = static_cast<uint32_t>((kk * 16 + (mi & 1) * 8 + mr) * SM::kV + cO + m * 16 + (mi >> 1) * 8);
        uint32_t b0, b1, b2, b3, d0, d1, d2, d3;
        ldmatrix_x4_trans(ptx::smem_u32(sm.sh + at), b0, b1, b2, b3);
        ldmatrix_x4_trans(ptx::smem_u32(sm.sl + at), d0, d1, d2, d3);
        mma16816<bf>(O[2 * m], ah[0], ah[1], ah[2], ah[3], b0, b1);
        mma16816<bf>(O[2 * m + 1], ah[0], ah[1], ah[2], ah[3], b2, b3);
        mma16816<bf>(O[2 * m], ah[0], ah[1], ah[2], ah[3], d0, d1);
        mma16816<bf>(O[2 * m + 1], ah[0], ah[1], ah[2], ah[3], d2, d3);
        mma16816<bf>(O[2 * m], al[0], al[1], al[2], al[3], b0, b1);
        mma16816<bf>(O[2 * m + 1], al[0], al[1], al[2], al[3], b2, b3);
      }
    }
    for (int j = 0; j <= rb; ++j) {
      const uint32_t off = static_cast<uint32_t>((rb * kGcB + (mi & 1) * 8 + mr) * SM::kA + j * kGcB + (mi >> 1) * 8);
      uint32_t ah[4], al[4];
      ldmatrix_x4(ptx::smem_u32(sm.ah + off), ah[0], ah[1], ah[2], ah[3]);
      ldmatrix_x4(ptx::smem_u32(sm.al + off), al[0], al[1], al[2], al[3]);
#pragma unroll
      for (int m = 0; m < NO / 2; ++m) {
        const uint32_t at = static_cast<uint32_t>((j * kGcB + (mi & 1) * 8 + mr) * SM::kV + cO + m * 16 + (mi >> 1) * 8);
        uint32_t b0, b1, b2, b3;
        ldmatrix_x4_trans(ptx::smem_u32(sm.v + at), b0, b1, b2, b3);
        mma16816<bf>(O[2 * m], ah[0], ah[1], ah[2], ah[3], b0, b1);
        mma16816<bf>(O[2 * m + 1], ah[0], ah[1], ah[2], ah[3], b2, b3);
        mma16816<bf>(O[2 * m], al[0], al[1], al[2], al[3], b0, b1);
        mma16816<bf>(O[2 * m + 1], al[0], al[1], al[2], al[3], b2, b3);
      }
    }
    {
      float s0 = 0.f, s1 = 0.f;
#pragma unroll
      for (int n = 0; n < NO; ++n) {
        s0 += O[n][0] * O[n][0] + O[n][1] * O[n][1];
        s1 += O[n][2] * O[n][2] + O[n][3] * O[n][3];
      }
#pragma unroll
      for (int o = 1; o <= 2; o <<= 1) {
        s0 += __shfl_xor_sync(0xffffffffu, s0, o);
        s1 += __shfl_xor_sync(0xffffffffu, s1, o);
      }
      if (t4 == 0) {
        sm.part[warp & 3][rb * 16 + g] = s0;
        sm.part[warp & 3][rb * 16 + g + 8] = s1;
      }
    }
    if (ch + 1 < nchunks) keep_borders(ch + 1);
    __syncthreads();
    // sums of squares of this CTA's columns to every CTA of the head (two sets by parity: a CTA is at most one chunk ahead)
    if (tid < kGcC) {
      const float s = (sm.part[0][tid] + sm.part[1][tid]) + (sm.part[2][tid] + sm.part[3][tid]);
      const uint32_t mine = ptx::smem_u32(&sm.ss[ch & 1][rank][tid]);
      for (int d = 0; d < nrank; ++d) ptx::st_shared_cluster_f32(ptx::mapa_shared(mine, d), s);
    }
    ptx::cluster_arrive_release();

    // ---- 4. state update (meanwhile the sums travel)
    if (tid < 4) sm.wide[tid] = 0;
    if (has_state) {
      const float* fe = sm.fe + rowS;
      const float d0 = fe[4 * DK], d1 = fe[4 * DK + 8];
#pragma unroll
      for (int n = 0; n < NT; ++n) {
        S[n][0] *= d0; S[n][1] *= d0;
        S[n][2] *= d1; S[n][3] *= d1;
      }
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float f0 = fe[j * DK], f1 = fe[j * DK + 8];
        const float* kc = sm.k + (j * kGcB + 2 * t4) * SM::kK + rowS;
        uint32_t ah[4], al[4];
        split2(kc[0] * f0, kc[SM::kK] * f0, ah[0], al[0]);
        split2(kc[8] * f1, kc[SM::kK + 8] * f1, ah[1], al[1]);
        split2(kc[8 * SM::kK] * f0, kc[9 * SM::kK] * f0, ah[2], al[2]);
        split2(kc[8 * SM::kK + 8] * f1, kc[9 * SM::kK + 8] * f1, ah[3], al[3]);
#pragma unroll
        for (int m = 0; m < NT / 2; ++m) {
          const uint32_t at = static_cast<uint32_t>((j * kGcB + (mi & 1) * 8 + mr) * SM::kV + cS + m * 16 + (mi >> 1) * 8);
          uint32_t b0, b1, b2, b3;
          ldmatrix_x4_trans(ptx::smem_u32(sm.v + at), b0, b1, b2, b3);
          mma16816<bf>(S[2 * m], ah[0], ah[1], ah[2], ah[3], b0, b1);
          mma16816<bf>(S[2 * m + 1], ah[0], ah[1], ah[2], ah[3], b2, b3);
          mma16816<bf>(S[2 * m], al[0], al[1], al[2], al[3], b0, b1);
          mma16816<bf>(S[2 * m + 1], al[0], al[1], al[2], al[3], b2, b3);
        }
      }
      publish_state();
    }
    ptx::cluster_wait_acquire();

    // ---- 5. output norm and gate
#pragma unroll
    for (int half = 0; half < 2; ++half) {
      const int t = rb * 16 + g + half * 8;
      if (t < n_tok) {
        float ss = 0.f;
        for (int d = 0; d < nrank; ++d) ss += sm.ss[ch & 1][d][t];
        const float scale = rsqrtf(ss / static_cast<float>(p.vdim) + p.eps);
        const int64_t tok = t_beg + base + t;
#pragma unroll
        for (int n = 0; n < NO; ++n) {
          const int col = cO + n * 8 + 2 * t4;
          if (col < nv) {
            const float2 w = *reinterpret_cast<const float2*>(sm.norm + col), z = cvt2<bf>(gate[half][n]);
            stf2(p.out + tok * p.out_stride + h * p.vdim + v0 + col, O[n][2 * half] * scale * w.x * silu_ex2(z.x),
                 O[n][2 * half + 1] * scale * w.y * silu_ex2(z.y));
          }
        }
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int n = 0; n < NT; ++n)
#pragma unroll
    for (int e = 0; e < 4; ++e) {
      const int c = rowS + (e >> 1) * 8, col = cS + n * 8 + 2 * t4 + (e & 1);
      if (has_state && c < p.dim && col < nv) gstate[static_cast<int64_t>(c) * p.vdim + col] = S[n][e];
    }
}

template <int DK, int VB, bool WKV>
static cudaError_t launch_gla_chunk(const GlaChunkParams& p, int rows, cudaStream_t stream) {
  auto kern = gla_chunk_kernel<DK, VB, WKV>;
  constexpr int smem = (int)sizeof(GcSmem<DK, VB>);
  static_assert(smem <= 227 * 1024, "shared memory");
  static PerDeviceOnce once;
  cudaError_t e = once.run([&] { return cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem); });
  if (e != cudaSuccess) return e;
  const unsigned vb = (p.vdim + VB - 1) / VB;
  return launch_pdl_cluster(kern, dim3(vb, p.heads, rows), dim3(kGcThreads), (size_t)smem, vb, stream, p);
}

// 128 value columns per block halve the work that every block of a head repeats (scaled operands, scores); 64 give twice
// as many blocks, which is worth more while they do not fill the GPU.
template <int DK, bool WKV>
static cudaError_t launch_gla_width(const GlaChunkParams& p, int rows, int sms, cudaStream_t stream) {
  const bool wide = p.vdim > kGcV && (int64_t)rows * p.heads * ((p.vdim + kGcV - 1) / kGcV) > sms;
  return wide ? launch_gla_chunk<DK, 2 * kGcV, WKV>(p, rows, stream) : launch_gla_chunk<DK, kGcV, WKV>(p, rows, stream);
}

template <bool WKV>
static int gla_chunk_any(const GlaChunkParams& p, int rows, int max_len, cudaStream_t stream) {
  if (p.heads > 65535 || rows > 65535 || (p.row & 7) || (p.out_stride & 1)) return -1;
  for (const void* x : {p.q, p.k, p.v})
    if (reinterpret_cast<uintptr_t>(x) & 15) return -1;
  if (WKV && (reinterpret_cast<uintptr_t>(p.bonus) & 15)) return -1;
  if ((reinterpret_cast<uintptr_t>(p.g) | reinterpret_cast<uintptr_t>(p.out)) & 3) return -1;
  if (reinterpret_cast<uintptr_t>(p.cum) & 15) return -1;
  const int hk = p.heads * p.dim;
  const size_t smem = (size_t)p.rank * (kGdPitch + kGdThreads) * sizeof(float);
  static PerDeviceOnce once;
  cudaError_t e = once.run([] {
    return cudaFuncSetAttribute(gla_decay_kernel<WKV>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                kGdMaxRank * (kGdPitch + kGdThreads) * (int)sizeof(float));
  });
  if (e != cudaSuccess) return (int)e;
  e = launch_pdl(gla_decay_kernel<WKV>, dim3((hk + kGdThreads - 1) / kGdThreads, (max_len + kGcC - 1) / kGcC, rows),
                             dim3(kGdThreads), smem, stream, p);
  if (e != cudaSuccess) return (int)e;
  const int sms = device_sm_count();
  e = p.dim <= 32   ? launch_gla_width<32, WKV>(p, rows, sms, stream)
      : p.dim <= 64 ? launch_gla_width<64, WKV>(p, rows, sms, stream)
                    : launch_gla_width<128, WKV>(p, rows, sms, stream);
  return (int)e;
}

}  // namespace blitz

extern "C" {
using namespace blitz;

// Whether the chunked kernel takes these sizes (bf16 only; vectors of 8 elements).
int blitz_gla_chunk_supported(int dim, int vdim, int rank) {
  return dim > 0 && dim <= 128 && (dim & 7) == 0 && vdim > 0 && (vdim & 7) == 0 && vdim <= kGcV * kGcMaxCluster && rank > 0 &&
         rank <= kGdMaxRank;
}

// Rows of at least one token each: tokens tok_indptr[r] .. tok_indptr[r + 1]; max_len: the longest row.  cum: fp32 scratch
// [tokens][heads * dim], indexed by token number.  The pitch `row` and the five column pointers are multiples of 8 elements.
int blitz_gla_chunk(const void* q, const void* k, const void* v, const void* g, const void* low, int64_t row, const void* a2,
                    const void* a2_b, const void* norm, float* cum, float* state, void* out, int64_t out_stride,
                    const int32_t* pos, const int32_t* tok_indptr, const int32_t* seq_slot, int rows, int max_len, int heads,
                    int dim, int vdim, int rank, int num_slots, float q_scale, float tau, float eps, int* status,
                    cudaStream_t stream) {
  using bf = __nv_bfloat16;
  if (rows <= 0 || max_len <= 0) return 0;
  if (!blitz_gla_chunk_supported(dim, vdim, rank) || !(tau > 0.f)) return -1;
  GlaChunkParams p{(const bf*)q, (const bf*)k, (const bf*)v, (const bf*)g, (const bf*)low, row, nullptr, 0, (const bf*)a2,
                   (const bf*)a2_b, (const bf*)norm, nullptr, 0, cum, state, (bf*)out, out_stride, pos, tok_indptr, seq_slot,
                   heads, dim, vdim, rank, num_slots, q_scale, 1.f / tau, eps, status};
  return gla_chunk_any<false>(p, rows, max_len, stream);
}

// The second form (see blitz_wkv_recurrent for what differs); bonus 16-byte aligned, dim a multiple of 8.
int blitz_wkv_chunk(const void* q, const void* k, const void* v, const void* g, int64_t row, const float* low, int64_t low_row,
                    const void* a2, const void* a2_b, const void* bonus, const void* norm, float* cum, float* state, void* out,
                    int64_t out_stride, const int32_t* pos, const int32_t* tok_indptr, const int32_t* seq_slot, int rows,
                    int max_len, int heads, int dim, int vdim, int rank, int num_slots, float eps, int* status, cudaStream_t stream) {
  using bf = __nv_bfloat16;
  if (rows <= 0 || max_len <= 0) return 0;
  if (!blitz_gla_chunk_supported(dim, vdim, rank) || low == nullptr || bonus == nullptr) return -1;
  GlaChunkParams p{(const bf*)q, (const bf*)k, (const bf*)v, (const bf*)g, nullptr, row, low, low_row, (const bf*)a2,
                   (const bf*)a2_b, (const bf*)norm, (const bf*)bonus, vdim, cum, state, (bf*)out, out_stride, pos, tok_indptr, seq_slot,
                   heads, dim, vdim, rank, num_slots, 1.f, 1.f, eps, status};
  return gla_chunk_any<true>(p, rows, max_len, stream);
}

}  // extern "C"
