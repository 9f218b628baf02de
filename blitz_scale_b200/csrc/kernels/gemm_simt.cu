// Matrix product on the CUDA cores in true fp32 arithmetic, for what the tcgen05 kernels do not take: fp32 operands
// (the 32-bit mode of the engine: no TF32) and 16-bit problems whose sizes are not multiples of 8.  Any size, any
// pitch; 64 x 64 output tiles, 4 x 4 per thread, K in steps of 16 through shared memory.
//
// Epilogues: store (as T or as fp32), C += alpha * acc on an fp32 C (residual stream), silu(gate) * up, soft-capped fp32
// store (alpha * tanh(acc / alpha)).
// groups > 1: block-diagonal product.  B holds `groups` blocks [K, N] stacked along K; group g multiplies the K
// columns of A from g * a_step on and writes the N columns of C from g * c_step on.
//
// The second kernel is the grouped product of a mixture of experts (see gemm_grouped.cu) in the same arithmetic.
#include "launch.cuh"
#include "ptx.cuh"
#include "scalar.cuh"
#include "grouped.cuh"
#include "gemm_gate.cuh"

namespace blitz {

constexpr int kSgT = 64, kSgK = 16, kSgThreads = 256;

struct SimtGemmParams {
  const void* A;
  const void* B;
  void* C;
  int64_t lda, ldb, ldc;
  int M, N, K, up_off, a_step, c_step;
  float alpha, beta;
  const void* bias;
};

enum SimtEpilogue : int { kSimtStore = 0, kSimtSiluMul = 2, kSimtStoreF32 = 4, kSimtAxpyF32 = 5, kSimtCapF32 = 6, kSimtClampGlu = kEpiClampGlu };

template <typename T, int EPI>
__global__ void __launch_bounds__(kSgThreads) gemm_simt_kernel(const SimtGemmParams p) {
  ptx::griddep_launch_dependents();
  ptx::griddep_wait();
  constexpr int H = epi_gated(EPI) ? 2 : 1;
  __shared__ float sA[kSgK][kSgT + 1];
  __shared__ float sB[H][kSgK][kSgT];
  const int m0 = blockIdx.y * kSgT, n0 = blockIdx.x * kSgT, g = blockIdx.z;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  const T* A = reinterpret_cast<const T*>(p.A) + static_cast<int64_t>(g) * p.a_step;
  const T* B = reinterpret_cast<const T*>(p.B) + static_cast<int64_t>(g) * p.K * p.ldb;
  float acc[H][4][4];
#pragma unroll
  for (int h = 0; h < H; ++h)
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
      for (int j = 0; j < 4; ++j) acc[h][i][j] = 0.f;
  for (int k0 = 0; k0 < p.K; k0 += kSgK) {
#pragma unroll
    for (int e = threadIdx.x; e < kSgT * kSgK; e += kSgThreads) {
      const int m = e / kSgK, k = e % kSgK;
      sA[k][m] = (m0 + m < p.M && k0 + k < p.K) ? ldf<T>(A + static_cast<int64_t>(m0 + m) * p.lda + k0 + k) : 0.f;
      const int n = e % kSgT, kb = e / kSgT;
      const bool ok = n0 + n < p.N && k0 + kb < p.K;
#pragma unroll
      for (int h = 0; h < H; ++h)
        sB[h][kb][n] = ok ? ldf<T>(B + static_cast<int64_t>(k0 + kb) * p.ldb + n0 + n + h * p.up_off) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kSgK; ++k) {
      float a[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) a[i] = sA[k][ty * 4 + i];
#pragma unroll
      for (int h = 0; h < H; ++h)
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const float b = sB[h][k][tx + 16 * j];
#pragma unroll
          for (int i = 0; i < 4; ++i) acc[h][i][j] += a[i] * b;
        }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = m0 + ty * 4 + i;
    if (m >= p.M) continue;
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx + 16 * j;
      if (n >= p.N) continue;
      const int64_t at = static_cast<int64_t>(m) * p.ldc + static_cast<int64_t>(g) * p.c_step + n;
      if (EPI == kSimtAxpyF32) {
        float* c = reinterpret_cast<float*>(p.C) + at;
        *c += p.alpha * acc[0][i][j];
      } else if (EPI == kSimtCapF32) {
        reinterpret_cast<float*>(p.C)[at] = p.alpha * tanhf(acc[0][i][j] / p.alpha);
      } else if (EPI == kSimtStoreF32) {
        reinterpret_cast<float*>(p.C)[at] = acc[0][i][j];
      } else if (EPI == kSimtClampGlu) {
        const T* bias = reinterpret_cast<const T*>(p.bias) + n;
        const float z = fminf(acc[0][i][j] + ldf<T>(bias), p.alpha);
        const float u = fminf(fmaxf(acc[H - 1][i][j] + ldf<T>(bias + p.up_off), -p.alpha), p.alpha);
        stf<T>(reinterpret_cast<T*>(p.C) + at, z * sigmoid_f(p.beta * z) * (u + 1.f));
      } else if (EPI == kSimtSiluMul) {
        stf<T>(reinterpret_cast<T*>(p.C) + at, silu_acc(acc[0][i][j]) * acc[H - 1][i][j]);
      } else {
        stf<T>(reinterpret_cast<T*>(p.C) + at, acc[0][i][j]);
      }
    }
  }
}

template <typename T>
static cudaError_t launch_simt(const SimtGemmParams& p, int epi, int groups, cudaStream_t stream) {
  const dim3 grid((p.N + kSgT - 1) / kSgT, (p.M + kSgT - 1) / kSgT, groups), block(kSgThreads);
  switch (epi) {
    case kSimtSiluMul: return launch_pdl(gemm_simt_kernel<T, kSimtSiluMul>, grid, block, 0, stream, p);
    case kSimtClampGlu: return launch_pdl(gemm_simt_kernel<T, kSimtClampGlu>, grid, block, 0, stream, p);
    case kSimtStoreF32: return launch_pdl(gemm_simt_kernel<T, kSimtStoreF32>, grid, block, 0, stream, p);
    case kSimtCapF32: return launch_pdl(gemm_simt_kernel<T, kSimtCapF32>, grid, block, 0, stream, p);
    case kSimtAxpyF32: return launch_pdl(gemm_simt_kernel<T, kSimtAxpyF32>, grid, block, 0, stream, p);
    default: return launch_pdl(gemm_simt_kernel<T, kSimtStore>, grid, block, 0, stream, p);
  }
}

// ------------------------------------------------------------------ grouped product
template <typename T>
__global__ void __launch_bounds__(kSgThreads) gemm_grouped_simt_kernel(const GroupedParams p) {
  ptx::griddep_launch_dependents();
  ptx::griddep_wait();
  __shared__ float sA[kSgK][kSgT + 1];
  __shared__ float sB[kSgK][kSgT];
  const GroupedTile g = grouped_tile(p, blockIdx.y, *p.num_tiles);
  const int n0 = blockIdx.x * kSgT;
  if (g.rows <= 0 || n0 >= g.N) return;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  const T* A = reinterpret_cast<const T*>(p.A);
  const T* B = reinterpret_cast<const T*>(g.shared ? p.B_shared : p.B) + static_cast<int64_t>(g.b_row) * g.N;
  float acc[4][4] = {};
  for (int k0 = 0; k0 < g.K; k0 += kSgK) {
#pragma unroll
    for (int e = threadIdx.x; e < kSgT * kSgK; e += kSgThreads) {
      const int m = e / kSgK, k = e % kSgK;
      float a = 0.f;
      if (m < g.rows && k0 + k < g.K) {
        const int row = p.src ? p.src[g.row0 + m] : g.row0 + m;
        a = ldf<T>(A + static_cast<int64_t>(row) * p.lda + k0 + k);
      }
      sA[k][m] = a;
      const int n = e % kSgT, kb = e / kSgT;
      sB[kb][n] = n0 + n < g.N && k0 + kb < g.K ? ldf<T>(B + static_cast<int64_t>(k0 + kb) * g.N + n0 + n) : 0.f;
    }
    __syncthreads();
#pragma unroll
    for (int k = 0; k < kSgK; ++k) {
      float a[4];
#pragma unroll
      for (int i = 0; i < 4; ++i) a[i] = sA[k][ty * 4 + i];
#pragma unroll
      for (int j = 0; j < 4; ++j) {
        const float b = sB[k][tx + 16 * j];
#pragma unroll
        for (int i = 0; i < 4; ++i) acc[i][j] += a[i] * b;
      }
    }
    __syncthreads();
  }
#pragma unroll
  for (int i = 0; i < 4; ++i) {
    const int m = ty * 4 + i;
    if (m >= g.rows) continue;
    const float2 f = p.factors ? p.factors[g.row0 + m] : make_float2(1.f, 1.f);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
      const int n = n0 + tx + 16 * j;
      T* dst = reinterpret_cast<T*>(p.C) + static_cast<int64_t>(g.row0 + m) * p.ldc;
      if (p.act == kActSiluGate) {  // columns 0 .. 31 of the tile gate columns 32 .. 63
        if (j < 2 && n < g.N) {
          const float z = acc[i][j] * f.x;
          stf<T>(dst + n0 / 2 + tx + 16 * j, silu_acc(z) * (acc[i][(j + 2) & 3] * f.x) * f.y);
        }
      } else if (n < g.N) {
        stf<T>(dst + n, grouped_act(p.act, acc[i][j], f));
      }
    }
  }
}

}  // namespace blitz

extern "C" {
using namespace blitz;

// C[M, N] = A[M, K] B[K, N] per group; dtype 0 fp16, 1 bf16, 2 fp32 (of A and B, and of C unless the epilogue says
// fp32).  epilogue 0 store, 2 silu(gate) * up with the up columns of B from up_off on, 4 store as fp32,
// 5 C += alpha * acc with C fp32, 6 alpha * tanh(acc / alpha) as fp32, 7 clamped gated unit
// (gemm_gate.cuh).  a_step, c_step: columns of A and C between two groups.
int blitz_gemm_simt(const void* A, int64_t lda, const void* B, int64_t ldb, void* C, int64_t ldc, int M, int N, int K,
                    int epilogue, int up_off, const void* bias, float alpha, float beta, int groups, int a_step, int c_step, int dtype, cudaStream_t stream) {
  if (M <= 0 || N <= 0 || K <= 0 || groups <= 0) return 0;
  if (epilogue != 0 && epilogue != 2 && epilogue != 4 && epilogue != 5 && epilogue != 6 && epilogue != kEpiClampGlu) return -1;
  if (epilogue == kEpiClampGlu && bias == nullptr) return -1;
  if (epilogue == 6 && !(alpha > 0.f)) return -1;
  if ((M + kSgT - 1) / kSgT > 65535 || groups > 65535) return -1;
  SimtGemmParams p{A, B, C, lda, ldb, ldc, M, N, K, up_off, a_step, c_step, alpha, beta, bias};
  cudaError_t e = cudaSuccess;
  BLITZ_DISPATCH_DTYPE3(dtype, (e = launch_simt<T>(p, epilogue, groups, stream)));
  return (int)e;
}

// Grouped product on the CUDA cores; arguments as for blitz_gemm_grouped (work list with tile_rows 64).
int blitz_gemm_grouped_simt(const void* A, int64_t lda, const int* src, const void* B, int N, int K, const void* B_shared,
                            int N_shared, int K_shared, void* C, int64_t ldc, const void* factors, const void* tiles,
                            const int* num_tiles, int max_tiles, int shared_row0, int shared_rows, int act, int dtype,
                            cudaStream_t stream) {
  GroupedParams p{A, B, B_shared, C, lda, ldc, N, K, N_shared, K_shared, src, reinterpret_cast<const float2*>(factors),
                  reinterpret_cast<const int4*>(tiles), num_tiles, shared_row0, B_shared ? shared_rows : 0, kSgT, act};
  const int y = max_tiles + (p.shared_rows + kSgT - 1) / kSgT, n = N > N_shared ? N : N_shared;
  if (y <= 0 || N <= 0 || K <= 0) return 0;
  if (y > 65535) return -1;
  cudaError_t e = cudaSuccess;
  BLITZ_DISPATCH_DTYPE3(dtype, (e = launch_pdl(gemm_grouped_simt_kernel<T>, dim3((n + kSgT - 1) / kSgT, y), dim3(kSgThreads), 0, stream, p)));
  return (int)e;
}

}  // extern "C"
