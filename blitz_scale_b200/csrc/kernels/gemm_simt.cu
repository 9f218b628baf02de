// Matrix product on the CUDA cores in true fp32 arithmetic, for what the tcgen05 kernels do not take: fp32 operands
// (the 32-bit mode of the engine: no TF32) and 16-bit problems whose sizes are not multiples of 8.  Any size, any
// pitch; 64 x 64 output tiles, 4 x 4 per thread, K in steps of 16 through shared memory.
//
// Epilogues: store (as T or as fp32), C += alpha * acc on an fp32 C (residual stream), silu(gate) * up.
// groups > 1: block-diagonal product.  B holds `groups` blocks [K, N] stacked along K; group g multiplies the K
// columns of A from g * K on and writes the N columns of C from g * N on.
#include "launch.cuh"
#include "ptx.cuh"
#include "scalar.cuh"

namespace blitz {

constexpr int kSgT = 64, kSgK = 16, kSgThreads = 256;

struct SimtGemmParams {
  const void* A;
  const void* B;
  void* C;
  int64_t lda, ldb, ldc;
  int M, N, K, up_off;
  float alpha;
};

enum SimtEpilogue : int { kSimtStore = 0, kSimtSiluMul = 2, kSimtStoreF32 = 4, kSimtAxpyF32 = 5 };

template <typename T, int EPI>
__global__ void __launch_bounds__(kSgThreads) gemm_simt_kernel(const SimtGemmParams p) {
  ptx::griddep_launch_dependents();
  ptx::griddep_wait();
  constexpr int H = EPI == kSimtSiluMul ? 2 : 1;
  __shared__ float sA[kSgK][kSgT + 1];
  __shared__ float sB[H][kSgK][kSgT];
  const int m0 = blockIdx.y * kSgT, n0 = blockIdx.x * kSgT, g = blockIdx.z;
  const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
  const T* A = reinterpret_cast<const T*>(p.A) + static_cast<int64_t>(g) * p.K;
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
      const int64_t at = static_cast<int64_t>(m) * p.ldc + static_cast<int64_t>(g) * p.N + n;
      if (EPI == kSimtAxpyF32) {
        float* c = reinterpret_cast<float*>(p.C) + at;
        *c += p.alpha * acc[0][i][j];
      } else if (EPI == kSimtStoreF32) {
        reinterpret_cast<float*>(p.C)[at] = acc[0][i][j];
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
    case kSimtStoreF32: return launch_pdl(gemm_simt_kernel<T, kSimtStoreF32>, grid, block, 0, stream, p);
    case kSimtAxpyF32: return launch_pdl(gemm_simt_kernel<T, kSimtAxpyF32>, grid, block, 0, stream, p);
    default: return launch_pdl(gemm_simt_kernel<T, kSimtStore>, grid, block, 0, stream, p);
  }
}

}  // namespace blitz

extern "C" {
using namespace blitz;

// C[M, N] = A[M, K] B[K, N] per group; dtype 0 fp16, 1 bf16, 2 fp32 (of A and B, and of C unless the epilogue says
// fp32).  epilogue 0 store, 2 silu(gate) * up with the up columns of B from up_off on, 4 store as fp32,
// 5 C += alpha * acc with C fp32.
int blitz_gemm_simt(const void* A, int64_t lda, const void* B, int64_t ldb, void* C, int64_t ldc, int M, int N, int K,
                    int epilogue, int up_off, float alpha, int groups, int dtype, cudaStream_t stream) {
  if (M <= 0 || N <= 0 || K <= 0 || groups <= 0) return 0;
  if (epilogue != 0 && epilogue != 2 && epilogue != 4 && epilogue != 5) return -1;
  if ((M + kSgT - 1) / kSgT > 65535 || groups > 65535) return -1;
  SimtGemmParams p{A, B, C, lda, ldb, ldc, M, N, K, up_off, alpha};
  cudaError_t e = cudaSuccess;
  BLITZ_DISPATCH_DTYPE3(dtype, (e = launch_simt<T>(p, epilogue, groups, stream)));
  return (int)e;
}

}  // extern "C"
