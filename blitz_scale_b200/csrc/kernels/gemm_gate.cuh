// Epilogues of a product with gate and up columns, shared by the products' kernels:
//
//   2   silu(g) * u
//   7   clamped gated unit with biases:  g <- min(g + b_g, limit),  u <- clamp(u + b_u, -limit, limit),
//       g sigmoid(beta g) (u + 1)
#pragma once
#include "scalar.cuh"

namespace blitz {

constexpr int kEpiClampGlu = 7;
__host__ __device__ constexpr bool epi_gated(int epi) { return epi == 2 || epi == kEpiClampGlu; }
__host__ __device__ constexpr bool epi_f32(int epi) { return epi >= 4 && epi <= 6; }

__device__ __forceinline__ float clamp_glu(float g, float u, float limit, float beta) {
  g = fminf(g, limit);
  u = fminf(fmaxf(u, -limit), limit);
  return __fdividef(g, 1.f + __expf(fminf(-beta * g, 80.f))) * (u + 1.f);
}

// 32 gate and up values of columns n .. n + 31 in place: biases added, then the unit; the results are in g.  bias: the gate
// columns' from `bias` on, the up columns' from `bias + up` on (both 16-byte aligned, up a multiple of 8).
template <typename T>
__device__ __forceinline__ void clamp_glu32(const T* bias, int up, int n, int N, float limit, float beta, const float (&g)[32],
                                            const float (&u)[32], float (&out)[32]) {
#pragma unroll
  for (int j = 0; j < 4; ++j) {
    float bg[8] = {}, bu[8] = {};
    if (n + 8 * j < N) {
      ldf8<T>(bias + n + 8 * j, bg);
      ldf8<T>(bias + up + n + 8 * j, bu);
    }
#pragma unroll
    for (int i = 0; i < 8; ++i) out[8 * j + i] = clamp_glu(g[8 * j + i] + bg[i], u[8 * j + i] + bu[i], limit, beta);
  }
}

}  // namespace blitz
