// Work list of a grouped product (the experts of a mixture, see moe_route.cu), shared by its tensor-core and CUDA-core
// kernels.
#pragma once
#include <cuda_runtime.h>
#include <stdint.h>

namespace blitz {

// kActSiluGate: a matrix holds 32 gate columns, the 32 up columns they gate, the next 32 gate columns, and so on; the output
// has half as many columns, silu(gate) * up.
enum GroupedAct : int { kActNone = 0, kActReluSquared = 1, kActSiluGate = 2 };

struct GroupedParams {
  const void* A;
  const void* B;         // [experts * K][N]
  const void* B_shared;  // [K_shared][N_shared], or null
  void* C;
  int64_t lda, ldc;
  int N, K, N_shared, K_shared;
  const int* src;          // row of A behind sorted row r, or null: row r
  const float2* factors;   // per sorted row: (before, after) the activation, or null
  const int4* tiles;       // (expert, first sorted row, rows)
  const int* num_tiles;
  int shared_row0, shared_rows;  // sorted rows of the shared expert
  int tile_rows, act;
};

struct GroupedTile {
  int row0, rows, b_row, N, K;  // rows 0: nothing
  bool shared;
};

// The m-th tile of rows: those of the shared expert come first.
__device__ __forceinline__ GroupedTile grouped_tile(const GroupedParams& p, int m, int num_tiles) {
  const int sh = (p.shared_rows + p.tile_rows - 1) / p.tile_rows;
  GroupedTile g;
  g.shared = m < sh;
  if (g.shared) {
    g.row0 = p.shared_row0 + m * p.tile_rows;
    g.rows = min(p.tile_rows, p.shared_rows - m * p.tile_rows);
    g.b_row = 0;
    g.N = p.N_shared;
    g.K = p.K_shared;
  } else {
    const int4 t = m - sh < num_tiles ? p.tiles[m - sh] : make_int4(0, 0, 0, 0);
    g.row0 = t.y;
    g.rows = t.z;
    g.b_row = t.x * p.K;
    g.N = p.N;
    g.K = p.K;
  }
  return g;
}

__device__ __forceinline__ float grouped_act(int act, float acc, float2 f) {
  float z = acc * f.x;
  if (act == kActReluSquared) {
    z = fmaxf(z, 0.f);
    z *= z;
  }
  return z * f.y;
}

// silu(gate) * up with the factors before (of both accumulators) and after
__device__ __forceinline__ float grouped_silu_gate(float gate, float up, float2 f) {
  const float z = gate * f.x;
  return z / (1.f + __expf(-z)) * (up * f.x) * f.y;
}

}  // namespace blitz
