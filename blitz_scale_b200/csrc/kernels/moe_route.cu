// Router of a mixture of experts: from logits to the work list of the grouped products (gemm_grouped.cu), in one kernel.
//
//   score(t, e)  = sigmoid(z[t][e]), or softmax(z[t])[e]
//   choice(t, e) = score (+ correction[e])              the `top` largest per token are its experts
//   groups       : equal ones of neighbours; only experts of the `keep` groups with the largest choice scores can be chosen
//   weight       = score, or score / sum of the chosen  multiplies the expert's input or its output
//   shared       = sigmoid(z[t][experts])               multiplies the shared expert's output
//
// The last `identity` of the router's outputs are experts that return their input: a token that chooses one gets no row for it
// (its place is -1); the weights of its identity experts are added up in ident[t].
//
// Every (token, expert) pair gets a row of the sorted activations: pairs of one expert are neighbours, experts follow one
// another without gaps, the rows of the shared expert (token t is row pairs + t) come last.  Per row: the token it reads and
// the factors before and after the expert.  `place[t][k]` names the rows of token t.  The work list has one entry (expert,
// first row, rows) per `tile_rows` rows of an expert.
//
// A warp picks a token's experts; the block that finishes last finds where every expert's rows begin and clears the counters
// for the next launch.  The pairs are put into their rows (counting sort) by that block too, or, where they are many, by a
// second kernel.  The order of an expert's rows is not fixed, and nothing that is computed depends on it.
#include "launch.cuh"
#include "ptx.cuh"
#include "scalar.cuh"

namespace blitz {

constexpr int kMoeMaxExperts = 1024;
constexpr int kMoeKeep = 4;           // keys a lane keeps in registers: up to 32 * kMoeKeep experts
constexpr int kMoeSortPairs = 2048;   // more pairs than this go to the second kernel
constexpr int kMoePlacePairs = 4;     // pairs per thread there

struct MoeRouteParams {
  const float* z;        // [tokens][ld]
  int64_t ld;
  int tokens, experts, top, shared, weight_on_input, renormalize, tile_rows, max_tiles, second;
  int identity, softmax, groups, keep;   // groups 0: any expert can be chosen
  const void* correction;                // [experts + identity], or null
  int correction_type;
  float* ident;                          // [tokens] (identity > 0)
  int2* pairs;           // [tokens * top] (expert, weight bits), scratch
  int* counters;         // [2 experts + 1]: rows per expert and finished blocks (zero between launches), next free rows
  int* src;              // [rows] token of a sorted row
  float2* factors;       // [rows] (before, after) the expert
  int* place;            // [tokens][top + shared]
  int4* tiles;           // [max_tiles]
  int* num_tiles;
  int* status;
};

// order-preserving map of a float to an unsigned integer
__device__ __forceinline__ uint32_t order_key(float x) {
  const uint32_t u = __float_as_uint(x);
  return (u & 0x80000000u) ? ~u : (u | 0x80000000u);
}

__device__ __forceinline__ float key_value(uint32_t k) {
  return __uint_as_float((k & 0x80000000u) ? k & 0x7fffffffu : ~k);
}

__device__ __forceinline__ float typed_load(const void* p, int i, int dtype) {
  if (dtype == 2) return reinterpret_cast<const float*>(p)[i];
  return dtype == 1 ? to_f<__nv_bfloat16>(reinterpret_cast<const __nv_bfloat16*>(p)[i]) : to_f<__half>(reinterpret_cast<const __half*>(p)[i]);
}

// Row r belongs to pair i (expert and weight in pr).
__device__ __forceinline__ void place_pair(const MoeRouteParams& p, int i, int2 pr, int r) {
  const int tok = i / p.top;
  const float w = __int_as_float(pr.y);
  p.src[r] = tok;
  p.factors[r] = p.weight_on_input ? make_float2(w, 1.f) : make_float2(1.f, w);
  p.place[tok * (p.top + p.shared) + (i - tok * p.top)] = r;
}

__global__ void __launch_bounds__(1024) moe_route_kernel(const MoeRouteParams p) {
  ptx::griddep_launch_dependents();
  ptx::griddep_wait();
  extern __shared__ int s_dyn[];
  int* s_count = s_dyn;                 // [experts]
  int* s_cursor = s_count + p.experts;  // [experts]
  int* s_tile = s_cursor + p.experts;   // [experts]
  const int E = p.experts, O = E + p.identity, per = p.top + p.shared, pairs = p.tokens * p.top;
  uint32_t* s_groups = reinterpret_cast<uint32_t*>(s_tile + E);                     // [warps][groups]
  uint32_t* s_keys = s_groups + static_cast<int>(blockDim.x >> 5) * p.groups;       // [warps][router outputs]
  __shared__ int s_scan[2][33];
  __shared__ int s_last;
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
  for (int e = threadIdx.x; e < E; e += blockDim.x) s_count[e] = 0;
  __syncthreads();

  const int t = blockIdx.x * warps + warp;
  if (t < p.tokens) {
    const float* z = p.z + t * p.ld;
    uint32_t* keys = s_keys + warp * O;  // only beyond what the registers hold
    uint32_t kept[kMoeKeep];
    const bool in_regs = O <= 32 * kMoeKeep;
    float zmax = 0.f, zsum = 1.f;        // softmax over all outputs
    if (p.softmax) {
      zmax = -INFINITY;
      for (int e = lane; e < O; e += 32) zmax = fmaxf(zmax, z[e]);
      zmax = warp_max(zmax);
      zsum = 0.f;
      for (int e = lane; e < O; e += 32) zsum += expf(z[e] - zmax);
      zsum = warp_sum(zsum);
    }
    // what the choice is made by (plain sigmoid scores are in the order of their logits)
    auto choice = [&](int e) {
      float c = z[e];
      if (p.softmax) c = expf(c - zmax) / zsum;
      if (p.correction) c = (p.softmax ? c : sigmoid_f(c)) + typed_load(p.correction, e, p.correction_type);
      return max(order_key(c), 1u);
    };
    uint32_t best = 0;  // this lane's largest key (0: none left) and its expert
    int best_e = 0x7fffffff;
    auto consider = [&](uint32_t k, int e) {
      if (k > best) {
        best = k;
        best_e = e;
      }
    };
    if (in_regs) {
#pragma unroll
      for (int j = 0; j < kMoeKeep; ++j) {
        const int e = lane + 32 * j;
        kept[j] = e < O ? choice(e) : 0u;
      }
    } else {
      for (int e = lane; e < O; e += 32) keys[e] = choice(e);
    }
    if (p.groups > 0) {
      uint32_t* gk = s_groups + warp * p.groups;  // a group's largest key, then whether it is kept
      const int size = O / p.groups;
      for (int g = lane; g < p.groups; g += 32) gk[g] = 0;
      __syncwarp();
      if (in_regs) {
#pragma unroll
        for (int j = 0; j < kMoeKeep; ++j)
          if (lane + 32 * j < O) atomicMax(&gk[(lane + 32 * j) / size], kept[j]);
      } else {
        for (int e = lane; e < O; e += 32) atomicMax(&gk[e / size], keys[e]);
      }
      __syncwarp();
      uint32_t stay = 0;  // bit i: group lane + 32 i
      for (int g = lane; g < p.groups; g += 32) {
        int before = 0;
        for (int o = 0; o < p.groups; ++o) before += gk[o] > gk[g] || (gk[o] == gk[g] && o < g);
        if (before < p.keep) stay |= 1u << (g >> 5);
      }
      __syncwarp();
      for (int g = lane; g < p.groups; g += 32) gk[g] = (stay >> (g >> 5)) & 1u;
      __syncwarp();
      if (in_regs) {
#pragma unroll
        for (int j = 0; j < kMoeKeep; ++j)
          if (lane + 32 * j < O && gk[(lane + 32 * j) / size] == 0) kept[j] = 0;
      } else {
        for (int e = lane; e < O; e += 32)
          if (gk[e / size] == 0) keys[e] = 0;
      }
    }
    if (in_regs) {
#pragma unroll
      for (int j = 0; j < kMoeKeep; ++j) consider(kept[j], lane + 32 * j);
    } else {
      for (int e = lane; e < O; e += 32) consider(keys[e], e);
    }
    float weight = 0.f, sum = 0.f;  // lane k < top keeps the k-th pair's weight (top <= 32), the sum is everyone's
    int expert = 0;
    for (int k = 0; k < p.top; ++k) {
      const uint32_t mx = __reduce_max_sync(0xffffffffu, best);
      const int e = __reduce_min_sync(0xffffffffu, best == mx ? best_e : 0x7fffffff);
      if (lane == k) {
        weight = key_value(mx);
        expert = e;
      }
      if ((e & 31) == lane) {  // the expert's owner looks for its next best
        best = 0;
        best_e = 0x7fffffff;
        if (in_regs) {
#pragma unroll
          for (int j = 0; j < kMoeKeep; ++j) {
            if (lane + 32 * j == e) kept[j] = 0;
            consider(kept[j], lane + 32 * j);
          }
        } else {
          keys[e] = 0;
          for (int j = lane; j < O; j += 32) consider(keys[j], j);
        }
      }
    }
    if (lane >= p.top) weight = 0.f;
    else if (p.softmax) weight = expf(z[expert] - zmax) / zsum;
    else weight = sigmoid_f(p.correction ? z[expert] : weight);
    if (p.renormalize) {
      sum = warp_sum(weight) + 1e-20f;
      weight /= sum;
    }
    const bool same = lane < p.top && expert >= E;  // an identity expert
    if (p.identity > 0) {
      const float id = warp_sum(same ? weight : 0.f);
      if (lane == 0) p.ident[t] = id;
    }
    if (same) {
      p.pairs[t * p.top + lane] = make_int2(-1, 0);
      p.place[t * per + lane] = -1;
    } else if (lane < p.top) {
      p.pairs[t * p.top + lane] = make_int2(expert, __float_as_int(weight));
      atomicAdd(&s_count[expert], 1);
    }
    if (p.shared && lane == 0) {
      p.src[pairs + t] = t;
      p.factors[pairs + t] = make_float2(1.f, sigmoid_f(z[E]));
      p.place[t * per + p.top] = pairs + t;
    }
  }
  __syncthreads();
  const bool alone = gridDim.x == 1;
  if (!alone) {
    for (int e = threadIdx.x; e < E; e += blockDim.x)
      if (s_count[e]) atomicAdd(&p.counters[e], s_count[e]);
    __threadfence();
    __syncthreads();
    if (threadIdx.x == 0) s_last = atomicAdd(&p.counters[E], 1) == static_cast<int>(gridDim.x) - 1;
    __syncthreads();
    if (!s_last) return;
    __threadfence();
  }

  // rows and tiles of every expert: exclusive sums over the experts
  int rows_before = 0, tiles_before = 0;
  for (int e0 = 0; e0 < E; e0 += blockDim.x) {
    const int e = e0 + threadIdx.x;
    const int n = e < E ? (alone ? s_count[e] : __ldcg(&p.counters[e])) : 0;
    const int nt = (n + p.tile_rows - 1) / p.tile_rows;
    int a = n, b = nt;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int x = __shfl_up_sync(0xffffffffu, a, o), y = __shfl_up_sync(0xffffffffu, b, o);
      if (lane >= o) {
        a += x;
        b += y;
      }
    }
    if (lane == 31) {
      s_scan[0][warp] = a;
      s_scan[1][warp] = b;
    }
    __syncthreads();
    if (threadIdx.x == 0) {
      int x = 0, y = 0;
      for (int w = 0; w < warps; ++w) {
        const int u = s_scan[0][w], v = s_scan[1][w];
        s_scan[0][w] = x;
        s_scan[1][w] = y;
        x += u;
        y += v;
      }
      s_scan[0][32] = x;
      s_scan[1][32] = y;
    }
    __syncthreads();
    if (e < E) {
      s_count[e] = n;
      s_cursor[e] = rows_before + s_scan[0][warp] + a - n;
      s_tile[e] = tiles_before + s_scan[1][warp] + b - nt;
    }
    rows_before += s_scan[0][32];
    tiles_before += s_scan[1][32];
    __syncthreads();
  }
  if (threadIdx.x == 0) {
    if (tiles_before > p.max_tiles) {
      if (p.status) atomicCAS(p.status, 0, kStatusTooLarge);
      tiles_before = p.max_tiles;
    }
    *p.num_tiles = tiles_before;
  }
  for (int e = warp; e < E; e += warps) {
    const int n = s_count[e], r0 = s_cursor[e], t0 = s_tile[e];
    for (int i = lane; i * p.tile_rows < n; i += 32)
      if (t0 + i < p.max_tiles) p.tiles[t0 + i] = make_int4(e, r0 + i * p.tile_rows, min(p.tile_rows, n - i * p.tile_rows), 0);
  }
  if (!alone)
    for (int e = threadIdx.x; e <= E; e += blockDim.x) p.counters[e] = 0;
  if (p.second) {
    for (int e = threadIdx.x; e < E; e += blockDim.x) p.counters[E + 1 + e] = s_cursor[e];
    return;
  }
  __syncthreads();
  constexpr int kAhead = 4;  // pairs a thread reads at once
  for (int i0 = threadIdx.x; i0 < pairs; i0 += kAhead * blockDim.x) {
    int2 pr[kAhead];
#pragma unroll
    for (int j = 0; j < kAhead; ++j) {
      const int i = i0 + j * blockDim.x;
      if (i < pairs) pr[j] = __ldcg(&p.pairs[i]);
    }
#pragma unroll
    for (int j = 0; j < kAhead; ++j) {
      const int i = i0 + j * blockDim.x;
      if (i < pairs && pr[j].x >= 0) place_pair(p, i, pr[j], atomicAdd(&s_cursor[pr[j].x], 1));
    }
  }
}

// Many pairs: a block counts its share per expert, takes that many rows of each, and fills them.
__global__ void __launch_bounds__(256) moe_place_kernel(const MoeRouteParams p) {
  ptx::griddep_launch_dependents();
  ptx::griddep_wait();
  extern __shared__ int s_row[];  // [experts]: this block's pairs, then the next free row
  const int E = p.experts, pairs = p.tokens * p.top, i0 = blockIdx.x * blockDim.x * kMoePlacePairs + threadIdx.x;
  for (int e = threadIdx.x; e < E; e += blockDim.x) s_row[e] = 0;
  __syncthreads();
  int2 pr[kMoePlacePairs];
  int nth[kMoePlacePairs];
#pragma unroll
  for (int j = 0; j < kMoePlacePairs; ++j) {
    const int i = i0 + j * blockDim.x;
    pr[j] = i < pairs ? p.pairs[i] : make_int2(-1, 0);
  }
#pragma unroll
  for (int j = 0; j < kMoePlacePairs; ++j)
    if (pr[j].x >= 0) nth[j] = atomicAdd(&s_row[pr[j].x], 1);
  __syncthreads();
  for (int e = threadIdx.x; e < E; e += blockDim.x)
    if (s_row[e]) s_row[e] = atomicAdd(&p.counters[E + 1 + e], s_row[e]);
  __syncthreads();
#pragma unroll
  for (int j = 0; j < kMoePlacePairs; ++j) {
    const int i = i0 + j * blockDim.x;
    if (pr[j].x >= 0) place_pair(p, i, pr[j], s_row[pr[j].x] + nth[j]);
  }
}

}  // namespace blitz

extern "C" {
using namespace blitz;

// z [tokens][ld] fp32: router logits, the shared expert's in column `experts` (shared = 1, not with identity experts).
// correction: [experts + identity] of type correction_type (0 fp16, 1 bf16, 2 fp32), or null; groups 0: none.  Scratch: pairs (tokens * top
// int2), counters (2 experts + 1 int32, zeroed once).  Results as described at the top of the file; rows = tokens * (top + shared).
int blitz_moe_route(const float* z, int64_t ld, int tokens, int experts, int top, int shared, int weight_on_input, int renormalize,
                    int identity, int softmax, int groups, int keep, const void* correction, int correction_type, float* ident, int tile_rows, int max_tiles, void* pairs, int* counters, int* src, void* factors, int* place, void* tiles,
                    int* num_tiles, int* status, cudaStream_t stream) {
  if (tokens <= 0) return 0;
  const int outputs = experts + identity;
  if (experts < 1 || identity < 0 || outputs > kMoeMaxExperts || top < 1 || top > outputs || top > 32 || tile_rows < 1) return -1;
  if (identity > 0 && (shared || ident == nullptr)) return -1;
  if (groups < 0 || (groups > 0 && (outputs % groups != 0 || keep < 1 || keep > groups || keep * (outputs / groups) < top))) return -1;
  int warps = 32;
  while (warps > 1 && warps * (outputs + groups) * 4 > 32768) warps >>= 1;
  // small steps: all of it in one block, or tokens side by side on several SMs
  while (tokens > warps && warps > 4 && (tokens + warps - 1) / warps < 16) warps >>= 1;
  MoeRouteParams p{z, ld, tokens, experts, top, shared, weight_on_input, renormalize, tile_rows, max_tiles,
                   tokens * top > kMoeSortPairs, identity, softmax, groups, keep, correction, correction_type, ident, reinterpret_cast<int2*>(pairs), counters, src, reinterpret_cast<float2*>(factors),
                   place, reinterpret_cast<int4*>(tiles), num_tiles, status};
  cudaError_t e = launch_pdl(moe_route_kernel, dim3((tokens + warps - 1) / warps), dim3(warps * 32),
                             (size_t)(3 * experts + warps * (groups + (outputs > 32 * kMoeKeep ? outputs : 0))) * sizeof(int), stream, p);
  if (e == cudaSuccess && p.second) {
    const int per = 256 * kMoePlacePairs;
    e = launch_pdl(moe_place_kernel, dim3((tokens * top + per - 1) / per), dim3(256), (size_t)experts * sizeof(int), stream, p);
  }
  return (int)e;
}

}  // extern "C"
