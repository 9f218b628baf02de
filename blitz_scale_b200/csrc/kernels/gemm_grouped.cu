// Grouped product of a mixture of experts on tcgen05: every expert's rows times that expert's matrix, in one launch.
//
//   C[r] = after_r * act(before_r * (A[src(r)] * B[expert(r)]))        16-bit operands, fp32 accumulation in TMEM
//
// Sorted rows r and their work list come from moe_route.cu on the device, so the launch does not depend on how tokens are
// spread over the experts and can be captured in a graph.  The shared expert, whose matrix may have another size, is one
// more group over all tokens.  The first product of an expert gathers its rows through `src` while loading, so tokens are
// never copied into expert order; the second one reads the first one's sorted rows.  Two ways to gather: TMA gather (four
// rows per request, about 90 cycles each: right for the few rows per expert of a decode step), and four more warps that copy
// 16-byte pieces with cp.async into the swizzled tile (which keeps up with full tiles).
//
// A work item is one tile of at most 128 rows of one expert and BN columns.  Persistent grid, warp-specialised as in
// gemm_tcgen05.cu: load warp (every lane requests four gathered rows, or one box; some lanes a 64-column slab of B), one
// issuing thread, four epilogue warps, the accumulator double buffered in TMEM.  Rows beyond a tile's end hold whatever
// the stage held before: a row of the accumulator depends on its own row of A only, and rows beyond the end are not stored.
// With few rows per expert (decode) the kernel is a stream over the chosen experts' weights; a stage of A is then only as
// tall as the step has tokens, which leaves the shared memory to weights in flight.
#include "launch.cuh"
#include "ptx.cuh"
#include "tmap.cuh"
#include "common.cuh"
#include "grouped.cuh"

namespace blitz {

constexpr int kGgRows = 128, kGgK = 64, kGgThreads = 192, kGgMaxStages = 16;
constexpr int kGgGather4Rows = 64;   // tiles of more rows than this are gathered by the copying warps
constexpr int kGgCopyThreads = 128;

// how a tile of A is fetched: sorted rows by boxes, or gathered by TMA or by copying warps
enum GgFetch : int { kGgBoxes = 0, kGgGather4 = 1, kGgCopy = 2 };

struct GroupedTcParams {
  GroupedParams g;
  int a_rows;      // rows a stage of A holds: min(128, rows any tile can have), a multiple of 32
  int box;         // rows per box of A: 32, or 128 where tiles are mostly full
  int src_rows;    // rows of A (bound of src)
  int sh_tiles, tn, tn_shared;
  int* status;
};

template <int BN>
struct GgCfg {
  static constexpr int kBBytes = BN * kGgK * 2;
  static constexpr int kBarBytes = (2 * kGgMaxStages + 4) * 8 + 16;
  static constexpr int kSmemBytes = 227 * 1024;
  static constexpr int kUsable = kSmemBytes - 1024 - kBarBytes;
  // (the 128-row view of the last short stage of A ends in the B stages that follow, which are larger than a tile of A)
  __host__ __device__ static constexpr int stages(int a_rows) {
    const int s = kUsable / (a_rows * 128 + kBBytes);
    return s > kGgMaxStages ? kGgMaxStages : s;
  }
};

struct Ring {  // position in the ring of pipeline stages
  int stage;
  uint32_t phase;
  int size;
  __device__ __forceinline__ void next() {
    if (++stage == size) {
      stage = 0;
      phase ^= 1u;
    }
  }
};

struct GgItem {
  GroupedTile t;
  int n0;
};
__device__ __forceinline__ GgItem gg_item(const GroupedTcParams& p, int w, int num_tiles) {
  const int sh_items = p.sh_tiles * p.tn_shared;
  GgItem it;
  int m, n, per;
  if (w < sh_items) {
    per = p.tn_shared;
    m = w / per;
    n = w - m * per;
  } else {
    per = p.tn;
    m = (w - sh_items) / per;
    n = (w - sh_items) - m * per;
    m += p.sh_tiles;
  }
  it.t = grouped_tile(p.g, m, num_tiles);
  it.n0 = n;  // column block; the caller scales it
  return it;
}

template <typename T, int BN, int FETCH>
__global__ void __launch_bounds__(FETCH == kGgCopy ? kGgThreads + kGgCopyThreads : kGgThreads, 1)
gemm_grouped_kernel(const __grid_constant__ CUtensorMap tmap_a, const __grid_constant__ CUtensorMap tmap_a_shared,
                    const __grid_constant__ CUtensorMap tmap_b, const __grid_constant__ CUtensorMap tmap_b_shared,
                    const GroupedTcParams p) {
  using Cfg = GgCfg<BN>;
  constexpr uint32_t kFmt = std::is_same<T, __nv_bfloat16>::value ? 1u : 0u;
  constexpr uint32_t kIdesc = ptx::make_idesc_f16(kFmt, 0u, 1u, kGgRows, BN);
  const int S = Cfg::stages(p.a_rows);
  const int a_stage = p.a_rows * 128;

  extern __shared__ uint8_t smem_raw[];
  const uint32_t raw_addr = ptx::smem_u32(smem_raw);
  uint8_t* smem = smem_raw + (((raw_addr + 1023u) & ~1023u) - raw_addr);
  uint8_t* smem_a = smem;
  uint8_t* smem_b = smem + S * a_stage;
  uint64_t* full_bar = reinterpret_cast<uint64_t*>(smem + Cfg::kUsable);  // [S]
  uint64_t* empty_bar = full_bar + kGgMaxStages;                          // [S]
  uint64_t* tfull_bar = empty_bar + kGgMaxStages;                         // [2]
  uint64_t* tempty_bar = tfull_bar + 2;                                   // [2]
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(tempty_bar + 2);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

  if (threadIdx.x == 0) {
    for (int i = 0; i < S; ++i) {
      ptx::mbar_init(&full_bar[i], FETCH == kGgCopy ? 1 + kGgCopyThreads : 1);
      ptx::mbar_init(&empty_bar[i], 1);
    }
    for (int i = 0; i < 2; ++i) {
      ptx::mbar_init(&tfull_bar[i], 1);
      ptx::mbar_init(&tempty_bar[i], 128);
    }
    *abort_flag = 0;
    ptx::fence_mbar_init();
    ptx::tma_prefetch_desc(&tmap_a);
    ptx::tma_prefetch_desc(&tmap_b);
  }
  if (warp == 1) {
    ptx::tmem_alloc(tmem_slot, 2 * BN);
    ptx::tmem_relinquish();
  }
  ptx::tc_fence_before_sync();
  __syncthreads();
  ptx::tc_fence_after_sync();
  const uint32_t tmem_base = *tmem_slot;
  ptx::griddep_launch_dependents();
  ptx::griddep_wait();
  const int num_tiles = *p.g.num_tiles;
  const int items = p.sh_tiles * p.tn_shared + num_tiles * p.tn;

  if (warp == 0) {
    // ------------------------------------------------------------ load warp
    Ring g{0, 0u, S};
    bool ok = true;
    for (int w = blockIdx.x; w < items && ok; w += gridDim.x) {
      const GgItem it = gg_item(p, w, num_tiles);
      const int n0 = it.n0 * BN, num_kb = (it.t.K + kGgK - 1) / kGgK;
      const CUtensorMap* ta = it.t.shared ? &tmap_a_shared : &tmap_a;
      const CUtensorMap* tb = it.t.shared ? &tmap_b_shared : &tmap_b;
      int pieces = 0;
      int idx[4] = {0, 0, 0, 0};
      // the shared expert's rows are the tokens in order: no need to gather them row by row
      const bool gather = FETCH == kGgGather4 && !it.t.shared;
      if (gather) {
        pieces = (it.t.rows + 3) >> 2;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
          const int r = 4 * lane + j;
          if (r < it.t.rows) idx[j] = p.g.src[it.t.row0 + r];
          if (idx[j] < 0 || idx[j] >= p.src_rows) {
            if (p.status) atomicCAS(p.status, 0, kStatusBadIndex);
            idx[j] = 0;
          }
        }
      } else if (FETCH != kGgCopy) {
        pieces = (it.t.rows + p.box - 1) / p.box;
      }
      const uint32_t tx = static_cast<uint32_t>(pieces) * (gather ? 512u : p.box * 128u) + Cfg::kBBytes;
      const int row0 = FETCH == kGgGather4 ? it.t.row0 - p.g.shared_row0 : it.t.row0;  // of the boxes
      for (int kb = 0; kb < num_kb; ++kb) {
        int good = 1;
        if (lane == 0) {
          good = ptx::bounded_mbar_wait(&empty_bar[g.stage], g.phase ^ 1u, abort_flag) ? 1 : 0;
          if (good) ptx::mbar_expect_tx(&full_bar[g.stage], tx);
          else if (p.status) atomicCAS(p.status, 0, kStatusTimeoutProducer);
        }
        ok = __shfl_sync(0xffffffffu, good, 0) != 0;
        if (!ok) break;
        if (lane < BN / 64)  // slabs of 64 columns x 64 K rows
          ptx::tma_load_2d(smem_b + g.stage * Cfg::kBBytes + lane * 8192, tb, &full_bar[g.stage], n0 + lane * 64, it.t.b_row + kb * kGgK);
        if (lane < pieces) {
          uint8_t* sa = smem_a + g.stage * a_stage;
          if (gather)
            ptx::tma_gather4(sa + lane * 512, ta, &full_bar[g.stage], kb * kGgK, idx[0], idx[1], idx[2], idx[3]);
          else
            ptx::tma_load_2d(sa + lane * (p.box * 128), ta, &full_bar[g.stage], kb * kGgK, row0 + lane * p.box);
        }
        g.next();
      }
    }
  } else if (warp == 1) {
    // ------------------------------------------------------------ UMMA issuer
    if (lane == 0) {
      Ring g{0, 0u, S};
      int acc = 0;
      uint32_t acc_phase = 0;
      bool ok = true;
      for (int w = blockIdx.x; w < items && ok; w += gridDim.x) {
        const GgItem it = gg_item(p, w, num_tiles);
        const int num_kb = (it.t.K + kGgK - 1) / kGgK;
        if (!ptx::bounded_mbar_wait(&tempty_bar[acc], acc_phase ^ 1u, abort_flag)) {
          if (p.status) atomicCAS(p.status, 0, kStatusTimeoutMma);
          break;
        }
        ptx::tc_fence_after_sync();
        const uint32_t d_tmem = tmem_base + static_cast<uint32_t>(acc * BN);
        for (int kb = 0; kb < num_kb; ++kb) {
          if (!ptx::bounded_mbar_wait(&full_bar[g.stage], g.phase, abort_flag)) {
            if (p.status) atomicCAS(p.status, 0, kStatusTimeoutMma);
            ok = false;
            break;
          }
          ptx::tc_fence_after_sync();
          const uint32_t a_base = ptx::smem_u32(smem_a + g.stage * a_stage);
          const uint32_t b_base = ptx::smem_u32(smem_b + g.stage * Cfg::kBBytes);
#pragma unroll
          for (int k = 0; k < kGgK / 16; ++k) {
            const uint64_t adesc = ptx::make_smem_desc(a_base + k * 32, 16, 1024, ptx::kLayoutSw128);
            const uint64_t bdesc = ptx::make_smem_desc(b_base + k * 2048, 8192, 1024, ptx::kLayoutSw128);
            ptx::umma_f16_ss(d_tmem, adesc, bdesc, kIdesc, (kb | k) != 0 ? 1u : 0u);
          }
          ptx::umma_commit(&empty_bar[g.stage]);
          g.next();
        }
        if (!ok) break;
        ptx::umma_commit(&tfull_bar[acc]);
        acc ^= 1;
        if (acc == 0) acc_phase ^= 1u;
      }
    }
  } else if (FETCH == kGgCopy && warp >= 6) {
    // ------------------------------------------------------------ copying warps: eight lanes per row of 128 bytes
    const int tid = threadIdx.x - kGgThreads, chunk = tid & 7, r0 = tid >> 3;
    constexpr int kPasses = kGgRows * 8 / kGgCopyThreads, kStep = kGgCopyThreads / 8;
    constexpr int kAhead = Cfg::stages(kGgRows) - 2;  // stages in flight behind the one being requested
    Ring g{0, 0u, S};
    int behind = 0, signal = 0;  // stages requested but not signalled yet, the next of them
    bool ok = true;
    auto done = [&]() {  // the oldest stage's pieces have landed: hand them to the tensor core's proxy
      ptx::fence_proxy_async_smem();
      ptx::mbar_arrive(&full_bar[signal]);
      if (++signal == S) signal = 0;
      --behind;
    };
    for (int w = blockIdx.x; w < items && ok; w += gridDim.x) {
      const GgItem it = gg_item(p, w, num_tiles);
      const int num_kb = (it.t.K + kGgK - 1) / kGgK;
      const T* row[kPasses];
#pragma unroll
      for (int j = 0; j < kPasses; ++j) {
        const int r = r0 + j * kStep;
        int i = r < it.t.rows ? p.g.src[it.t.row0 + r] : -1;
        if (i >= p.src_rows || (i < 0 && r < it.t.rows)) {
          if (p.status) atomicCAS(p.status, 0, kStatusBadIndex);
          i = -1;
        }
        row[j] = i < 0 ? nullptr : reinterpret_cast<const T*>(p.g.A) + static_cast<int64_t>(i) * p.g.lda + chunk * 8;
      }
      for (int kb = 0; kb < num_kb; ++kb) {
        if (!ptx::bounded_mbar_wait(&empty_bar[g.stage], g.phase ^ 1u, abort_flag)) {
          if (p.status && tid == 0) atomicCAS(p.status, 0, kStatusTimeoutProducer);
          ok = false;
          break;
        }
        const uint32_t sa = ptx::smem_u32(smem_a + g.stage * a_stage);
        const bool inside = kb * kGgK + chunk * 8 < it.t.K;  // beyond K: zeros
#pragma unroll
        for (int j = 0; j < kPasses; ++j) {
          const int r = r0 + j * kStep;
          if (row[j] != nullptr)
            ptx::cp_async_16(sa + r * 128 + ((chunk ^ (r & 7)) << 4), inside ? row[j] + kb * kGgK : row[j], inside ? 16u : 0u);
        }
        ptx::cp_async_commit();
        g.next();
        if (++behind > kAhead) {
          ptx::cp_async_wait<kAhead>();
          done();
        }
      }
    }
    ptx::cp_async_wait<0>();
    while (behind > 0) done();
  } else {
    // ------------------------------------------------------------ epilogue warps
    const int q = warp & 3;  // TMEM lane quarter this warp may read
    int acc = 0;
    uint32_t acc_phase = 0;
    for (int w = blockIdx.x; w < items; w += gridDim.x) {
      const GgItem it = gg_item(p, w, num_tiles);
      const int n0 = it.n0 * BN, r = q * 32 + lane;
      const bool row_ok = r < it.t.rows;
      const int row = it.t.row0 + r;
      float2 f = make_float2(1.f, 1.f);
      if (p.g.factors && row_ok) f = p.g.factors[row];
      if (!ptx::bounded_mbar_wait(&tfull_bar[acc], acc_phase, abort_flag)) {
        if (p.status && lane == 0) atomicCAS(p.status, 0, kStatusTimeoutEpilogue);
        break;
      }
      ptx::tc_fence_after_sync();
      if (q * 32 < it.t.rows) {
        const uint32_t taddr = tmem_base + (static_cast<uint32_t>(q * 32) << 16) + static_cast<uint32_t>(acc * BN);
        const bool gated = p.g.act == kActSiluGate;
        T* dst = reinterpret_cast<T*>(p.g.C) + static_cast<int64_t>(row) * p.g.ldc + (gated ? n0 / 2 : n0);
        const int cols = min(BN, it.t.N - n0);
        if (gated) {
#pragma unroll 1
          for (int c = 0; c < cols; c += 64) {
            uint32_t v[32], u[32];
            ptx::tmem_ld_32x32(taddr + c, v);
            ptx::tmem_ld_32x32(taddr + c + 32, u);
            ptx::tmem_ld_wait();
            if (row_ok) {
#pragma unroll
              for (int j = 0; j < 4; ++j) {
                float x[8];
#pragma unroll
                for (int i = 0; i < 8; ++i) x[i] = grouped_silu_gate(__uint_as_float(v[8 * j + i]), __uint_as_float(u[8 * j + i]), f);
                *reinterpret_cast<uint4*>(dst + c / 2 + 8 * j) = pack8<T>(x);
              }
            }
          }
        } else
#pragma unroll 1
        for (int c = 0; c < cols; c += 32) {
          uint32_t v[32];
          ptx::tmem_ld_32x32(taddr + c, v);
          ptx::tmem_ld_wait();
          if (row_ok) {
#pragma unroll
            for (int j = 0; j < 4; ++j) {
              if (c + 8 * j < cols) {
                float x[8];
#pragma unroll
                for (int i = 0; i < 8; ++i) x[i] = grouped_act(p.g.act, __uint_as_float(v[8 * j + i]), f);
                *reinterpret_cast<uint4*>(dst + c + 8 * j) = pack8<T>(x);
              }
            }
          }
        }
      }
      ptx::tc_fence_before_sync();
      ptx::mbar_arrive(&tempty_bar[acc]);
      acc ^= 1;
      if (acc == 0) acc_phase ^= 1u;
    }
  }

  ptx::tc_fence_before_sync();
  __syncthreads();
  if (warp == 1) {
    ptx::tc_fence_after_sync();
    ptx::tmem_dealloc(tmem_base, 2 * BN);
  }
}

template <typename T, int BN, int FETCH>
static int launch_grouped(const CUtensorMap& ta, const CUtensorMap& tas, const CUtensorMap& tb, const CUtensorMap& tbs,
                          const GroupedTcParams& p, int grid, cudaStream_t stream) {
  auto kern = gemm_grouped_kernel<T, BN, FETCH>;
  static PerDeviceOnce once;
  cudaError_t e = once.run([&] { return cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, GgCfg<BN>::kSmemBytes); });
  if (e != cudaSuccess) return (int)e;
  return (int)launch_pdl(kern, dim3(grid), dim3(FETCH == kGgCopy ? kGgThreads + kGgCopyThreads : kGgThreads), GgCfg<BN>::kSmemBytes, stream, ta, tas, tb, tbs, p);
}

}  // namespace blitz

extern "C" {
using namespace blitz;

// A [a_rows][lda]; src: row of A behind each sorted row (null: the sorted row itself); those of the shared expert are rows
// 0 .. shared_rows - 1.  B: the experts' matrices [K][N]
// stacked along K; B_shared [K_shared][N_shared] or null.  C [sorted rows][ldc].  factors: per sorted row (before, after), or
// null.  tiles / num_tiles / max_tiles: work list with tile_rows 128; typical_*: expected tiles and rows of a tile,
// max_rows: most rows any tile can have (all three for the launch's shape only).  act: 0 none, 1 square of relu, 2 silu(gate) * up
// (grouped.cuh; N a multiple of 64, C has N / 2 columns; without a shared expert).  dtype 0 fp16, 1 bf16.  bn_hint: 0 = choose, else 64 / 128 / 256.  fetch_hint: 0 = choose
// how rows are gathered, 1 TMA, 2 copying warps.  N, K, pitches: multiples of 8.  Expert's K rows are read up to the next multiple of 64: what lies behind them meets zero columns of A.
int blitz_gemm_grouped(const void* A, int64_t lda, int a_rows, const int* src, const void* B, int experts, int N, int K,
                       const void* B_shared, int N_shared, int K_shared, void* C, int64_t ldc, const void* factors,
                       const void* tiles, const int* num_tiles, int max_tiles, int typical_tiles, int typical_rows, int shared_row0, int shared_rows,
                       int max_rows, int act, int bn_hint, int fetch_hint, int* status, int dtype, cudaStream_t stream) {
  if (a_rows <= 0 || N <= 0 || K <= 0) return 0;
  if (((N | K | N_shared | K_shared) & 7) || (lda & 7) || (ldc & 7) || act < 0 || act > 2) return -1;
  if (act == kActSiluGate && ((N & 63) || B_shared)) return -1;
  if ((reinterpret_cast<uintptr_t>(C) & 15) != 0 || (reinterpret_cast<uintptr_t>(tiles) & 15) != 0) return -1;
  if (lda < K || (B_shared && lda < K_shared)) return -1;
  const int sms = device_sm_count();
  GroupedTcParams p;
  p.g = GroupedParams{A, B, B_shared, C, lda, ldc, N, K, N_shared, K_shared, src, reinterpret_cast<const float2*>(factors),
                      reinterpret_cast<const int4*>(tiles), num_tiles, shared_row0, B_shared ? shared_rows : 0, kGgRows, act};
  p.a_rows = max_rows >= kGgRows ? kGgRows : (max_rows + 31) / 32 * 32;
  p.box = p.a_rows == kGgRows && typical_rows > 64 ? kGgRows : 32;
  p.src_rows = a_rows;
  p.status = status;
  p.sh_tiles = (p.g.shared_rows + kGgRows - 1) / kGgRows;
  int bn = bn_hint;
  if (bn != 64 && bn != 128 && bn != 256) {
    // Rounds of items per SM times the cycles of a 64-deep step.  Full tiles are bound by the tensor pipe (a 128-row MMA of
    // K = 16 takes 95 / 105 / 150 cycles at N = 64 / 128 / 256), tiles of few rows by what one SM can stream (50 GB/s).
    const bool stream_bound = max_rows <= kGgRows;
    int64_t best = INT64_MAX;
    for (int b = 256; b >= 64; b /= 2) {
      const int64_t items = (int64_t)p.sh_tiles * ((N_shared + b - 1) / b) + (int64_t)typical_tiles * ((N + b - 1) / b);
      const int step = b == 64 ? 430 : b == 128 ? (stream_bound ? 630 : 480) : (stream_bound ? 1260 : 650);
      const int64_t cost = (items + sms - 1) / sms * step;
      if (cost < best) {
        best = cost;
        bn = b;
      }
    }
  }
  p.tn = (N + bn - 1) / bn;
  p.tn_shared = B_shared ? (N_shared + bn - 1) / bn : 0;
  const bool copy = src && (fetch_hint ? fetch_hint == kGgCopy : max_rows > kGgGather4Rows);
  if (copy) p.a_rows = kGgRows;
  CUtensorMap ta, tas, tb, tbs;
  if (src) {
    if (!get_tmap_2d(&ta, A, (uint64_t)K, (uint64_t)a_rows, (uint64_t)lda * 2, kGgK, 1)) return -2;
    tas = ta;
    if (B_shared && !get_tmap_2d(&tas, A, (uint64_t)K_shared, (uint64_t)a_rows, (uint64_t)lda * 2, kGgK, (uint32_t)p.box)) return -2;
  } else {
    if (!get_tmap_2d(&ta, A, (uint64_t)K, (uint64_t)a_rows, (uint64_t)lda * 2, kGgK, (uint32_t)p.box)) return -2;
    tas = ta;
    if (B_shared && !get_tmap_2d(&tas, A, (uint64_t)K_shared, (uint64_t)a_rows, (uint64_t)lda * 2, kGgK, (uint32_t)p.box)) return -2;
  }
  if (!get_tmap_2d(&tb, B, (uint64_t)N, (uint64_t)experts * K, (uint64_t)N * 2, 64, kGgK)) return -2;
  tbs = tb;
  if (B_shared && !get_tmap_2d(&tbs, B_shared, (uint64_t)N_shared, (uint64_t)K_shared, (uint64_t)N_shared * 2, 64, kGgK)) return -2;
  const int64_t most = (int64_t)p.sh_tiles * p.tn_shared + (int64_t)max_tiles * p.tn;
  const int grid = (int)(most < sms ? most : sms);
  if (grid <= 0) return 0;
  auto go = [&](auto type, auto width) -> int {
    using T = decltype(type);
    constexpr int BN = decltype(width)::value;
    if (src == nullptr) return launch_grouped<T, BN, kGgBoxes>(ta, tas, tb, tbs, p, grid, stream);
    return copy ? launch_grouped<T, BN, kGgCopy>(ta, tas, tb, tbs, p, grid, stream)
                : launch_grouped<T, BN, kGgGather4>(ta, tas, tb, tbs, p, grid, stream);
  };
  auto width = [&](auto type) -> int {
    if (bn == 256) return go(type, std::integral_constant<int, 256>{});
    if (bn == 128) return go(type, std::integral_constant<int, 128>{});
    return go(type, std::integral_constant<int, 64>{});
  };
  return dtype == 1 ? width(__nv_bfloat16{}) : width(__half{});
}

}  // extern "C"
