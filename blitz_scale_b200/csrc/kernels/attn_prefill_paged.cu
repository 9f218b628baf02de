// Causal prefill attention over the paged KV cache on tcgen05 for sm_100a: GQA, heads of up to 128, queries of
// the current chunk against everything the cache holds for the sequence (earlier chunks and the chunk itself).
//
// Q comes from the fused QKV activation of the chunk (2-D TMA boxes); K and V come from the paged pool, where
// rope_kv_store has already put the chunk's own keys and values, as 3-D TMA boxes of one page (or 64 tokens of
// one) each, looked up through the page table.  A prompt that does not fit one batch is therefore prefetched in
// chunks with no other kernel: the first chunk has an empty prefix, later ones a prefix of whole earlier chunks.
//
// A work item is 256 query rows of one sequence and one q head, as two tiles of 128 rows that walk the KV blocks
// of 128 tokens up to the diagonal once for both:
//
//   S_t = Q_t K^T      tcgen05.mma, A = Q_t (smem), B = K block (smem), S_t in TMEM                      t = 0, 1
//   P_t = softmax      warpgroup t (4 warps, thread = row): one tcgen05.ld pass over S_t, running max and sum in
//                      fp32, P_t written back over S_t's first 64 columns (two 16-bit values per column)
//   O_t += P_t V       tcgen05.mma with A = P_t from tensor memory, accumulating in TMEM over all blocks
//
// A ninth warp issues the MMAs (one thread), a tenth the TMA loads.  While warpgroup 0 turns S_0 into P_0 the
// tensor core works on S_1 and on O_1, and the other way round: the two tiles ping-pong, and every K and V block
// feeds two tiles from one load.  O stays in TMEM for the whole walk: the maximum a row's probabilities refer to
// only moves when the true maximum has grown by more than 2^8 (the probabilities then stay below 256, harmless in
// 16 bits and fp32), and only then the warp rescales its O rows in place (tcgen05.ld, multiply, tcgen05.st); with
// ordinary inputs that happens in the first block or two of a row and never again.
//
// The grid is persistent: one CTA per SM takes work items in a fixed order (heaviest first, dealt back and forth
// over the CTAs so that every CTA gets a similar sum).  The three roles walk the same list on their own, all
// barrier phases come from running counts, and nothing is drained between items: the next item's Q, K and V are
// loaded and its first S products issued while the warpgroups still write the previous item's output, so the
// latency of starting an item (its page ids, its first loads, the first MMA) is paid once per CTA, not per item.
//
// Models that ask for it (template parameter EXT) get a sliding window with kept first tokens, soft-capped scores and a
// per-head sink.  The two tiles of an item then walk the key blocks of the kept tokens and those from the first row's
// window edge on; blocks in between are never loaded.  A block that is wholly visible to a tile needs no mask.  The cap,
// cap * tanh(s / cap), is applied to the scores as they turn into probabilities.  Where all of a warp's scores of the
// block stay below half the cap (one vote per block, the usual case), that is an odd polynomial on the FMA pipe, two
// scores per instruction, and the largest magnitude serves as the row's reference instead of its maximum, so that one
// pass over the scores decides both; else the special-function unit does it (tanh being monotonic, the row maximum is
// capped alone).  The sink is one more term of the row sum at the end.
//
// Keys and values may differ in size, and either may be smaller than the tile it is computed in (64 or 128 columns, a
// multiple of 8): TMA fills the columns behind a head's end with zeros.  A gate (one number per head and row, through a
// sigmoid) multiplies a head's output rows as they leave tensor memory.
//
// A bias by distance per head (template parameter BIAS): bias[h][min(i - j, bias_len - 1)] is added to the scaled scores.  A
// block of 128 keys against a tile of 128 rows has 255 distances; the tile's warpgroup fetches their biases (two a thread,
// requested before it waits for the scores) into shared memory, where the lanes of a warp, rows that follow one another, read
// neighbouring words.  Blocks whose every distance is beyond the table share its last entry, which moves the reference.
//
// The window may be a chunk counted from position 0 (`chunked`): a row sees the keys of its own chunk.  Weights may be sigmoids of
// the scores (template parameter SIG; EXT with it): no maximum, no row sum, no rescaling.  sigmoid(x) = 1 / (1 + e^-x); four
// neighbours share a reciprocal, 1 / a = b (c d) / (a b c d), unless a product of some four leaves the range of fp32 (one vote per
// half a block).
//
// Replaces FlashInfer's BatchPrefillWithRaggedKVCacheWrapper / paged wrapper calls and their host Plan()
// (src/kernel/attention_prefill.cu:11-45, src/kernel/flashinfer_types.cu:24-49).
#include "launch.cuh"
#include "ptx.cuh"
#include "tmap.cuh"
#include "common.cuh"
#include <cmath>

namespace blitz {

constexpr int kPpThreads = 320;  // warpgroup 0, warpgroup 1, MMA warp, load warp
constexpr int kPpTile = 128;     // q rows per tile and kv tokens per block
constexpr float kPpRescaleAt = 8.f;  // log2 units
constexpr int kPpWorkInts = 8;   // per (sequence, pair of tiles): first row, rows, first page entry, pages, cached tokens, pair

struct PagedPrefillParams {
  void* out;  // [tokens, q_heads * vdim]
  const void* gate;  // [tokens][gate_stride], a column per query head, or null
  int64_t out_stride, gate_stride;
  const int32_t* page_indices;  // page ids of every sequence, back to back
  const int32_t* work;          // [entries][kPpWorkInts], heaviest first
  int entries, q_heads, kv_heads, vdim, page_size, page_rows, box_tokens, oob_row;  // page n's token `off`: pool row n * page_rows + off
  float scale_log2;
  int chunked;                // EXT: the window is a chunk
  int window, keep_first;     // EXT: a row sees the last `window` positions (0: all) and the first `keep_first`
  float cap_scale, cap_log2;  // EXT: soft cap (cap_log2 > 0): score in log2 units = cap_log2 * tanh(q.k * cap_scale)
  float small_max;            // EXT: largest |q.k| the polynomial takes (0: never)
  float poly[4];              // EXT: score in log2 units = x (poly[0] + poly[1] x^2 + poly[2] x^4 + poly[3] x^6), x = q.k
  const void* sink;           // EXT: [q_heads] in the activation type, or null
  const void* bias;           // BIAS: [q_heads][bias_len] in the activation type (SIG: [q_heads], or null)
  int bias_len;
  int* status;
  long long* trace;  // profiling aid (null in production): clock stamps of CTA 0's first item, see the set_trace call
};

constexpr int kPpTraceIters = 32, kPpTraceSlots = 8;
// role 0 / 1: first lane of warpgroup 0 / 1; role 2: the MMA thread
__device__ __forceinline__ void pp_trace(const PagedPrefillParams& p, bool on, int role, int j, int slot) {
  if (on && p.trace != nullptr && j < kPpTraceIters) p.trace[(role * kPpTraceIters + j) * kPpTraceSlots + slot] = clock64();
}

template <int HD, int VD>
struct PpCfg {
  static constexpr int kSlabBytes = kPpTile * 128;     // 64 columns of a tile: 128 rows x 128 bytes
  static constexpr int kSlabs = HD / 64, kValueSlabs = VD / 64;
  static constexpr int kTileBytes = kSlabs * kSlabBytes, kValueBytes = kValueSlabs * kSlabBytes;  // a Q or K tile, a V tile
  static constexpr int kBarBytes = 256;
  static constexpr int kBiasFloats = 2 * 2 * 256;  // per tile: two blocks' distances
  static constexpr int kSmemBytes = 4 * kTileBytes + 2 * kValueBytes + 1024 + kBarBytes;  // Q x 2 tiles, K x 2 stages, V x 2 stages
};

struct PpItem {
  int seq_start, q_len, pg0, npages, kv_len, prefix, q0, nt, nblk, head, kv_head;
  int nblk_t[2];
  int n_first, b_window;  // key blocks walked: [0, n_first), then from b_window on
  __device__ __forceinline__ int block(int j) const { return j < n_first ? j : b_window + j - n_first; }
};
// Work item `idx` of the flattened list (entry x q head; the heads of one entry are neighbours, so CTAs that run
// at the same time share its K and V in L2).
template <bool EXT>
__device__ __forceinline__ PpItem pp_item(const PagedPrefillParams& p, int idx) {
  PpItem it;
  const int entry = idx / p.q_heads;
  it.head = idx - entry * p.q_heads;
  it.kv_head = it.head / (p.q_heads / p.kv_heads);
  const int4 a = __ldg(reinterpret_cast<const int4*>(p.work + entry * kPpWorkInts));
  const int4 b = __ldg(reinterpret_cast<const int4*>(p.work + entry * kPpWorkInts + 4));
  it.seq_start = a.x; it.q_len = a.y; it.pg0 = a.z; it.npages = a.w; it.kv_len = b.x;
  it.prefix = it.kv_len - it.q_len;  // tokens of earlier chunks
  it.q0 = b.y * 2 * kPpTile;
  it.nt = (it.q0 + kPpTile < it.q_len) ? 2 : 1;
#pragma unroll
  for (int t = 0; t < 2; ++t) {  // blocks tile t needs: keys up to its last row's position
    const int last = min(it.kv_len, it.prefix + min(it.q_len, it.q0 + kPpTile * (t + 1)));
    it.nblk_t[t] = t < it.nt ? (last + kPpTile - 1) / kPpTile : 0;
  }
  it.n_first = it.b_window = 0;
  if (EXT && p.window > 0) {
    const int p0 = it.prefix + it.q0, lo = p.chunked ? p0 - p0 % p.window : max(0, p0 - p.window + 1);  // first key in the window of the item's first row
    it.n_first = (min(p.keep_first, lo) + kPpTile - 1) / kPpTile;
    it.b_window = max(lo / kPpTile, it.n_first);
#pragma unroll
    for (int t = 0; t < 2; ++t)
      if (it.nblk_t[t] > 0) it.nblk_t[t] = it.n_first + max(0, it.nblk_t[t] - it.b_window);
  }
  it.nblk = max(it.nblk_t[0], it.nblk_t[1]);
  return it;
}
// The r-th item of this CTA: rounds alternate direction over the CTAs.  -1: this CTA has none in round r.
__device__ __forceinline__ int pp_index(int r, int total) {
  const int G = gridDim.x;
  const int idx = r * G + ((r & 1) ? G - 1 - static_cast<int>(blockIdx.x) : static_cast<int>(blockIdx.x));
  return idx < total ? idx : -1;
}

template <typename T, int HD, int VD, bool POLY, bool EXT, bool BIAS, bool SIG>
__global__ void __launch_bounds__(kPpThreads, 1)
attn_prefill_paged_kernel(const __grid_constant__ CUtensorMap tmap_q, const __grid_constant__ CUtensorMap tmap_k,
                          const __grid_constant__ CUtensorMap tmap_v, const PagedPrefillParams p) {
  using C = PpCfg<HD, VD>;
  constexpr int TB = C::kTileBytes, VB = C::kValueBytes, SB = C::kSlabBytes;
  constexpr uint32_t kFmt = std::is_same<T, __nv_bfloat16>::value ? 1u : 0u;
  constexpr uint32_t kIdescS = ptx::make_idesc_f16(kFmt, 0u, 0u, 128, 128);
  constexpr uint32_t kIdescPV = ptx::make_idesc_f16(kFmt, 0u, 1u, 128, VD);

  extern __shared__ uint8_t smem_raw[];
  const uint32_t raw_addr = ptx::smem_u32(smem_raw);
  uint8_t* smem = smem_raw + (((raw_addr + 1023u) & ~1023u) - raw_addr);
  uint8_t* sQ = smem;            // [2 tiles]
  uint8_t* sK = sQ + 2 * TB;     // [2 stages]
  uint8_t* sV = sK + 2 * TB;     // [2 stages]
  uint64_t* bars = reinterpret_cast<uint64_t*>(sV + 2 * VB);
  uint64_t* q_full = bars;        // once per item
  uint64_t* q_empty = bars + 1;   // once per item: its last S products are done
  uint64_t* k_full = bars + 2;    // [2] per block
  uint64_t* k_empty = bars + 4;   // [2]
  uint64_t* v_full = bars + 6;    // [2]
  uint64_t* v_empty = bars + 8;   // [2]
  uint64_t* s_full = bars + 10;   // [2] per tile and block
  uint64_t* p_ready = bars + 12;  // [2]
  uint64_t* o_full = bars + 14;   // [2]
  uint64_t* o_free = bars + 16;   // [2] per tile and item: the warpgroup has read its output rows
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 18);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  float* s_bias = reinterpret_cast<float*>(sV + 2 * VB + C::kBarBytes);  // BIAS only

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int total = p.entries * p.q_heads;

  if (threadIdx.x == 0) {
    ptx::mbar_init(q_full, 1);
    ptx::mbar_init(q_empty, 1);
    for (int i = 0; i < 2; ++i) {
      ptx::mbar_init(&k_full[i], 1);
      ptx::mbar_init(&k_empty[i], 1);
      ptx::mbar_init(&v_full[i], 1);
      ptx::mbar_init(&v_empty[i], 1);
      ptx::mbar_init(&s_full[i], 1);
      ptx::mbar_init(&p_ready[i], 128);
      ptx::mbar_init(&o_full[i], 1);
      ptx::mbar_init(&o_free[i], 128);
    }
    *abort_flag = 0;
    ptx::fence_mbar_init();
    ptx::tma_prefetch_desc(&tmap_q);
    ptx::tma_prefetch_desc(&tmap_k);
    ptx::tma_prefetch_desc(&tmap_v);
  }
  if (warp == 8) {
    ptx::tmem_alloc(tmem_slot, 512);
    ptx::tmem_relinquish();
  }
  ptx::tc_fence_before_sync();
  __syncthreads();
  ptx::tc_fence_after_sync();
  const uint32_t tmem_base = *tmem_slot;
  const uint32_t tmem_S = tmem_base;        // S_t (and P_t over its first 64 columns) at + 128 t
  const uint32_t tmem_O = tmem_base + 256;  // O_t at + VD t

  if (warp == 9) {
    // ------------------------------------------------------------ load warp: Q, then K and V block by block
    // K or V block j -> one tile of 128 token rows: every lane fetches one box (a page, or 64 tokens of one)
    const int bt = p.box_tokens;
    const bool mine = lane < kPpTile / bt;
    auto box_row = [&](const PpItem& it, int j) {  // this lane's first row of block j in the pools
      const int tok = it.block(j) * kPpTile + lane * bt;
      const int slot = tok / p.page_size;
      if (!mine || slot >= it.npages) return p.oob_row;  // past the pool: the box arrives as zeros
      return p.page_indices[it.pg0 + slot] * p.page_rows + (tok & (p.page_size - 1));
    };
    auto load_kv = [&](uint8_t* dst, const CUtensorMap* map, int slabs, uint64_t* bar, int kv_head, int row) {
      if (lane == 0) ptx::mbar_expect_tx(bar, slabs * SB);
      __syncwarp();
      if (mine) {
#pragma unroll
        for (int s = 0; s < slabs; ++s) ptx::tma_load_3d(dst + s * SB + lane * bt * 128, map, bar, s * 64, kv_head, row);
      }
    };
    auto wait = [&](uint64_t* bar, uint32_t parity) {
      int ok = 1;
      if (lane == 0) ok = ptx::bounded_mbar_wait(bar, parity, abort_flag) ? 1 : 0;
      return __shfl_sync(0xffffffffu, ok, 0) != 0;
    };
    bool ok = true;
    uint32_t g = 0, n_items = 0;  // blocks and items loaded so far
    for (int r = 0; r * static_cast<int>(gridDim.x) < total && ok; ++r) {
      const int idx = pp_index(r, total);
      if (idx < 0) continue;
      const PpItem it = pp_item<EXT>(p, idx);
      if (n_items > 0) ok = wait(q_empty, (n_items - 1) & 1);  // the previous item's S products have read Q
      if (!ok) break;
      if (lane == 0) {
        ptx::mbar_expect_tx(q_full, it.nt * TB);
        for (int t = 0; t < it.nt; ++t)
#pragma unroll
          for (int s = 0; s < C::kSlabs; ++s)
            ptx::tma_load_3d(sQ + t * TB + s * SB, &tmap_q, q_full, s * 64, it.head, it.seq_start + it.q0 + t * kPpTile);
      }
      int row = box_row(it, 0);
      for (int j = 0; j < it.nblk && ok; ++j, ++g) {
        const int row_next = j + 1 < it.nblk ? box_row(it, j + 1) : p.oob_row;  // looked up a block ahead of its use
        // a block's K goes where the K of two blocks ago was, once the S products of that block are done; V likewise
        if (g >= 2) ok = wait(&k_empty[g & 1], ((g - 2) >> 1) & 1);
        if (!ok) break;
        load_kv(sK + (g & 1) * TB, &tmap_k, C::kSlabs, &k_full[g & 1], it.kv_head, row);
        if (g >= 2) ok = wait(&v_empty[g & 1], ((g - 2) >> 1) & 1);
        if (!ok) break;
        load_kv(sV + (g & 1) * VB, &tmap_v, C::kValueSlabs, &v_full[g & 1], it.kv_head, row);
        row = row_next;
      }
      ++n_items;
    }
    if (!ok && lane == 0 && p.status) atomicCAS(p.status, 0, kStatusTimeoutProducer);
  } else if (warp == 8) {
    // ------------------------------------------------------------ MMA warp: one thread issues
    if (lane == 0) {
      auto issue_S = [&](int t, int stage) {
        const uint32_t a = ptx::smem_u32(sQ + t * TB), bb = ptx::smem_u32(sK + stage * TB);
#pragma unroll
        for (int k = 0; k < HD / 16; ++k) {
          const uint32_t off = (k >> 2) * SB + (k & 3) * 32;
          ptx::umma_f16_ss(tmem_S + t * 128, ptx::make_smem_desc(a + off, 16, 1024, ptx::kLayoutSw128),
                           ptx::make_smem_desc(bb + off, 16, 1024, ptx::kLayoutSw128), kIdescS, k != 0 ? 1u : 0u);
        }
        ptx::umma_commit(&s_full[t]);
      };
      auto issue_PV = [&](int t, int stage, bool accumulate) {
        const uint32_t bb = ptx::smem_u32(sV + stage * VB);
#pragma unroll
        for (int k = 0; k < kPpTile / 16; ++k) {
          // A = P in tensor memory: row = lane, 16 tokens = 8 columns.  B = V: N-major, slabs of 64 head-dim
          // columns; 16 tokens (K) advance 2 KB.
          ptx::umma_f16_ts(tmem_O + t * VD, tmem_S + t * 128 + k * 8,
                           ptx::make_smem_desc(bb + k * 2048, SB, 1024, ptx::kLayoutSw128), kIdescPV,
                           (accumulate || k != 0) ? 1u : 0u);
        }
        ptx::umma_commit(&o_full[t]);
      };
      auto wait = [&](uint64_t* bar, uint32_t parity) { return ptx::bounded_mbar_wait(bar, parity, abort_flag); };
      // Everything this thread touches between two MMAs stays in registers (no arrays indexed by the tile number):
      // it is the one thread the tensor pipe waits for.
      bool ok = true;
      uint32_t g = 0, n_items = 0;   // blocks and items started so far
      uint32_t cnt0 = 0, cnt1 = 0;   // blocks tile t has been through
      uint32_t outs0 = 0, outs1 = 0; // items tile t has produced output for
      for (int r = 0; r * static_cast<int>(gridDim.x) < total && ok; ++r) {
        const int idx = pp_index(r, total);
        if (idx < 0) continue;
        const PpItem it = pp_item<EXT>(p, idx);
        const int nb0 = it.nblk_t[0], nb1 = it.nblk_t[1], nblk = it.nblk;
        const bool tr = n_items == 0 && blockIdx.x == 0;
        ok = wait(q_full, n_items & 1) && wait(&k_full[g & 1], (g >> 1) & 1);
        if (!ok) break;
        ptx::tc_fence_after_sync();
        // S of the first block: the tiles' score columns are free (their last P of the previous item was waited for)
        issue_S(0, g & 1);
        if (nb1 > 0) issue_S(1, g & 1);
        ptx::umma_commit(&k_empty[g & 1]);
        if (nblk == 1) ptx::umma_commit(q_empty);
        for (int j = 0; j < nblk && ok; ++j) {
          const uint32_t gj = g + j;
          pp_trace(p, tr, 2, j, 0);
          bool v_here = false, k_next = false;
          // one tile's turn: wait for its P, then its P V and its next S
          auto turn = [&](const int t, const int nbt, const uint32_t cnt_t, const uint32_t outs_t) {
            if (j >= nbt || !ok) return;
            ok = wait(&p_ready[t], (cnt_t + j) & 1);  // P_t of block j is written; S_t and (after a rescale) O_t are settled
            pp_trace(p, tr, 2, j, 2 + 2 * t);
            if (ok && !v_here) {
              ok = wait(&v_full[gj & 1], (gj >> 1) & 1);
              v_here = true;
            }
            if (ok && j + 1 < nbt && !k_next) {
              ok = wait(&k_full[(gj + 1) & 1], ((gj + 1) >> 1) & 1);
              k_next = true;
            }
            // the first product of an item overwrites O_t: the warpgroup must have read the previous item's rows
            if (ok && j == 0 && outs_t > 0) ok = wait(&o_free[t], (outs_t - 1) & 1);
            if (!ok) return;
            ptx::tc_fence_after_sync();
            issue_PV(t, gj & 1, j > 0);
            if (j + 1 < nbt) issue_S(t, (gj + 1) & 1);
            pp_trace(p, tr, 2, j, 3 + 2 * t);
          };
          turn(0, nb0, cnt0, outs0);
          turn(1, nb1, cnt1, outs1);
          if (!ok) break;
          if (k_next) ptx::umma_commit(&k_empty[(gj + 1) & 1]);
          ptx::umma_commit(&v_empty[gj & 1]);
          if (j + 2 == nblk) ptx::umma_commit(q_empty);  // the S products of the last block have just been issued
        }
        cnt0 += nb0;
        cnt1 += nb1;
        outs0 += 1;
        outs1 += nb1 > 0 ? 1 : 0;
        g += nblk;
        ++n_items;
      }
      if (!ok && p.status) atomicCAS(p.status, 0, kStatusTimeoutMma);
    }
  } else {
    // ------------------------------------------------------------ softmax warpgroups (thread = query row)
    const int t = warp >> 2;
    const int r_ = (warp & 3) * 32 + lane;
    const uint32_t lane_addr = static_cast<uint32_t>((warp & 3) * 32) << 16;
    const uint32_t tS = tmem_S + t * 128 + lane_addr;
    const uint32_t tO = tmem_O + t * VD + lane_addr;
    bool ok = true;
    uint32_t cnt = 0;  // blocks this tile has been through
    bool first = true;
    for (int r = 0; r * static_cast<int>(gridDim.x) < total && ok; ++r) {
      const int idx = pp_index(r, total);
      if (idx < 0) continue;
      const PpItem it = pp_item<EXT>(p, idx);
      const int my_blocks = it.nblk_t[t];
      if (my_blocks == 0) continue;  // a short last pair has no second tile
      const bool tracer = first && blockIdx.x == 0 && (warp & 3) == 0 && lane == 0;
      first = false;
      const int q_idx = it.q0 + t * kPpTile + r_;  // row within the chunk
      const int limit = it.prefix + q_idx;         // last key position this row may see
      const int chunk_from = EXT && p.chunked ? limit - limit % p.window : -1;  // first key of the row's chunk
      float m_ref = 0.f, l = 0.f;
      const float sig_bias = SIG && p.bias ? -1.4426950408889634f * to_f<T>(reinterpret_cast<const T*>(p.bias)[it.head]) : 0.f;
      const T* bias_row = BIAS ? reinterpret_cast<const T*>(p.bias) + static_cast<int64_t>(it.head) * p.bias_len : nullptr;
      const float far_bias = BIAS ? to_f<T>(bias_row[p.bias_len - 1]) * 1.4426950408889634f : 0.f;
      for (int j = 0; j < my_blocks; ++j) {
        pp_trace(p, tracer, t, j, 0);
        // the block's smallest distance; is any of them inside the table?
        const int nearest = it.prefix + it.q0 + t * kPpTile - (it.block(j) * kPpTile + kPpTile - 1);
        const bool near = BIAS && nearest < p.bias_len - 1;
        float bias_pair[2];
        if (near) {
#pragma unroll
          for (int k = 0; k < 2; ++k)
            bias_pair[k] = to_f<T>(bias_row[min(max(nearest + r_ + k * kPpTile, 0), p.bias_len - 1)]) * 1.4426950408889634f;
        }
        if (!ptx::bounded_mbar_wait(&s_full[t], (cnt + j) & 1, abort_flag)) {
          ok = false;
          break;
        }
        pp_trace(p, tracer, t, j, 1);
        ptx::tc_fence_after_sync();
        if constexpr (SIG) {
          const int kv0 = it.block(j) * kPpTile, row0 = it.prefix + it.q0 + t * kPpTile;
          // the block's visible keys, of this row and of all rows of the tile
          const int from = p.window > 0 ? chunk_from >= 0 ? chunk_from : limit - p.window + 1 : 0;
          const int lo = from - kv0, hi = limit - kv0, last = row0 + kPpTile - 1;
          const bool early = p.window > 0 && kv0 < (p.chunked ? last / p.window * p.window : last - p.window + 1);  // keys before some row's first
          const bool masked = kv0 + kPpTile - 1 > row0 || early;
          const uint64_t scale2 = ptx::f32x2(-p.scale_log2, -p.scale_log2), bias2 = ptx::f32x2(sig_bias, sig_bias),
                         one2 = ptx::f32x2(1.f, 1.f);
          auto weights = [&](auto&& hidden) {
#pragma unroll
            for (int h = 0; h < 2; ++h) {  // 64 scores -> 32 columns of pairs
              uint32_t v[2][32], pk[32];
              ptx::tmem_ld_32x32(tS + h * 64, v[0]);
              ptx::tmem_ld_32x32(tS + h * 64 + 32, v[1]);
              ptx::tmem_ld_wait();
              // 1 + e^-x of scores c and c + 1
              auto denominators = [&](int c) {
                const int k = c - h * 64;
                const float2 x = ptx::f32x2_get(
                    ptx::fma_f32x2(ptx::f32x2(__uint_as_float(v[k >> 5][k & 31]), __uint_as_float(v[k >> 5][(k & 31) + 1])), scale2, bias2));
                return ptx::fma_f32x2(ptx::f32x2(ptx::ex2_approx(x.x), ptx::ex2_approx(x.y)), one2, one2);
              };
              float smallest = 1.f;
#pragma unroll
              for (int i = 0; i < 32; i += 2) {
                const int c = h * 64 + 2 * i;
                const uint64_t ab = denominators(c), cd = denominators(c + 2);
                const float2 f = ptx::f32x2_get(ab), g = ptx::f32x2_get(cd);
                const float fp = f.x * f.y, gp = g.x * g.y, r = ptx::rcp_approx(fp * gp);
                smallest = fminf(smallest, r);
                const float rf = r * gp, rg = r * fp;
                const float2 w = ptx::f32x2_get(ptx::mul_f32x2(ptx::f32x2(f.y, f.x), ptx::f32x2(rf, rf)));
                const float2 z = ptx::f32x2_get(ptx::mul_f32x2(ptx::f32x2(g.y, g.x), ptx::f32x2(rg, rg)));
                pk[i] = pk2<T>(hidden(c) ? 0.f : w.x, hidden(c + 1) ? 0.f : w.y);
                pk[i + 1] = pk2<T>(hidden(c + 2) ? 0.f : z.x, hidden(c + 3) ? 0.f : z.y);
              }
              if (__any_sync(0xffffffffu, !(smallest > 1e-36f))) {  // a product left the range: one reciprocal each
#pragma unroll
                for (int i = 0; i < 32; ++i) {
                  const int c = h * 64 + 2 * i;
                  const float2 d = ptx::f32x2_get(denominators(c));
                  pk[i] = pk2<T>(hidden(c) ? 0.f : ptx::rcp_approx(d.x), hidden(c + 1) ? 0.f : ptx::rcp_approx(d.y));
                }
              }
              ptx::tmem_st_32x32(tS + h * 32, pk);
            }
          };
          if (!masked) weights([](int) { return false; });
          else if (!early) weights([&](int i) { return i > hi; });
          else weights([&](int i) { return i > hi || i < lo; });
          ptx::tmem_st_wait();
          ptx::tc_fence_before_sync();
          ptx::mbar_arrive(&p_ready[t]);
          l = 1.f;
          continue;
        }
        uint32_t v0[32], v1[32], v2[32], v3[32];  // the row's 128 scores (fp32 bits)
        ptx::tmem_ld_32x32(tS, v0);
        ptx::tmem_ld_32x32(tS + 32, v1);
        ptx::tmem_ld_32x32(tS + 64, v2);
        ptx::tmem_ld_32x32(tS + 96, v3);
        ptx::tmem_ld_wait();
        pp_trace(p, tracer, t, j, 2);
        auto score = [&](int i) -> uint32_t& { return i < 32 ? v0[i] : i < 64 ? v1[i - 32] : i < 96 ? v2[i - 64] : v3[i - 96]; };
        const int kv0 = it.block(j) * kPpTile;
        const int row0 = it.prefix + it.q0 + t * kPpTile;  // position of the tile's first row
        // does the block hold a key that some row of the tile may not see?
        bool masked = kv0 + kPpTile - 1 > row0;
        if (EXT && p.window > 0)
          masked = masked || (p.chunked ? kv0 < (row0 + kPpTile - 1) / p.window * p.window
                                        : kv0 <= row0 + kPpTile - 1 - p.window && kv0 + kPpTile > p.keep_first);
        const int from = (EXT && p.window > 0) ? chunk_from >= 0 ? chunk_from : limit - p.window + 1 : 0;
        auto visible = [&](int i) {  // key i of the block to this row
          return kv0 + i <= limit && (!EXT || kv0 + i >= from || kv0 + i < p.keep_first);
        };
        const bool capped = EXT && p.cap_log2 > 0.f;
        float bias = 0.f;  // of every score of the block, in log2 units
        if (near) {
          float* sb = s_bias + (t * 2 + (j & 1)) * 256;  // (the buffer of two blocks ago: every warp has passed the last barrier)
          sb[r_] = bias_pair[0];
          sb[r_ + kPpTile] = bias_pair[1];
          if (t == 0) asm volatile("bar.sync 1, 128;" ::: "memory");
          else asm volatile("bar.sync 2, 128;" ::: "memory");
          // distance of key i to this row: nearest + r_ + 127 - i
#pragma unroll
          for (int i = 0; i < kPpTile; ++i)
            score(i) = __float_as_uint(fmaf(__uint_as_float(score(i)), p.scale_log2, sb[r_ + kPpTile - 1 - i]));
        } else if (BIAS) {
          bias = far_bias;
        }
        const float score_scale = near ? 1.f : p.scale_log2;
        // largest of the row's 128 scores, or of their magnitudes: eight independent chains of three-input maxima (with two
        // softmax warps per scheduler nothing else hides a serial one)
        auto largest = [&](auto&& max3) {
          float mxs[8];
#pragma unroll
          for (int i = 0; i < 8; ++i) mxs[i] = __uint_as_float(score(i));
#pragma unroll
          for (int i = 8; i < kPpTile - 8; i += 16)
#pragma unroll
            for (int k = 0; k < 8; ++k)
              mxs[k] = max3(mxs[k], __uint_as_float(score(i + 2 * k)), __uint_as_float(score(i + 2 * k + 1)));
#pragma unroll
          for (int i = kPpTile - 8; i < kPpTile; ++i) mxs[i & 7] = max3(mxs[i & 7], __uint_as_float(score(i)), __uint_as_float(score(i)));
          const float mx = fmaxf(max3(mxs[0], mxs[1], mxs[2]), max3(mxs[3], mxs[4], mxs[5]));
          return max3(mx, mxs[6], mxs[7]);
        };
        float mx = 0.f;
        bool small = false;
        if (capped && std::is_same<T, __nv_bfloat16>::value) {  // (fp16 probabilities need the maximum itself)
          mx = largest([](float a, float b, float c) { return ptx::fmax3_abs(a, b, c); });
          small = __all_sync(0xffffffffu, mx <= p.small_max);
        }
        if (small) {
          mx *= p.scale_log2;  // |cap tanh(x / cap)| <= |x|
        } else {
          if (masked) {
#pragma unroll
            for (int i = 0; i < kPpTile; ++i)
              if (!visible(i)) score(i) = 0xff800000u;  // -inf
          }
          mx = largest([](float a, float b, float c) { return ptx::fmax3(a, b, c); });
          if (capped) mx = mx == -INFINITY ? mx : p.cap_log2 * ptx::tanh_ex2(mx * p.cap_scale);
          else mx = BIAS ? fmaf(mx, score_scale, bias) : mx * p.scale_log2;
        }
        // (S of this block was issued after P V of the previous one, so that product is complete: O_t is stable and
        // the columns P is about to overwrite have been read)
        if (j == 0) {
          m_ref = (!EXT && mx == -INFINITY) ? 0.f : mx;  // EXT: a row may see nothing of its first blocks
        } else {
          const bool grow = mx > m_ref + kPpRescaleAt;
          if (__any_sync(0xffffffffu, grow)) {
            const float alpha = grow ? ptx::ex2_approx(m_ref - mx) : 1.f;
#pragma unroll 1
            for (int c = 0; c < VD; c += 32) {
              uint32_t o[32];
              ptx::tmem_ld_32x32(tO + c, o);
              ptx::tmem_ld_wait();
#pragma unroll
              for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * alpha);
              ptx::tmem_st_32x32(tO + c, o);
            }
            ptx::tmem_st_wait();
            l *= alpha;
            if (grow) m_ref = mx;
          }
        }
        pp_trace(p, tracer, t, j, 3);
        // probabilities (16 bit) -> tensor memory over the scores; row sum
        float rs[4] = {0.f, 0.f, 0.f, 0.f};
        const float neg_m = ((EXT && m_ref == -INFINITY) ? 0.f : -m_ref) + (BIAS ? bias : 0.f);
        auto probabilities = [&](auto&& exponents) {  // exponents(c): those of scores c and c + 1
#pragma unroll
          for (int h = 0; h < 2; ++h) {  // 64 scores -> 32 columns of pairs
            uint32_t pk[32];
#pragma unroll
            for (int i = 0; i < 32; ++i) {
              const float2 x = exponents(h * 64 + 2 * i);
              const float e0 = ptx::ex2_approx(x.x);
              const float e1 = (POLY && (i & 1)) ? ptx::ex2_poly(x.y) : ptx::ex2_approx(x.y);
              rs[i & 3] += e0 + e1;
              pk[i] = pk2<T>(e0, e1);
            }
            ptx::tmem_st_32x32(tS + h * 32, pk);
          }
        };
        if (EXT && small) {
          const uint64_t c0 = ptx::f32x2(p.poly[0], p.poly[0]), c1 = ptx::f32x2(p.poly[1], p.poly[1]),
                         c2 = ptx::f32x2(p.poly[2], p.poly[2]), c3 = ptx::f32x2(p.poly[3], p.poly[3]), nm = ptx::f32x2(neg_m, neg_m);
          auto poly = [&](int c) {
            const uint64_t x = ptx::f32x2(__uint_as_float(score(c)), __uint_as_float(score(c + 1)));
            const uint64_t y = ptx::mul_f32x2(x, x);
            uint64_t r = ptx::fma_f32x2(c3, y, c2);
            r = ptx::fma_f32x2(r, y, c1);
            r = ptx::fma_f32x2(r, y, c0);
            return ptx::f32x2_get(ptx::fma_f32x2(x, r, nm));
          };
          if (masked) {
            probabilities([&](int c) {
              float2 e = poly(c);
              if (!visible(c)) e.x = -INFINITY;
              if (!visible(c + 1)) e.y = -INFINITY;
              return e;
            });
          } else {
            probabilities(poly);
          }
        } else if (capped) {
          auto cap = [&](float x) { return x == -INFINITY ? x : fmaf(ptx::tanh_ex2(x * p.cap_scale), p.cap_log2, neg_m); };
          probabilities([&](int c) { return make_float2(cap(__uint_as_float(score(c))), cap(__uint_as_float(score(c + 1)))); });
        } else {
          probabilities([&](int c) {
            return make_float2(fmaf(__uint_as_float(score(c)), BIAS ? score_scale : p.scale_log2, neg_m),
                               fmaf(__uint_as_float(score(c + 1)), BIAS ? score_scale : p.scale_log2, neg_m));
          });
        }
        pp_trace(p, tracer, t, j, 4);
        ptx::tmem_st_wait();
        l += (rs[0] + rs[1]) + (rs[2] + rs[3]);
        ptx::tc_fence_before_sync();
        ptx::mbar_arrive(&p_ready[t]);
        pp_trace(p, tracer, t, j, 5);
      }
      if (ok) ok = ptx::bounded_mbar_wait(&o_full[t], (cnt + my_blocks - 1) & 1, abort_flag);
      if (!ok) break;
      cnt += my_blocks;
      ptx::tc_fence_after_sync();
      if (EXT && p.sink != nullptr && l > 0.f)
        l += ptx::ex2_approx(to_f<T>(reinterpret_cast<const T*>(p.sink)[it.head]) * 1.4426950408889634f - m_ref);
      float inv = l > 0.f ? 1.f / l : 0.f;
      if (p.gate != nullptr && q_idx < it.q_len) {
        const T z = reinterpret_cast<const T*>(p.gate)[static_cast<int64_t>(it.seq_start + q_idx) * p.gate_stride + it.head];
        inv /= 1.f + expf(-to_f<T>(z));
      }
      T* dst = reinterpret_cast<T*>(p.out) + static_cast<int64_t>(it.seq_start + q_idx) * p.out_stride + it.head * p.vdim;
#pragma unroll 1
      for (int c = 0; c < VD; c += 32) {
        uint32_t o[32];
        ptx::tmem_ld_32x32(tO + c, o);
        ptx::tmem_ld_wait();
        if (c + 32 >= VD) {  // all of this item's output rows are in registers: the next item may overwrite them
          ptx::tc_fence_before_sync();
          ptx::mbar_arrive(&o_free[t]);
        }
        if (q_idx < it.q_len) {
#pragma unroll
          for (int i = 0; i < 32; i += 8) {
            if (c + i < p.vdim) *reinterpret_cast<uint4*>(dst + c + i) = make_uint4(
                pk2<T>(__uint_as_float(o[i]) * inv, __uint_as_float(o[i + 1]) * inv),
                pk2<T>(__uint_as_float(o[i + 2]) * inv, __uint_as_float(o[i + 3]) * inv),
                pk2<T>(__uint_as_float(o[i + 4]) * inv, __uint_as_float(o[i + 5]) * inv),
                pk2<T>(__uint_as_float(o[i + 6]) * inv, __uint_as_float(o[i + 7]) * inv));
          }
        }
      }
    }
    if (!ok && p.status && lane == 0) atomicCAS(p.status, 0, kStatusTimeoutEpilogue);
  }

  ptx::tc_fence_before_sync();
  __syncthreads();
  if (warp == 8) {
    ptx::tc_fence_after_sync();
    ptx::tmem_dealloc(tmem_base, 512);
  }
}

template <typename T, int HD, int VD, bool POLY, bool EXT, bool BIAS, bool SIG>
static int launch_paged_prefill(const CUtensorMap (&tm)[3], const PagedPrefillParams& p, int grid, cudaStream_t stream) {
  constexpr int kSmem = PpCfg<HD, VD>::kSmemBytes + (BIAS ? PpCfg<HD, VD>::kBiasFloats * 4 : 0);
  static PerDeviceOnce once;
  cudaError_t e = once.run([] {
    return cudaFuncSetAttribute(attn_prefill_paged_kernel<T, HD, VD, POLY, EXT, BIAS, SIG>, cudaFuncAttributeMaxDynamicSharedMemorySize, kSmem);
  });
  if (e != cudaSuccess) return (int)e;
  attn_prefill_paged_kernel<T, HD, VD, POLY, EXT, BIAS, SIG><<<grid, kPpThreads, kSmem, stream>>>(tm[0], tm[1], tm[2], p);
  return (int)cudaGetLastError();
}

static long long* g_pp_trace = nullptr;

}  // namespace blitz

extern "C" {
using namespace blitz;

// Profiling aid: while `buf` (3 roles x 32 iterations x 8 int64 clock stamps, device memory) is set, CTA 0 of every
// following launch records when its warpgroups and its MMA thread pass each phase of its first work item.
void blitz_attn_prefill_paged_set_trace(long long* buf) { blitz::g_pp_trace = buf; }

// q: [num_tokens, q_stride >= q_heads * dim] of the current chunk, rotated; k_pool, v_pool: the layer's pools
// [max_pages][page_rows][kv_heads][dim or vdim], a page's tokens in its first page_size rows (one tensor for keys and values:
// page_rows = 2 page_size, v_pool at the first value plane), which already hold the chunk's keys and values;
// out: [num_tokens, q_heads * vdim].  page_indices: device array of the sequences' page ids, back to back (the
// lists cover prefix + chunk).  work: device array (16-byte aligned) of `entries` records of 8 int32, one per
// (sequence, 256 rows of it), heaviest first: first row of the sequence in qkv, rows of the sequence in this chunk,
// index of its first page id, number of its pages, tokens cached for it (chunk included), which 256-row pair, 0, 0.
// page_size: a power of two >= 8.  dim and vdim: multiples of 8 up to 128.  flags bit 0: compute a quarter of the
// exponentials on the FMA pipe (not with a window, cap or sink).  window (0 = none) / keep_first, softcap (0 = none), sink
// and gate (null = none), chunked and sigmoid: see the top of the file.  bias: [q_heads][bias_len] in the activation type, or null
// (not with a window, cap or sink; with sigmoid weights only bias_len 1).
int blitz_attn_prefill_paged(const void* q, int64_t q_stride, const void* k_pool, const void* v_pool, void* out, int64_t out_stride,
                             const int32_t* page_indices, const int32_t* work, int entries, int num_tokens,
                             int q_heads, int kv_heads, int dim, int vdim, int page_size, int page_rows, int max_pages,
                             float sm_scale, int flags, int window, int keep_first, int chunked, int sigmoid, float softcap, const void* sink,
                             const void* bias, int bias_len, const void* gate, int64_t gate_stride, int* status, int dtype, cudaStream_t stream) {
  if (num_tokens <= 0 || entries <= 0) return 0;
  if (dim < 8 || dim > 128 || (dim & 7) || vdim < 8 || vdim > 128 || (vdim & 7)) return -1;
  if (kv_heads < 1 || (q_heads % kv_heads) != 0 || (out_stride & 7) || (q_stride & 7)) return -1;
  if (window < 0 || keep_first < 0 || softcap < 0.f) return -1;
  if ((chunked && (window < 1 || keep_first)) || (sigmoid && (sink || softcap > 0.f || keep_first || (bias && bias_len != 1)))) return -1;
  if (page_size < 8 || (page_size & (page_size - 1)) != 0 || page_rows < page_size || work == nullptr) return -1;
  if ((reinterpret_cast<uintptr_t>(work) & 15) != 0 || (reinterpret_cast<uintptr_t>(out) & 15) != 0) return -1;
  const int bt = page_size < 64 ? page_size : 64;
  // rows of a pool: those of the last page end with its tokens
  const uint64_t rows = (uint64_t)(max_pages - 1) * page_rows + page_size;
  CUtensorMap tm[3];
  if (!get_tmap_3d(&tm[0], q, (uint64_t)dim, (uint64_t)q_heads, (uint64_t)num_tokens, (uint64_t)dim * 2, (uint64_t)q_stride * 2, 64, 1, kPpTile))
    return -2;
  for (int i = 1; i < 3; ++i) {
    const uint64_t d = i == 1 ? dim : vdim;
    if (!get_tmap_3d(&tm[i], i == 1 ? k_pool : v_pool, d, (uint64_t)kv_heads, rows, d * 2, d * 2 * kv_heads, 64, 1, (uint32_t)bt)) return -2;
  }
  PagedPrefillParams p;
  p.out = out; p.out_stride = out_stride; p.page_indices = page_indices; p.work = work; p.entries = entries;
  p.gate = gate; p.gate_stride = gate_stride; p.vdim = vdim; p.page_rows = page_rows;
  p.q_heads = q_heads; p.kv_heads = kv_heads; p.page_size = page_size; p.box_tokens = bt;
  p.oob_row = (int)rows;
  p.scale_log2 = sm_scale * 1.4426950408889634f; p.status = status; p.trace = g_pp_trace;
  p.chunked = chunked;
  p.window = window; p.keep_first = keep_first; p.sink = sink; p.bias = bias; p.bias_len = bias_len;
  p.cap_scale = softcap > 0.f ? sm_scale / softcap : 0.f; p.cap_log2 = softcap * 1.4426950408889634f;
  // tanh(z) = z (k0 + k1 z^2 + k2 z^4 + k3 z^6) for |z| <= 0.5 (Chebyshev interpolation of tanh(z) / z in z^2, absolute
  // error 2.5e-7), with z = q.k * cap_scale folded in.  Scores below 40 log2 units keep every probability that refers to
  // the largest magnitude above 2^-80.  A tiny scale / cap would underflow in the coefficients: no polynomial then.
  const double z = p.cap_scale, k[4] = {0.99999945, -0.33326284, 0.13189939, -0.04439274};
  double zn = z * p.cap_log2;
  for (int i = 0; i < 4; ++i, zn *= z * z) p.poly[i] = (float)(k[i] * zn);
  p.small_max = z > 1e-5 ? (float)fmin(0.5 / z, 40.0 / p.scale_log2) : 0.f;
  const long long total = (long long)entries * q_heads;
  const int sms = device_sm_count();
  const int grid = (int)(total < sms ? total : sms);
  const bool poly = (flags & 1) != 0, ext = window > 0 || softcap > 0.f || sink != nullptr;
  if (bias != nullptr && !sigmoid && (ext || bias_len < 1)) return -1;
  auto sized = [&](auto type, auto poly_, auto ext_, auto bias_, auto sig_) {
    using T = decltype(type);
    constexpr bool P = decltype(poly_)::value, X = decltype(ext_)::value, B = decltype(bias_)::value, G = decltype(sig_)::value;
    if (dim > 64)
      return vdim > 64 ? launch_paged_prefill<T, 128, 128, P, X, B, G>(tm, p, grid, stream)
                       : launch_paged_prefill<T, 128, 64, P, X, B, G>(tm, p, grid, stream);
    return vdim > 64 ? launch_paged_prefill<T, 64, 128, P, X, B, G>(tm, p, grid, stream)
                     : launch_paged_prefill<T, 64, 64, P, X, B, G>(tm, p, grid, stream);
  };
  auto launch = [&](auto type) {
    const std::false_type no{};
    const std::true_type yes{};
    if (sigmoid) return sized(type, no, yes, no, yes);
    if (bias != nullptr) return sized(type, no, no, yes, no);
    if (ext) return sized(type, no, yes, no, no);
    if (poly) return sized(type, yes, no, no, no);
    return sized(type, no, no, no, no);
  };
  return dtype == 1 ? launch(__nv_bfloat16{}) : launch(__half{});
}

}  // extern "C"
