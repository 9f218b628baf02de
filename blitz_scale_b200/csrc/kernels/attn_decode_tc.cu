// Paged-KV decode attention, tensor-core version (the serving path).
//
// Decode attention is a stream over the K and V pages of every sequence; with
// GQA the 4-8 query heads that share a KV head turn the per-token work into a
// small matrix product, so the FLOPs go to mma.sync (m16n8k16, query heads
// padded to 16 rows) and the instruction stream per token drops ~10x against a
// CUDA-core dot product; the kernel is then bound by HBM as it should be.
// tcgen05 is not used here on purpose: its minimum M of 64 rows would waste
// 94 % of each instruction on padding for one query token per sequence.
//
// Data movement: a producer warp walks the page table and issues TMA
// (cp.async.bulk.tensor.3d, plain per-CTA loads) boxes of [tokens x 64 dims]
// straight from the paged layout [page][K|V][token][kv_head][head_dim] into
// 128-byte-swizzled shared memory, 4 stages of 64 tokens (128 KB in flight
// per SM for head_dim 128).  Four consumer warps each own 16 of the 64 tokens
// of a stage: S = Q K^T via ldmatrix + mma, online softmax in registers
// (exp2, fp32), O += P V via ldmatrix.trans + mma.  Warps merge their partial
// (m, l, O) through shared memory; with num_splits > 1 each item writes an fp32
// partial and a merge kernel combines the splits (flash-decoding).
//
// The kernel is persistent: one CTA per SM walks the work items (sequence,
// KV head, split) in a grid-stride loop and the TMA pipeline runs across item
// boundaries, so it never drains between sequences (5.6 TB/s at batch 256,
// context 1024).  It is launched with programmatic dependent launch: shared
// memory is cleared and the barriers are set up while the previous kernel is
// still running; the first load waits for it.
//
// Models that ask for it get a sliding window with kept first tokens (only the 64-token chunks that hold a visible key
// are fetched: a sequence costs at most window + kept tokens whatever its length), soft-capped scores
// (cap * tanh(s / cap)) and a per-head sink, a term e^sink in the softmax denominator, which the merge adds once.
//
// The cache must hold finite values in every slot of an allocated page (the
// pool is zero-filled at creation): masked positions get probability 0, and
// 0 x NaN would still poison the accumulator.
//
// Keys and values may differ in size, and either may be smaller than the tile it is computed in (64 or 128 columns, a
// multiple of 8): TMA fills the columns behind a head's end with zeros.  A gate (one number per head and row, through a
// sigmoid) multiplies a head's output as it is stored.  More than 8 query heads per KV head run as several groups that
// read the same keys and values (the second one from L2).
//
// A bias by distance per head, bias[h][min(i - j, bias_len - 1)], is added to the scaled scores; only chunks with a distance
// inside the table look it up (four entries a lane, requested before the wait for the chunk).
//
// The window may be a chunk counted from position 0 (`chunked`: the keys of the position's own chunk are visible), and weights may
// be sigmoids of the scores instead of a softmax (`sigmoid`): then nothing refers to a maximum or is normalised, and warps and
// splits just add up.
//
// Replaces src/kernel/attention_decode.cu:13-40 and the host-side plan of
// src/kernel/flashinfer_types.cu:52-80.
#include "launch.cuh"
#include "ptx.cuh"
#include "tmap.cuh"
#include "common.cuh"
#include "mma.cuh"

namespace blitz {

constexpr int kTcThreads = 160;
constexpr int kTcChunk = 64;
constexpr int kTcStages = 6;
constexpr int kTcSlabBytes = kTcChunk * 128;

struct DecodeTcParams {
  const void* q;
  int64_t q_stride;
  const int32_t* indices;
  const int32_t* indptr;
  const int32_t* last_page_len;
  void* out;
  int64_t out_stride;
  float* part_o;
  float* part_lse;
  int batch, q_heads, kv_heads, group, page_size, max_pages, num_splits, box_tokens;
  int kv_div;               // kv_heads counts groups of at most 8 query heads: kv_div of them share a KV head
  int dim, vdim, page_rows; // page n's token `off` is row n * page_rows + off of both pools
  int v_rows;               // > 0: one tensor (and one map) for keys and values, which lie this many rows behind their keys
  const void* gate;         // [batch][gate_stride], a column per query head, or null
  int64_t gate_stride;
  int tail_box_tokens;  // box height of the second tensor map, used for the last (partly filled) chunk of a sequence
  float scale_log2;
  int chunked, sigmoid;         // see the top of the file
  int window, keep_first;       // 0: every key; else a token sees the last `window` positions and the first `keep_first`
  float cap_scale, cap_log2;    // soft cap (cap_log2 > 0): score in log2 units = cap_log2 * tanh(q.k * cap_scale)
  const void* sink;             // [q_heads] in the activation type, or null
  const void* bias;             // [q_heads][bias_len] in the activation type, or null
  int bias_len;
  int* status;
  long long* trace;  // profiling aid (null in production): clock stamps of CTA 0's first items, see blitz_attn_decode_set_trace
};

constexpr int kTcTraceItems = 16, kTcTraceSlots = 8;
__device__ __forceinline__ void tc_trace(const DecodeTcParams& p, int n, int slot) {
  if (p.trace != nullptr && blockIdx.x == 0 && n < kTcTraceItems) p.trace[n * kTcTraceSlots + slot] = clock64();
}

template <int HD, int VD = HD>
struct TcCfg {
  static constexpr int kSlabs = HD / 64, kValueSlabs = VD / 64;
  static constexpr int kStageBytes = (kSlabs + kValueSlabs) * kTcSlabBytes;
  static constexpr int kMergeFloats = 4 * 8 * VD + 2 * 4 * 8;
  static constexpr int kSmemBytes = kTcStages * kStageBytes + kMergeFloats * 4 + 1024 + 128;
};

template <typename T>
__device__ __forceinline__ float head_gate(const T* z) { return 1.f / (1.f + expf(-to_f<T>(*z))); }

// Work item = (sequence, kv head, split).  The kernel is persistent: each CTA walks items
// blockIdx.x, blockIdx.x + gridDim.x, ... and the producer keeps streaming the next item's pages while
// the consumers finish the current one, so the 4-stage pipeline never drains between items.
struct DecItem {
  int b, h, kv_head, split, pg_beg, seq_len, c_beg, c_end;  // c_beg .. c_end: this split's share of the visible chunks
  int lo, first;         // visible keys: [0, first) and [lo, seq_len)
  int n_first, c_window; // chunks of the kept tokens; first chunk of the window behind them
  // the n-th visible chunk
  __device__ __forceinline__ int chunk(int n) const { return n < n_first ? n : c_window + n - n_first; }
};
__device__ __forceinline__ DecItem dec_item(const DecodeTcParams& p, int item) {
  DecItem it;
  it.split = item % p.num_splits;
  it.h = (item / p.num_splits) % p.kv_heads;
  it.kv_head = p.kv_div == 1 ? it.h : it.h / p.kv_div;
  it.b = item / (p.num_splits * p.kv_heads);
  it.pg_beg = p.indptr[it.b];
  const int npages = p.indptr[it.b + 1] - it.pg_beg;
  it.seq_len = npages > 0 ? (npages - 1) * p.page_size + p.last_page_len[it.b] : 0;
  it.lo = p.window > 0 ? (p.chunked ? max(0, it.seq_len - 1) / p.window * p.window : max(0, it.seq_len - p.window)) : 0;
  it.first = min(p.keep_first, it.lo);
  it.n_first = (it.first + kTcChunk - 1) / kTcChunk;
  it.c_window = max(it.lo / kTcChunk, it.n_first);
  const int nchunks = it.n_first + max(0, (it.seq_len + kTcChunk - 1) / kTcChunk - it.c_window);
  const int cps = (nchunks + p.num_splits - 1) / p.num_splits;
  it.c_beg = min(nchunks, it.split * cps);
  it.c_end = min(nchunks, (it.split + 1) * cps);
  return it;
}

// PLAIN: heads as large as the tiles, one tensor for keys and values, no gate, at most 8 query heads per KV head.
template <typename T, int HD, int VD = HD, bool PLAIN = true>
__global__ void __launch_bounds__(kTcThreads, 1)
attn_decode_tc_kernel(const __grid_constant__ CUtensorMap tmap_k, const __grid_constant__ CUtensorMap tmap_k_tail,
                      const __grid_constant__ CUtensorMap tmap_v, const __grid_constant__ CUtensorMap tmap_v_tail,
                      const DecodeTcParams p) {
  using Cfg = TcCfg<HD, VD>;
  constexpr int SL = Cfg::kSlabs, SV = Cfg::kValueSlabs;
  const int dim = PLAIN ? HD : p.dim, vdim = PLAIN ? VD : p.vdim;
  extern __shared__ uint8_t smem_raw[];
  const uint32_t raw_addr = ptx::smem_u32(smem_raw);
  uint8_t* smem = smem_raw + (((raw_addr + 1023u) & ~1023u) - raw_addr);
  float* mrg_o = reinterpret_cast<float*>(smem + kTcStages * Cfg::kStageBytes);  // [4][8][VD]
  float* mrg_m = mrg_o + 4 * 8 * VD;                                              // [4][8]
  float* mrg_l = mrg_m + 32;                                                      // [4][8]
  uint64_t* full_bar = reinterpret_cast<uint64_t*>(mrg_l + 32);
  uint64_t* empty_bar = full_bar + kTcStages;
  volatile int* abort_flag = reinterpret_cast<volatile int*>(empty_bar + kTcStages);

  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int G = p.group;
  const int num_items = p.batch * p.kv_heads * p.num_splits;

  // zero the stages once: rows a short last chunk never fills must stay finite
  for (int i = threadIdx.x; i < kTcStages * Cfg::kStageBytes / 16; i += kTcThreads)
    reinterpret_cast<uint4*>(smem)[i] = make_uint4(0, 0, 0, 0);
  if (threadIdx.x == 0) {
    for (int i = 0; i < kTcStages; ++i) {
      ptx::mbar_init(&full_bar[i], 1);
      ptx::mbar_init(&empty_bar[i], 4);
    }
    *abort_flag = 0;
    ptx::fence_mbar_init();
    ptx::tma_prefetch_desc(&tmap_k);
    ptx::tma_prefetch_desc(&tmap_v);
    ptx::tma_prefetch_desc(&tmap_k_tail);
    ptx::tma_prefetch_desc(&tmap_v_tail);
  }
  ptx::fence_proxy_async_smem();
  __syncthreads();
  // programmatic dependent launch: the set-up above may overlap the previous kernel; q and the KV pages
  // are its outputs, so wait before the first load
  ptx::griddep_launch_dependents();
  ptx::griddep_wait();

  if (warp == 4) {
    // ------------------------------------------------------------ producer (whole warp; lane 0 issues)
    // A TMA box can only be issued once its page id is known, and a page id read from global memory right before
    // the issue costs one memory latency per chunk, which by itself caps the stream near 50 GB/s per SM.  So the
    // warp reads page ids 32 at a time (one coalesced load, lane l keeps entry l of the window), hands them out by
    // shuffle, and requests the next item's page-table window and lengths while the current item streams.
    const int ps = p.page_size;
    auto load_window = [&](const DecItem& it, int first_page) -> int {
      const int npages = p.indptr[it.b + 1] - it.pg_beg;
      return (first_page + lane < npages) ? p.indices[it.pg_beg + first_page + lane] : 0;
    };
    int stage = 0;
    uint32_t phase = 0;
    bool ok = true;
    int item = blockIdx.x;
    DecItem it = item < num_items ? dec_item(p, item) : DecItem{};
    int win_base = item < num_items ? (it.chunk(it.c_beg) * kTcChunk) / ps : 0;
    int win = item < num_items ? load_window(it, win_base) : 0;
    int n_done = 0;
    while (item < num_items && ok) {
      if (lane == 0) tc_trace(p, n_done, 4);
      // next item's metadata and first window: in flight while this item streams
      const int next = item + gridDim.x;
      DecItem nit = next < num_items ? dec_item(p, next) : DecItem{};
      const int nwin_base = next < num_items ? (nit.chunk(nit.c_beg) * kTcChunk) / ps : 0;
      const int nwin = next < num_items ? load_window(nit, nwin_base) : 0;
      for (int c = it.c_beg; c < it.c_end && ok; ++c) {
        const int tok0 = it.chunk(c) * kTcChunk;
        const int ntok = min(kTcChunk, it.seq_len - tok0);
        // a full chunk comes in boxes of box_tokens rows; the last chunk of a sequence only as far as it is
        // filled, in the smaller boxes of the second map (a 64-token page with 18 live tokens costs 32 rows)
        const bool tail = ntok < kTcChunk;
        const int bt = tail ? p.tail_box_tokens : p.box_tokens;
        const CUtensorMap* tk = tail ? &tmap_k_tail : &tmap_k;
        const CUtensorMap* tv = PLAIN || p.v_rows > 0 ? tk : tail ? &tmap_v_tail : &tmap_v;
        const uint32_t box_bytes = static_cast<uint32_t>(bt) * 128u;
        const int pieces = (ntok + bt - 1) / bt;
        const int last_page = (tok0 + ntok - 1) / ps;
        if (last_page >= win_base + 32) {  // sequences of more than 32 pages: move the window
          win_base = tok0 / ps;
          win = load_window(it, win_base);
        }
        int good = 1;
        if (lane == 0) {
          if (!ptx::bounded_mbar_wait(&empty_bar[stage], phase ^ 1u, abort_flag)) {
            if (p.status) atomicCAS(p.status, 0, kStatusTimeoutProducer);
            good = 0;
          } else {
            ptx::mbar_expect_tx(&full_bar[stage], static_cast<uint32_t>(pieces) * (SL + SV) * box_bytes);
          }
        }
        good = __shfl_sync(0xffffffffu, good, 0);
        if (!good) {
          ok = false;
          break;
        }
        uint8_t* sb = smem + stage * Cfg::kStageBytes;
        for (int i = 0; i < pieces; ++i) {
          const int t = tok0 + i * bt;
          int page = __shfl_sync(0xffffffffu, win, (t / ps - win_base) & 31);
          if (lane == 0) {
            if (page < 0 || page >= p.max_pages) {
              if (p.status) atomicCAS(p.status, 0, kStatusBadIndex);
              page = 0;
            }
            const int z = page * (PLAIN ? 2 * ps : p.page_rows) + (t % ps), h = PLAIN ? it.h : it.kv_head;
#pragma unroll
            for (int s = 0; s < (SL > SV ? SL : SV); ++s) {
              if (s < SL) ptx::tma_load_3d(sb + s * kTcSlabBytes + i * box_bytes, tk, &full_bar[stage], s * 64, h, z);
              if (s < SV) ptx::tma_load_3d(sb + (SL + s) * kTcSlabBytes + i * box_bytes, tv, &full_bar[stage], s * 64, h, z + (PLAIN ? ps : p.v_rows));
            }
          }
        }
        if (++stage == kTcStages) {
          stage = 0;
          phase ^= 1u;
        }
      }
      if (lane == 0) tc_trace(p, n_done, 5);
      ++n_done;
      item = next;
      it = nit;
      win_base = nwin_base;
      win = nwin;
    }
  } else {
    // ------------------------------------------------------------ consumers (128 threads, named barrier 1)
    const int g = lane >> 2, t4 = lane & 3;
    const int tokw = warp * 16;
    const int mi = lane >> 3, mr = lane & 7;  // ldmatrix: matrix index and row within it
    int stage = 0;
    uint32_t phase = 0;
    bool ok = true;  // after a timeout this warp stops waiting but keeps meeting the others at the barriers
    // The consumers stop consuming between two items (merge, then the next item's lengths and query rows), and a
    // pause longer than the pipeline can absorb empties the memory pipe, which then costs a full latency to refill.
    // So the next item's descriptor and Q fragments are requested while the current item is being processed.
    auto load_q = [&](const DecItem& d, uint32_t (&a0)[HD / 16], uint32_t (&a2)[HD / 16]) {
      // Q as A fragments (rows >= G and columns >= dim are zero padding; rows 8..15 are never populated since G <= 8)
      const int cols = g < G ? dim : 0;
      const T* qrow = reinterpret_cast<const T*>(p.q) + static_cast<int64_t>(d.b) * p.q_stride +
                      static_cast<int64_t>(d.h * G + g) * dim;
#pragma unroll
      for (int ks = 0; ks < HD / 16; ++ks) {
        a0[ks] = ks * 16 < cols ? *reinterpret_cast<const uint32_t*>(qrow + ks * 16 + 2 * t4) : 0u;
        a2[ks] = ks * 16 + 8 < cols ? *reinterpret_cast<const uint32_t*>(qrow + ks * 16 + 2 * t4 + 8) : 0u;
      }
    };
    DecItem it = blockIdx.x < num_items ? dec_item(p, blockIdx.x) : DecItem{};
    uint32_t qa0[HD / 16], qa2[HD / 16];
    if (blockIdx.x < num_items) load_q(it, qa0, qa2);
    int n_done = 0;
    const bool tracer = warp == 0 && lane == 0;
    for (int item = blockIdx.x; item < num_items; item += gridDim.x, ++n_done) {
      if (tracer) tc_trace(p, n_done, 0);
      const int next = item + gridDim.x;
      DecItem nit = DecItem{};
      uint32_t nqa0[HD / 16], nqa2[HD / 16];
      if (next < num_items) {
        nit = dec_item(p, next);
        load_q(nit, nqa0, nqa2);
      }
      float o[VD / 8][4];
#pragma unroll
      for (int i = 0; i < VD / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
      float m = -INFINITY, l = 0.f;
      const T* bias_row = nullptr;
      float far_bias = 0.f;
      if (!PLAIN && p.bias != nullptr && g < G) {
        bias_row = reinterpret_cast<const T*>(p.bias) + static_cast<int64_t>(it.h * G + g) * p.bias_len;
        far_bias = to_f<T>(bias_row[p.bias_len - 1]) * 1.4426950408889634f;
      }
      for (int c = it.c_beg; c < it.c_end; ++c) {
        float bias[4] = {far_bias, far_bias, far_bias, far_bias};  // of the lane's four keys, in log2 units
        if (!PLAIN && bias_row != nullptr) {
          const int d0 = it.seq_len - 1 - (it.chunk(c) * kTcChunk + tokw + 2 * t4);  // distance of the first of them
          if (it.seq_len - 1 - (it.chunk(c) * kTcChunk + tokw + 15) < p.bias_len - 1) {
#pragma unroll
            for (int k = 0; k < 4; ++k)
              bias[k] = to_f<T>(bias_row[min(max(d0 - (k & 1) - (k >> 1) * 8, 0), p.bias_len - 1)]) * 1.4426950408889634f;
          }
        }
        if (ok && !ptx::bounded_mbar_wait(&full_bar[stage], phase, abort_flag)) {
          if (p.status && lane == 0) atomicCAS(p.status, 0, kStatusTimeoutEpilogue);
          ok = false;
        }
        if (tracer && c == it.c_beg) tc_trace(p, n_done, 1);
        const int tok0 = it.chunk(c) * kTcChunk;
        const int nvalid = min(kTcChunk, it.seq_len - tok0);
        // visible keys of this warp's 16: below `kept` or from `from` on (both relative to the chunk)
        const int kept = it.first - tok0, from = it.lo - tok0;
        if (ok && tokw < nvalid && (tokw < kept || (tokw + 16 > from && nvalid > from))) {
          const uint32_t kbase = ptx::smem_u32(smem + stage * Cfg::kStageBytes);
          const uint32_t vbase = kbase + SL * kTcSlabBytes;
          float s_lo[4] = {0.f, 0.f, 0.f, 0.f}, s_hi[4] = {0.f, 0.f, 0.f, 0.f};
          {
            const int tok = tokw + (mi >> 1) * 8 + mr;
#pragma unroll
            for (int ks = 0; ks < HD / 16; ++ks) {
              const int ch = ks * 2 + (mi & 1);
              const uint32_t addr = kbase + (ch >> 3) * kTcSlabBytes + tok * 128 + (((ch & 7) ^ (tok & 7)) << 4);
              uint32_t b0, b1, b2, b3;
              ldmatrix_x4(addr, b0, b1, b2, b3);
              mma16816<T>(s_lo, qa0[ks], 0u, qa2[ks], 0u, b0, b1);
              mma16816<T>(s_hi, qa0[ks], 0u, qa2[ks], 0u, b2, b3);
            }
          }
          const int col = tokw + 2 * t4;
          auto visible = [&](int k) { return k < nvalid && (k >= from || k < kept); };
          const bool v0 = visible(col), v1 = visible(col + 1), v2 = visible(col + 8), v3 = visible(col + 9);
          auto score = [&](float x) {  // log2 units
            return p.cap_log2 > 0.f ? p.cap_log2 * ptx::tanh_ex2(x * p.cap_scale) : x * p.scale_log2;
          };
#pragma unroll
          for (int k = 0; k < 2; ++k) {  // rows 8..15 of the fragments are padding
            s_lo[k] = score(s_lo[k]) + (PLAIN ? 0.f : bias[k]);
            s_hi[k] = score(s_hi[k]) + (PLAIN ? 0.f : bias[2 + k]);
          }
          const bool plain_sum = !PLAIN && p.sigmoid;
          float mx = plain_sum ? 0.f : -INFINITY;
          if (!plain_sum) {
            if (v0) mx = fmaxf(mx, s_lo[0]);
            if (v1) mx = fmaxf(mx, s_lo[1]);
            if (v2) mx = fmaxf(mx, s_hi[0]);
            if (v3) mx = fmaxf(mx, s_hi[1]);
            mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
            mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
          }
          const float m_new = fmaxf(m, mx);
          const float alpha = exp2f(m - m_new);  // m = -inf -> 0
          auto weight = [&](float x) { return plain_sum ? __fdividef(1.f, 1.f + exp2f(fminf(-x, 120.f))) : exp2f(x - m_new); };
          const float p0 = v0 ? weight(s_lo[0]) : 0.f;
          const float p1 = v1 ? weight(s_lo[1]) : 0.f;
          const float p2 = v2 ? weight(s_hi[0]) : 0.f;
          const float p3 = v3 ? weight(s_hi[1]) : 0.f;
          l = l * alpha + (p0 + p1 + p2 + p3);
          m = m_new;
          const uint32_t pa0 = pk2<T>(p0, p1), pa2 = pk2<T>(p2, p3);
#pragma unroll
          for (int i = 0; i < VD / 8; ++i) {
            o[i][0] *= alpha;
            o[i][1] *= alpha;
          }
          {
            const int tok = tokw + (mi & 1) * 8 + mr;
#pragma unroll
            for (int np = 0; np < VD / 16; ++np) {
              const int ch = np * 2 + (mi >> 1);
              const uint32_t addr = vbase + (ch >> 3) * kTcSlabBytes + tok * 128 + (((ch & 7) ^ (tok & 7)) << 4);
              uint32_t b0, b1, b2, b3;
              ldmatrix_x4_trans(addr, b0, b1, b2, b3);
              mma16816<T>(o[2 * np], pa0, 0u, pa2, 0u, b0, b1);
              mma16816<T>(o[2 * np + 1], pa0, 0u, pa2, 0u, b2, b3);
            }
          }
        }
        __syncwarp();
        if (lane == 0) ptx::mbar_arrive(&empty_bar[stage]);
        if (++stage == kTcStages) {
          stage = 0;
          phase ^= 1u;
        }
      }
      if (tracer) tc_trace(p, n_done, 2);
      // per-warp partials -> shared memory (rows < 8 only), then the 4 warps combine them
      l += __shfl_xor_sync(0xffffffffu, l, 1);
      l += __shfl_xor_sync(0xffffffffu, l, 2);
      if (t4 == 0) {
        mrg_m[warp * 8 + g] = m;
        mrg_l[warp * 8 + g] = l;
      }
#pragma unroll
      for (int i = 0; i < VD / 8; ++i) {
        float2 v = make_float2(o[i][0], o[i][1]);
        *reinterpret_cast<float2*>(&mrg_o[(warp * 8 + g) * VD + i * 8 + 2 * t4]) = v;
      }
      asm volatile("bar.sync 1, 128;" ::: "memory");
      for (int e = threadIdx.x; e < G * VD; e += 128) {
        const int gg = e / VD, d = e % VD;
        if (!PLAIN && d >= vdim) continue;
        float M = -INFINITY;
#pragma unroll
        for (int w = 0; w < 4; ++w) M = fmaxf(M, mrg_m[w * 8 + gg]);
        const int head = it.h * G + gg;
        const bool with_sink = p.sink != nullptr && p.num_splits == 1;  // several splits: the merge kernel adds it
        const float sink = with_sink ? to_f<T>(reinterpret_cast<const T*>(p.sink)[head]) * 1.4426950408889634f : -INFINITY;
        M = fmaxf(M, sink);
        float L = 0.f, O = 0.f;
        if (M > -INFINITY) {
#pragma unroll
          for (int w = 0; w < 4; ++w) {
            const float sc = exp2f(mrg_m[w * 8 + gg] - M);
            L += mrg_l[w * 8 + gg] * sc;
            O += mrg_o[(w * 8 + gg) * VD + d] * sc;
          }
        }
        if (with_sink) L += exp2f(sink - M);
        if (!PLAIN && p.sigmoid) L = 1.f;
        float val = L > 0.f ? O / L : 0.f;
        if (p.num_splits == 1) {
          if (!PLAIN && p.gate != nullptr) val *= head_gate(reinterpret_cast<const T*>(p.gate) + it.b * p.gate_stride + head);
          T* op = reinterpret_cast<T*>(p.out) + static_cast<int64_t>(it.b) * p.out_stride +
                  static_cast<int64_t>(head) * vdim;
          if (std::is_same<T, __nv_bfloat16>::value)
            reinterpret_cast<__nv_bfloat16*>(op)[d] = __float2bfloat16(val);
          else
            reinterpret_cast<__half*>(op)[d] = __float2half(val);
        } else {
          const int64_t base = (static_cast<int64_t>(it.b) * p.q_heads + head) * p.num_splits + it.split;
          p.part_o[base * vdim + d] = val;
          if (d == 0) p.part_lse[base] = L > 0.f ? M + log2f(L) : -INFINITY;
        }
      }
      asm volatile("bar.sync 1, 128;" ::: "memory");  // merge buffers are reused by the next item
      if (tracer) tc_trace(p, n_done, 3);
      it = nit;
#pragma unroll
      for (int ks = 0; ks < HD / 16; ++ks) {
        qa0[ks] = nqa0[ks];
        qa2[ks] = nqa2[ks];
      }
    }
  }
}

// Combine split partials: out = sum_s w_s o_s / (sum_s w_s + e^sink), w_s = 2^(lse_s - max lse).
template <typename T>
__global__ void attn_merge_tc_kernel(const float* __restrict__ part_o, const float* __restrict__ part_lse,
                                     T* __restrict__ out, int64_t out_stride, int q_heads, int hd, int num_splits,
                                     const T* __restrict__ sink, const T* __restrict__ gate, int64_t gate_stride, int sum_only) {
  const int b = blockIdx.x, head = blockIdx.y;
  const int64_t base = (static_cast<int64_t>(b) * q_heads + head) * num_splits;
  float M = -INFINITY;
  for (int s = 0; s < num_splits; ++s) M = fmaxf(M, part_lse[base + s]);
  const float snk = sink ? to_f<T>(sink[head]) * 1.4426950408889634f : -INFINITY;
  M = fmaxf(M, snk);
  const float g = gate ? head_gate(gate + b * gate_stride + head) : 1.f;
  for (int d = threadIdx.x; d < hd; d += blockDim.x) {
    float acc = 0.f, wsum = 0.f;
    if (M > -INFINITY) {
      for (int s = 0; s < num_splits; ++s) {
        const float w = exp2f(part_lse[base + s] - M);
        wsum += w;
        acc += w * part_o[(base + s) * hd + d];
      }
      if (sink) wsum += exp2f(snk - M);
    }
    if (sum_only) wsum = 1.f;  // (every split's reference is zero: the weights are ones)
    const float val = wsum > 0.f ? acc / wsum * g : 0.f;
    T* op = out + static_cast<int64_t>(b) * out_stride + static_cast<int64_t>(head) * hd;
    if (std::is_same<T, __nv_bfloat16>::value)
      reinterpret_cast<__nv_bfloat16*>(op)[d] = __float2bfloat16(val);
    else
      reinterpret_cast<__half*>(op)[d] = __float2half(val);
  }
}

template <typename T, int HD, int VD, bool PLAIN>
static int launch_tc(const CUtensorMap (&tm)[4], const DecodeTcParams& p, int batch, cudaStream_t stream) {
  using Cfg = TcCfg<HD, VD>;
  auto kern = attn_decode_tc_kernel<T, HD, VD, PLAIN>;
  static PerDeviceOnce once;
  cudaError_t e = once.run([&] { return cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, Cfg::kSmemBytes); });
  if (e != cudaSuccess) return (int)e;
  const int items = batch * p.kv_heads * p.num_splits;
  const int sms = device_sm_count();
  return (int)launch_pdl(kern, dim3(items < sms ? items : sms), dim3(kTcThreads), Cfg::kSmemBytes, stream, tm[0], tm[1], tm[2],
                         tm[3], p);
}

template <typename T>
static int launch_tc(const CUtensorMap (&tm)[4], const DecodeTcParams& p, int batch, cudaStream_t stream) {
  const bool plain = p.dim == p.vdim && (p.dim == 64 || p.dim == 128) && p.v_rows > 0 && p.gate == nullptr && p.bias == nullptr && p.kv_div == 1 && !p.sigmoid;
  if (plain) return p.dim == 64 ? launch_tc<T, 64, 64, true>(tm, p, batch, stream) : launch_tc<T, 128, 128, true>(tm, p, batch, stream);
  if (p.dim > 64)
    return p.vdim > 64 ? launch_tc<T, 128, 128, false>(tm, p, batch, stream) : launch_tc<T, 128, 64, false>(tm, p, batch, stream);
  return p.vdim > 64 ? launch_tc<T, 64, 128, false>(tm, p, batch, stream) : launch_tc<T, 64, 64, false>(tm, p, batch, stream);
}

}  // namespace blitz

namespace blitz {
static long long* g_tc_trace = nullptr;
}

extern "C" {
// Profiling aid: while `buf` (16 items x 8 int64 clock stamps, device memory) is set, CTA 0 of every following
// blitz_attn_decode launch records, per work item, when its first consumer warp starts the item, gets its first chunk,
// finishes its last chunk and finishes the merge (slots 0-3), and when the producer starts and ends issuing the item's
// loads (slots 4-5).
void blitz_attn_decode_set_trace(long long* buf) { blitz::g_tc_trace = buf; }
using namespace blitz;

// Bytes of fp32 scratch the split path needs: part_o then part_lse.
int64_t blitz_attn_decode_workspace_bytes(int batch, int q_heads, int head_dim, int num_splits) {
  if (num_splits <= 1) return 0;
  return (int64_t)batch * q_heads * num_splits * (head_dim + 1) * (int64_t)sizeof(float);
}

// k_pool, v_pool: [max_pages][page_rows][kv_heads][dim or vdim], a page's tokens in its first page_size rows (one tensor for
// keys and values: page_rows = 2 page_size, v_pool at the first value plane).  workspace: scratch of
// blitz_attn_decode_workspace_bytes() bytes for value heads of vdim (may be null when num_splits == 1).
// page_size must be a power of two >= 8 (pages smaller than 64 tokens are fetched as several boxes per stage).  dim and
// vdim: multiples of 8 up to 128.  window (0 = none) / keep_first, softcap (0 = none), sink and gate (null = none) as
// described at the top of the file.  bias: [q_heads][bias_len] in the activation type, or null.
int blitz_attn_decode(const void* q, int64_t q_stride, const void* k_pool, const void* v_pool, const int32_t* indices,
                      const int32_t* indptr, const int32_t* last_page_len, void* out, int64_t out_stride,
                      void* workspace, int batch, int q_heads, int kv_heads, int dim, int vdim, int page_size, int page_rows,
                      int max_pages, int num_splits, float sm_scale, int window, int keep_first, int chunked, int sigmoid, float softcap,
                      const void* sink, const void* bias, int bias_len, const void* gate, int64_t gate_stride, int* status, int dtype, cudaStream_t stream) {
  if (batch <= 0) return 0;
  if (window < 0 || keep_first < 0 || softcap < 0.f || (bias != nullptr && bias_len < 1)) return -1;
  if ((chunked && (window < 1 || keep_first)) || (sigmoid && (sink || softcap > 0.f))) return -1;
  if (num_splits < 1 || kv_heads < 1 || (q_heads % kv_heads) != 0 || (q_stride & 1)) return -1;
  if (dim < 8 || dim > 128 || (dim & 7) || vdim < 8 || vdim > 128 || (vdim & 7)) return -1;
  if (page_size < 8 || (page_size & (page_size - 1)) != 0 || page_rows < page_size) return -1;
  if (num_splits > 1 && workspace == nullptr) return -1;
  const int group = q_heads / kv_heads;
  int div = (group + 7) / 8;
  while (group % div) ++div;
  const int bt = page_size < kTcChunk ? page_size : kTcChunk;
  const int bt_tail = bt < 16 ? bt : 16;
  const bool one = dim == vdim && page_rows == 2 * page_size &&
                   v_pool == reinterpret_cast<const char*>(k_pool) + (int64_t)page_size * kv_heads * dim * 2;
  if (one) v_pool = k_pool;
  // rows of a pool: those of the last page end with its tokens
  const uint64_t rows = one ? (uint64_t)max_pages * page_rows : (uint64_t)(max_pages - 1) * page_rows + page_size;
  CUtensorMap tm[4];
  for (int i = 0; i < 4; ++i) {
    const uint64_t d = i < 2 ? dim : vdim;
    if (!get_tmap_3d(&tm[i], i < 2 ? k_pool : v_pool, d, (uint64_t)kv_heads, rows, d * 2, d * 2 * kv_heads, 64, 1,
                     (uint32_t)(i & 1 ? bt_tail : bt)))
      return -2;
  }
  DecodeTcParams p;
  p.q = q; p.q_stride = q_stride; p.indices = indices; p.indptr = indptr; p.last_page_len = last_page_len;
  p.out = out; p.out_stride = out_stride;
  p.part_o = reinterpret_cast<float*>(workspace);
  p.part_lse = p.part_o ? p.part_o + (int64_t)batch * q_heads * num_splits * vdim : nullptr;
  p.batch = batch; p.q_heads = q_heads; p.kv_heads = kv_heads * div; p.kv_div = div; p.group = group / div;
  p.page_size = page_size; p.max_pages = max_pages; p.dim = dim; p.vdim = vdim; p.page_rows = page_rows; p.v_rows = one ? page_size : 0;
  p.num_splits = num_splits; p.box_tokens = bt; p.tail_box_tokens = bt_tail;
  p.scale_log2 = sm_scale * 1.4426950408889634f; p.status = status; p.trace = g_tc_trace;
  p.chunked = chunked; p.sigmoid = sigmoid;
  p.window = window; p.keep_first = keep_first; p.sink = sink; p.bias = bias; p.bias_len = bias_len; p.gate = gate; p.gate_stride = gate_stride;
  p.cap_scale = softcap > 0.f ? sm_scale / softcap : 0.f; p.cap_log2 = softcap * 1.4426950408889634f;
  int rc = dtype == 1 ? launch_tc<__nv_bfloat16>(tm, p, batch, stream) : launch_tc<__half>(tm, p, batch, stream);
  if (rc != 0) return rc;
  if (num_splits > 1) {
    auto merge = [&](auto type) {
      using T = decltype(type);
      attn_merge_tc_kernel<T><<<dim3(batch, q_heads), vdim > 64 ? 128 : 64, 0, stream>>>(
          p.part_o, p.part_lse, (T*)out, out_stride, q_heads, vdim, num_splits, (const T*)sink, (const T*)gate, gate_stride, sigmoid);
    };
    if (dtype == 1) merge(__nv_bfloat16{});
    else merge(__half{});
    rc = (int)cudaGetLastError();
  }
  return rc;
}

}  // extern "C"

// ---------------------------------------------------------------------------------------------------
// Allocation-free variant (declared and documented in attn_decode_noalloc.h).  The split-KV partials go to
// an array that is part of the library image instead of a caller-provided workspace.
#include "attn_decode_noalloc.h"

namespace blitz {

// Device global memory, present on every GPU that loads the library.  In host code this name is only a
// handle for the runtime: its device address is looked up once per device below and that address, not the
// name, is what the kernels receive.
static __device__ __align__(256) unsigned char g_noalloc_scratch[BLITZ_ATTN_NOALLOC_SCRATCH_BYTES];

constexpr int kNoallocMaxDevices = kMaxDevicesPerProcess;
// Device address of the scratch on each device: written once under the set-up lock and published with release
// order, so a host thread that sees a non-null value also sees a fully set-up device.
static std::atomic<void*> g_noalloc_ptr[kNoallocMaxDevices];
static PerDeviceOnce g_noalloc_once;

// Per-device set-up with that device current: resolve the scratch address, raise the shared-memory limits.
static cudaError_t noalloc_setup(int dev) {
  void* ptr = nullptr;
  cudaError_t e = cudaGetSymbolAddress(&ptr, g_noalloc_scratch);
  if (e != cudaSuccess) return e;
  if (ptr == nullptr) return cudaErrorInvalidSymbol;
  e = cudaFuncSetAttribute(attn_decode_tc_kernel<__nv_bfloat16, 128>, cudaFuncAttributeMaxDynamicSharedMemorySize, TcCfg<128>::kSmemBytes);
  if (e == cudaSuccess)
    e = cudaFuncSetAttribute(attn_decode_tc_kernel<__nv_bfloat16, 64>, cudaFuncAttributeMaxDynamicSharedMemorySize, TcCfg<64>::kSmemBytes);
  if (e == cudaSuccess)
    e = cudaFuncSetAttribute(attn_decode_tc_kernel<__half, 128>, cudaFuncAttributeMaxDynamicSharedMemorySize, TcCfg<128>::kSmemBytes);
  if (e == cudaSuccess)
    e = cudaFuncSetAttribute(attn_decode_tc_kernel<__half, 64>, cudaFuncAttributeMaxDynamicSharedMemorySize, TcCfg<64>::kSmemBytes);
  if (e != cudaSuccess) return e;
  g_noalloc_ptr[dev].store(ptr, std::memory_order_release);
  return cudaSuccess;
}

// Tensor map of one KV layer built on the stack (the cached builder keeps a host-side table; this path keeps nothing).
static bool noalloc_tmap(CUtensorMap* out, const void* kv_layer, int head_dim, int kv_heads, int max_pages, int page_size,
                         int box_tokens) {
  PFN_encodeTiled enc = get_encode_fn();
  if (!enc || (reinterpret_cast<uintptr_t>(kv_layer) & 15) != 0) return false;
  cuuint64_t dims[3] = {(cuuint64_t)head_dim, (cuuint64_t)kv_heads, (cuuint64_t)max_pages * 2 * page_size};
  cuuint64_t strides[2] = {(cuuint64_t)head_dim * 2, (cuuint64_t)kv_heads * head_dim * 2};
  cuuint32_t box[3] = {64, 1, (cuuint32_t)box_tokens};
  cuuint32_t estr[3] = {1, 1, 1};
  return enc(out, CU_TENSOR_MAP_DATA_TYPE_UINT16, 3, const_cast<void*>(kv_layer), dims, strides, box, estr,
             CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
             CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}

template <typename T, int HD>
static int noalloc_launch(const CUtensorMap (&tm)[4], const DecodeTcParams& p, int sms, cudaStream_t stream) {
  const int items = p.batch * p.kv_heads * p.num_splits;
  attn_decode_tc_kernel<T, HD><<<items < sms ? items : sms, kTcThreads, TcCfg<HD>::kSmemBytes, stream>>>(tm[0], tm[1], tm[2], tm[3], p);
  return (int)cudaGetLastError();
}

}  // namespace blitz

extern "C" int blitz_attn_decode_noalloc(const void* q, int64_t q_stride, const void* kv_layer, const int32_t* indices,
                                         const int32_t* indptr, const int32_t* last_page_len, void* out,
                                         int64_t out_stride, int batch, int q_heads, int kv_heads, int head_dim,
                                         int page_size, int max_pages, int num_splits, float sm_scale, int* status,
                                         int dtype, cudaStream_t stream) {
  using namespace blitz;
  if (batch <= 0) return 0;
  if (num_splits < 1 || kv_heads <= 0 || (q_heads % kv_heads) != 0 || (q_stride & 1) || (out_stride & 1)) return -1;
  const int G = q_heads / kv_heads;
  if (G > 8 || (head_dim != 64 && head_dim != 128)) return -1;
  if (page_size < 8 || (page_size & (page_size - 1)) != 0) return -1;
  const int64_t need = num_splits > 1 ? (int64_t)batch * q_heads * num_splits * (head_dim + 1) * (int64_t)sizeof(float) : 0;
  if (need > (int64_t)BLITZ_ATTN_NOALLOC_SCRATCH_BYTES) return BLITZ_ATTN_NOALLOC_TOO_LARGE;
  int dev = 0;
  cudaError_t e = cudaGetDevice(&dev);
  if (e != cudaSuccess) return (int)e;
  if (dev < 0 || dev >= kNoallocMaxDevices) return -1;
  e = g_noalloc_once.run([&] { return noalloc_setup(dev); });
  if (e != cudaSuccess) return (int)e;
  void* const scratch = g_noalloc_ptr[dev].load(std::memory_order_acquire);
  if (scratch == nullptr) return (int)cudaErrorInvalidSymbol;
  const int bt = page_size < kTcChunk ? page_size : kTcChunk;
  const int bt_tail = bt < 16 ? bt : 16;
  CUtensorMap tm[4];
  for (int i = 0; i < 4; ++i)
    if (!noalloc_tmap(&tm[i], kv_layer, head_dim, kv_heads, max_pages, page_size, i & 1 ? bt_tail : bt)) return -2;
  DecodeTcParams p;
  p.q = q; p.q_stride = q_stride; p.indices = indices; p.indptr = indptr; p.last_page_len = last_page_len;
  p.out = out; p.out_stride = out_stride;
  p.part_o = reinterpret_cast<float*>(scratch);
  p.part_lse = p.part_o + (int64_t)batch * q_heads * num_splits * head_dim;
  p.batch = batch; p.q_heads = q_heads; p.kv_heads = kv_heads; p.group = G; p.page_size = page_size;
  p.max_pages = max_pages; p.num_splits = num_splits; p.box_tokens = bt; p.tail_box_tokens = bt_tail;
  p.scale_log2 = sm_scale * 1.4426950408889634f; p.status = status; p.trace = nullptr;
  p.kv_div = 1; p.dim = p.vdim = head_dim; p.page_rows = 2 * page_size; p.v_rows = page_size; p.gate = nullptr; p.gate_stride = 0;
  p.chunked = p.sigmoid = 0;
  p.window = 0; p.keep_first = 0; p.sink = nullptr; p.bias = nullptr; p.bias_len = 0; p.cap_scale = p.cap_log2 = 0.f;
  int sms = 0;
  cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
  if (sms <= 0) sms = 148;
  int rc;
  if (dtype == 1)
    rc = head_dim == 128 ? noalloc_launch<__nv_bfloat16, 128>(tm, p, sms, stream)
                         : noalloc_launch<__nv_bfloat16, 64>(tm, p, sms, stream);
  else
    rc = head_dim == 128 ? noalloc_launch<__half, 128>(tm, p, sms, stream)
                         : noalloc_launch<__half, 64>(tm, p, sms, stream);
  if (rc != 0 || num_splits == 1) return rc;
  dim3 grid(batch, q_heads);
  if (dtype == 1)
    attn_merge_tc_kernel<__nv_bfloat16><<<grid, head_dim, 0, stream>>>(p.part_o, p.part_lse, (__nv_bfloat16*)out, out_stride,
                                                                       q_heads, head_dim, num_splits, nullptr, nullptr, 0, 0);
  else
    attn_merge_tc_kernel<__half><<<grid, head_dim, 0, stream>>>(p.part_o, p.part_lse, (__half*)out, out_stride, q_heads,
                                                                head_dim, num_splits, nullptr, nullptr, 0, 0);
  return (int)cudaGetLastError();
}
