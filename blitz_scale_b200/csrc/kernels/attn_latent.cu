// Decode attention over cached latent rows on tcgen05: one key and value for all heads, the value being the first `rank`
// columns of the key (queries and outputs are in the latent space, the projections on both sides are block-diagonal products).
//
//   out[b][h] = sigmoid(gate[b][h]) * sum_j softmax_j(scale * q[b][h] . row_j) row_j[0 .. rank)
//
// All heads of a token read the same rows, so a block of keys is one operand for up to 128 query rows (heads):
//
//   S = Q K^T      tcgen05.mma, A = Q (heads x width, smem), B = K (keys x width, smem), S in TMEM, two buffers
//   P = softmax    thread = head: one pass over its row of S, P written back over S's first columns (16 bit)
//   O += P V       tcgen05.mma, A = P (TMEM), B = the first columns of the same K tile in smem, O in TMEM
//
// Rows beyond the heads hold whatever the shared memory behind Q holds; they are computed and never looked at, and warps
// without a head do nothing.  Up to 256 value columns fit beside S in tensor memory; larger ranks run as two items that read
// the same keys, as do heads beyond what shared memory holds queries for.
//
// Load, MMA and softmax warps walk the blocks on their own; S of the next block is issued before P V of the current one if its
// keys are there, also across sequences, and Q has two buffers, so that the tensor core works while the softmax does.  The row maximum a head's
// probabilities refer to moves only when it has grown by more than 2^8; O is then rescaled in place.
//
// The key blocks of all sequences, laid end to end, are dealt to the CTAs in equal contiguous shares whatever the lengths
// are: the work list follows from the page table on the device, so that the launch can be captured in a graph.  A CTA's
// share begins and ends anywhere in a sequence; it leaves at most two incomplete pieces (fp32 partial sums), which a second
// kernel merges.
#include "launch.cuh"
#include "ptx.cuh"
#include "scalar.cuh"
#include "tmap.cuh"

namespace blitz {

constexpr int kLaThreads = 192;       // softmax warps 0-3, MMA warp, load warp
constexpr int kLaMaxHeads = 128;      // query rows of an item
constexpr int kLaValueCols = 256;     // value columns of an item
constexpr int kLaMaxStages = 6;
constexpr int kLaMaxBatch = 4096;
constexpr int kLaSmem = 227 * 1024;
constexpr float kLaRescaleAt = 8.f;   // log2 units

struct LatentParams {
  const int32_t *indices, *indptr, *last_page_len;
  void* out;                    // [batch][out_stride], head h's rank columns from h * rank on
  const void* gate;             // [batch][gate_stride], or null
  int64_t out_stride, gate_stride;
  float *part_o, *part_lse;     // [grid][2][group][value columns], [grid][2][group]
  int batch, heads, group, subs, halves, rank, vcols, slabs, steps, stages, page_size, max_pages, box_tokens, oob_row;
  float scale_log2;
  int* status;
};

template <int KT>
__device__ __forceinline__ int la_length(const LatentParams& p, int b) {
  const int npages = p.indptr[b + 1] - p.indptr[b];
  return npages > 0 ? (npages - 1) * p.page_size + p.last_page_len[b] : 0;
}

// A CTA's share of the blocks as pieces of sequences.  Blocks are numbered sequence by sequence, all blocks of one sub-item
// (head group, value half) before the next one's; s_pref[b] counts the blocks of a sub-item before sequence b.
struct LaPiece {
  int b, sub, beg, end, blocks;  // blocks [beg, end) of the sequence's `blocks`
};
struct LaWalk {
  const int* pref;
  int batch, subs;
  int64_t x, hi;
  int b;
  __device__ __forceinline__ LaWalk(const int* pref_, int batch_, int subs_, int cta, int ctas) : pref(pref_), batch(batch_), subs(subs_) {
    const int64_t total = static_cast<int64_t>(pref[batch]) * subs;
    x = total * cta / ctas;
    hi = total * (cta + 1) / ctas;
    int lo = 0, up = batch - 1;
    while (lo < up) {
      const int mid = (lo + up + 1) >> 1;
      if (static_cast<int64_t>(pref[mid]) * subs <= x) lo = mid; else up = mid - 1;
    }
    b = lo;
  }
  __device__ __forceinline__ bool next(LaPiece& q) {
    if (x >= hi) return false;
    while (static_cast<int64_t>(pref[b + 1]) * subs <= x) ++b;
    const int n = pref[b + 1] - pref[b];
    const int rem = static_cast<int>(x - static_cast<int64_t>(pref[b]) * subs);
    q.b = b;
    q.blocks = n;
    q.sub = rem / n;
    q.beg = rem - q.sub * n;
    q.end = static_cast<int>(min(static_cast<int64_t>(n), q.beg + (hi - x)));
    x += q.end - q.beg;
    return true;
  }
};

template <typename T, int KT>
__global__ void __launch_bounds__(kLaThreads, 1)
attn_latent_kernel(const __grid_constant__ CUtensorMap tmap_q, const __grid_constant__ CUtensorMap tmap_k, const LatentParams p) {
  constexpr uint32_t kFmt = std::is_same<T, __nv_bfloat16>::value ? 1u : 0u;
  constexpr int KB = KT * 128;  // bytes of a slab of 64 columns of a key block
  extern __shared__ uint8_t smem_raw[];
  const uint32_t raw_addr = ptx::smem_u32(smem_raw);
  uint8_t* smem = smem_raw + (((raw_addr + 1023u) & ~1023u) - raw_addr);
  const int QB = (p.group + 7) / 8 * 1024;  // bytes of a slab of Q
  uint8_t* sQ = smem;                        // [2]
  uint8_t* sK = sQ + 2 * p.slabs * QB;       // [stages]
  uint64_t* bars = reinterpret_cast<uint64_t*>(sK + p.stages * p.slabs * KB);
  uint64_t* q_full = bars;         // [2] per piece
  uint64_t* q_empty = bars + 2;    // [2]
  uint64_t* s_full = bars + 4;     // [2] per block
  uint64_t* p_ready = bars + 6;    // [2]
  uint64_t* pv_done = bars + 8;    // [2]
  uint64_t* o_full = bars + 10;    // per piece
  uint64_t* o_free = bars + 11;
  uint64_t* k_full = bars + 12;    // [stages]
  uint64_t* k_empty = k_full + kLaMaxStages;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(k_empty + kLaMaxStages);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  int* s_pref = reinterpret_cast<int*>(tmem_slot + 2);  // [batch + 1]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int active = (p.group + 31) / 32;  // softmax warps with a head

  if (threadIdx.x == 0) {
    for (int i = 0; i < 2; ++i) {
      ptx::mbar_init(&q_full[i], 1);
      ptx::mbar_init(&q_empty[i], 1);
      ptx::mbar_init(&s_full[i], 1);
      ptx::mbar_init(&p_ready[i], 32 * active);
      ptx::mbar_init(&pv_done[i], 1);
    }
    ptx::mbar_init(o_full, 1);
    ptx::mbar_init(o_free, 32 * active);
    for (int i = 0; i < p.stages; ++i) {
      ptx::mbar_init(&k_full[i], 1);
      ptx::mbar_init(&k_empty[i], 1);
    }
    *abort_flag = 0;
    ptx::fence_mbar_init();
    ptx::tma_prefetch_desc(&tmap_q);
    ptx::tma_prefetch_desc(&tmap_k);
  }
  if (warp == 4) {
    ptx::tmem_alloc(tmem_slot, 512);
    ptx::tmem_relinquish();
  }
  __syncthreads();
  ptx::griddep_launch_dependents();
  ptx::griddep_wait();
  for (int b = threadIdx.x; b < p.batch; b += kLaThreads) s_pref[b + 1] = (la_length<KT>(p, b) + KT - 1) / KT;
  if (threadIdx.x == 0) s_pref[0] = 0;
  __syncthreads();
  if (warp == 0) {
    int carry = 0;
    for (int b0 = 0; b0 < p.batch; b0 += 32) {
      int v = b0 + lane < p.batch ? s_pref[b0 + lane + 1] : 0;
#pragma unroll
      for (int o = 1; o < 32; o <<= 1) {
        const int u = __shfl_up_sync(0xffffffffu, v, o);
        if (lane >= o) v += u;
      }
      v += carry;
      if (b0 + lane < p.batch) s_pref[b0 + lane + 1] = v;
      carry = __shfl_sync(0xffffffffu, v, 31);
    }
  }
  ptx::tc_fence_before_sync();
  __syncthreads();
  ptx::tc_fence_after_sync();
  const uint32_t tmem_base = *tmem_slot;
  const uint32_t tmem_O = tmem_base + 256;  // S buffers at + 0 and + 128
  auto wait = [&](uint64_t* bar, uint32_t parity) { return ptx::bounded_mbar_wait(bar, parity, abort_flag); };

  if (warp == 5) {
    // ------------------------------------------------------------ load warp
    const int bt = p.box_tokens;
    const bool mine = lane < KT / bt;
    auto warp_wait = [&](uint64_t* bar, uint32_t parity) {
      int ok = 1;
      if (lane == 0) ok = wait(bar, parity) ? 1 : 0;
      return __shfl_sync(0xffffffffu, ok, 0) != 0;
    };
    auto box_row = [&](const LaPiece& q, int blk) {  // this lane's first row of a block in the pool
      const int tok = blk * KT + lane * bt, slot = tok / p.page_size;
      const int pg0 = p.indptr[q.b], npages = p.indptr[q.b + 1] - pg0;
      if (!mine || slot >= npages) return p.oob_row;  // past the pool: the box arrives as zeros
      int page = p.indices[pg0 + slot];
      if (page < 0 || page >= p.max_pages) {
        if (p.status) atomicCAS(p.status, 0, kStatusBadIndex);
        page = 0;
      }
      return page * p.page_size + (tok & (p.page_size - 1));
    };
    LaWalk walk(s_pref, p.batch, p.subs, blockIdx.x, gridDim.x);
    LaPiece q;
    bool ok = true;
    int stage = 0;
    uint32_t phase = 1, n = 0;  // a stage's first round needs no wait (the other parity counts as passed)
    for (; ok && walk.next(q); ++n) {
      if (n >= 2) ok = warp_wait(&q_empty[n & 1], ((n >> 1) - 1) & 1);
      if (!ok) break;
      if (lane == 0) {
        ptx::mbar_expect_tx(&q_full[n & 1], static_cast<uint32_t>(p.slabs * p.group) * 128u);
        for (int s = 0; s < p.slabs; ++s)
          ptx::tma_load_3d(sQ + ((n & 1) * p.slabs + s) * QB, &tmap_q, &q_full[n & 1], s * 64, q.sub / p.halves * p.group, q.b);
      }
      int row = box_row(q, q.beg);
      for (int blk = q.beg; blk < q.end; ++blk) {
        const int row_next = blk + 1 < q.end ? box_row(q, blk + 1) : p.oob_row;
        ok = warp_wait(&k_empty[stage], phase);
        if (!ok) break;
        if (lane == 0) ptx::mbar_expect_tx(&k_full[stage], static_cast<uint32_t>(p.slabs) * KB);
        __syncwarp();
        if (mine)
          for (int s = 0; s < p.slabs; ++s)
            ptx::tma_load_2d(sK + (stage * p.slabs + s) * KB + lane * bt * 128, &tmap_k, &k_full[stage], s * 64, row);
        row = row_next;
        if (++stage == p.stages) {
          stage = 0;
          phase ^= 1u;
        }
      }
    }
    if (!ok && lane == 0 && p.status) atomicCAS(p.status, 0, kStatusTimeoutProducer);
  } else if (warp == 4) {
    // ------------------------------------------------------------ MMA warp: one thread issues
    if (lane == 0) {
      const uint32_t idesc_s = ptx::make_idesc_f16(kFmt, 0u, 0u, 128, KT);
      LaWalk ws(s_pref, p.batch, p.subs, blockIdx.x, gridDim.x), wo = ws;
      LaPiece ps, po;
      bool ok = true, more_s = ws.next(ps), more_o = wo.next(po);
      uint32_t gs = 0, go = 0, ns = 0, no = 0;  // blocks and pieces whose S, and whose P V, has been issued
      int blk_s = ps.beg, blk_o = po.beg, stage_s = 0, stage_o = 0;
      uint32_t phase_s = 0;
      auto ready_S = [&]() {
        return ptx::mbar_test_wait(&k_full[stage_s], phase_s) && (blk_s != ps.beg || ptx::mbar_test_wait(&q_full[ns & 1], (ns >> 1) & 1));
      };
      auto issue_S = [&]() {
        ptx::tc_fence_after_sync();
        const uint32_t a = ptx::smem_u32(sQ + (ns & 1) * p.slabs * QB), bb = ptx::smem_u32(sK + stage_s * p.slabs * KB);
        const uint32_t d = tmem_base + (gs & 1) * 128;
        for (int k = 0; k < p.steps; ++k)
          ptx::umma_f16_ss(d, ptx::make_smem_desc(a + (k >> 2) * QB + (k & 3) * 32, 16, 1024, ptx::kLayoutSw128),
                           ptx::make_smem_desc(bb + (k >> 2) * KB + (k & 3) * 32, 16, 1024, ptx::kLayoutSw128), idesc_s, k != 0 ? 1u : 0u);
        ptx::umma_commit(&s_full[gs & 1]);
        ++gs;
        if (++stage_s == p.stages) {
          stage_s = 0;
          phase_s ^= 1u;
        }
        if (++blk_s == ps.end) {
          ptx::umma_commit(&q_empty[ns & 1]);
          ++ns;
          more_s = ws.next(ps);
          blk_s = ps.beg;
        }
      };
      uint32_t spins = 0;
      uint64_t t0 = 0;
      while (ok && more_o) {
        // whichever can go first: the next S (at most one block ahead of P V), or P V of the oldest block
        if (more_s && gs - go < 2 && ready_S()) {
          issue_S();
          spins = 0;
          continue;
        }
        if (gs == go || !ptx::mbar_test_wait(&p_ready[go & 1], (go >> 1) & 1)) {
          if ((++spins & 63u) == 0) {
            const uint64_t now = ptx::globaltimer_ns();
            if (spins == 64u) t0 = now;
            if (*abort_flag || now - t0 > ptx::kDefaultWaitNs) {
              *abort_flag = 1;
              ok = false;
            }
          }
          continue;
        }
        spins = 0;
        if (blk_o == po.beg && no > 0) ok = wait(o_free, (no - 1) & 1);  // the last piece's O has been read
        if (!ok) break;
        ptx::tc_fence_after_sync();
        const int half = po.sub % p.halves;
        const int cols = min(p.vcols, p.rank - half * kLaValueCols);
        const uint32_t idesc_o = ptx::make_idesc_f16(kFmt, 0u, 1u, 128, (cols + 15) / 16 * 16);
        const uint32_t bb = ptx::smem_u32(sK + stage_o * p.slabs * KB) + half * (kLaValueCols / 64) * KB;
#pragma unroll
        for (int k = 0; k < KT / 16; ++k)
          ptx::umma_f16_ts(tmem_O, tmem_base + (go & 1) * 128 + k * 8, ptx::make_smem_desc(bb + k * 2048, KB, 1024, ptx::kLayoutSw128),
                           idesc_o, (blk_o != po.beg || k != 0) ? 1u : 0u);
        ptx::umma_commit(&k_empty[stage_o]);
        ptx::umma_commit(&pv_done[go & 1]);
        ++go;
        if (++stage_o == p.stages) stage_o = 0;
        if (++blk_o == po.end) {
          ptx::umma_commit(o_full);
          ++no;
          more_o = wo.next(po);
          blk_o = po.beg;
        }
      }
      if (!ok && p.status) atomicCAS(p.status, 0, kStatusTimeoutMma);
    }
  } else if (warp < active) {
    // ------------------------------------------------------------ softmax warps: thread = head
    const int r = warp * 32 + lane;
    const uint32_t lane_addr = static_cast<uint32_t>(warp * 32) << 16;
    const uint32_t tO = tmem_O + lane_addr;
    LaWalk walk(s_pref, p.batch, p.subs, blockIdx.x, gridDim.x);
    LaPiece q;
    bool ok = true;
    uint32_t g = 0, n = 0;
    for (; ok && walk.next(q); ++n) {
      const int len = la_length<KT>(p, q.b), half = q.sub % p.halves, head = q.sub / p.halves * p.group + r;
      const int cols = min(p.vcols, p.rank - half * kLaValueCols);
      const bool mine = r < p.group;
      float gate = 1.f;
      if (p.gate != nullptr && mine) gate = sigmoid_f(to_f<T>(reinterpret_cast<const T*>(p.gate)[q.b * p.gate_stride + head]));
      float m_ref = 0.f, l = 0.f;
      for (int blk = q.beg; blk < q.end; ++blk, ++g) {
        if (!wait(&s_full[g & 1], (g >> 1) & 1)) {
          ok = false;
          break;
        }
        ptx::tc_fence_after_sync();
        const uint32_t tS = tmem_base + (g & 1) * 128 + lane_addr;
        uint32_t v[KT / 32][32];
#pragma unroll
        for (int i = 0; i < KT / 32; ++i) ptx::tmem_ld_32x32(tS + i * 32, v[i]);
        ptx::tmem_ld_wait();
        auto score = [&](int i) -> uint32_t& { return v[i >> 5][i & 31]; };
        const int valid = len - blk * KT;
        if (valid < KT) {
#pragma unroll
          for (int i = 0; i < KT; ++i)
            if (i >= valid) score(i) = 0xff800000u;  // -inf
        }
        float mxs[8];
#pragma unroll
        for (int i = 0; i < 8; ++i) mxs[i] = __uint_as_float(score(i));
#pragma unroll
        for (int i = 8; i < KT - 8; i += 16)
#pragma unroll
          for (int k = 0; k < 8; ++k) mxs[k] = ptx::fmax3(mxs[k], __uint_as_float(score(i + 2 * k)), __uint_as_float(score(i + 2 * k + 1)));
#pragma unroll
        for (int i = KT - 8; i < KT; ++i) mxs[i & 7] = fmaxf(mxs[i & 7], __uint_as_float(score(i)));
        float mx = fmaxf(ptx::fmax3(mxs[0], mxs[1], mxs[2]), ptx::fmax3(mxs[3], mxs[4], mxs[5]));
        mx = ptx::fmax3(mx, mxs[6], mxs[7]) * p.scale_log2;
        if (blk == q.beg) {
          m_ref = mx;
        } else {
          const bool grow = mx > m_ref + kLaRescaleAt;
          if (__any_sync(0xffffffffu, grow && mine)) {
            if (!wait(&pv_done[(g - 1) & 1], ((g - 1) >> 1) & 1)) {  // O is settled
              ok = false;
              break;
            }
            ptx::tc_fence_after_sync();
            const float alpha = grow ? ptx::ex2_approx(m_ref - mx) : 1.f;
#pragma unroll 1
            for (int c = 0; c < cols; c += 32) {
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
        float rs[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int h = 0; h < KT / 64; ++h) {  // 64 scores -> 32 columns of pairs
          uint32_t pk[32];
#pragma unroll
          for (int i = 0; i < 32; ++i) {
            const float e0 = ptx::ex2_approx(fmaf(__uint_as_float(score(h * 64 + 2 * i)), p.scale_log2, -m_ref));
            const float e1 = ptx::ex2_approx(fmaf(__uint_as_float(score(h * 64 + 2 * i + 1)), p.scale_log2, -m_ref));
            rs[i & 3] += e0 + e1;
            pk[i] = pk2<T>(e0, e1);
          }
          ptx::tmem_st_32x32(tS + h * 32, pk);
        }
        ptx::tmem_st_wait();
        l += (rs[0] + rs[1]) + (rs[2] + rs[3]);
        ptx::tc_fence_before_sync();
        ptx::mbar_arrive(&p_ready[g & 1]);
      }
      if (ok) ok = wait(o_full, n & 1);
      if (!ok) break;
      ptx::tc_fence_after_sync();
      const bool whole = q.beg == 0 && q.end == q.blocks;
      const float inv = l > 0.f ? (whole ? gate : 1.f) / l : 0.f;
      T* dst = reinterpret_cast<T*>(p.out) + q.b * p.out_stride + static_cast<int64_t>(head) * p.rank + half * kLaValueCols;
      const int64_t part = (static_cast<int64_t>(blockIdx.x) * 2 + (n > 0)) * p.group + r;
      if (!whole && mine) p.part_lse[part] = m_ref + log2f(l);
#pragma unroll 1
      for (int c = 0; c < cols; c += 32) {
        uint32_t o[32];
        ptx::tmem_ld_32x32(tO + c, o);
        ptx::tmem_ld_wait();
        if (c + 32 >= cols) {  // the next piece may overwrite O
          ptx::tc_fence_before_sync();
          ptx::mbar_arrive(o_free);
        }
        if (mine) {
#pragma unroll
          for (int i = 0; i < 32; i += 8) {
            if (c + i < cols) {
              float x[8];
#pragma unroll
              for (int k = 0; k < 8; ++k) x[k] = __uint_as_float(o[i + k]) * inv;
              if (whole) *reinterpret_cast<uint4*>(dst + c + i) = pack8<T>(x);
              else stf8<float>(p.part_o + part * p.vcols + c + i, x);
            }
          }
        }
      }
    }
    if (!ok && p.status && lane == 0) atomicCAS(p.status, 0, kStatusTimeoutEpilogue);
  }

  ptx::tc_fence_before_sync();
  __syncthreads();
  if (warp == 4) {
    ptx::tc_fence_after_sync();
    ptx::tmem_dealloc(tmem_base, 512);
  }
}

// Rows whose blocks lie in more than one CTA's share: out = sum_c w_c o_c / sum_c w_c, w_c = 2^(lse_c - max lse).  Rows without
// keys become zeros.  A warp per head.
template <typename T, int KT>
__global__ void __launch_bounds__(256) attn_latent_merge_kernel(const LatentParams p, int ctas) {
  ptx::griddep_launch_dependents();
  ptx::griddep_wait();
  __shared__ int s_sum[2];
  const int b = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  if (threadIdx.x < 2) s_sum[threadIdx.x] = 0;
  __syncthreads();
  int before = 0, all = 0;
  for (int i = threadIdx.x; i < p.batch; i += blockDim.x) {
    const int n = (la_length<KT>(p, i) + KT - 1) / KT;
    all += n;
    before += i < b ? n : 0;
  }
  before = __reduce_add_sync(0xffffffffu, before);
  all = __reduce_add_sync(0xffffffffu, all);
  if (lane == 0) {
    atomicAdd(&s_sum[0], before);
    atomicAdd(&s_sum[1], all);
  }
  __syncthreads();
  const int head = blockIdx.y * 8 + warp;
  if (head >= p.heads) return;
  const int64_t total = static_cast<int64_t>(s_sum[1]) * p.subs;
  const int blocks = (la_length<KT>(p, b) + KT - 1) / KT;
  const float gate = p.gate ? sigmoid_f(to_f<T>(reinterpret_cast<const T*>(p.gate)[b * p.gate_stride + head])) : 1.f;
  for (int half = 0; half < p.halves; ++half) {
    const int cols = min(p.vcols, p.rank - half * kLaValueCols);
    T* dst = reinterpret_cast<T*>(p.out) + b * p.out_stride + static_cast<int64_t>(head) * p.rank + half * kLaValueCols;
    if (blocks == 0) {
      for (int c = lane; c < cols; c += 32) stf<T>(dst + c, 0.f);
      continue;
    }
    const int64_t beg = static_cast<int64_t>(s_sum[0]) * p.subs + static_cast<int64_t>(head / p.group * p.halves + half) * blocks;
    const int c0 = static_cast<int>(((beg + 1) * ctas - 1) / total), c1 = static_cast<int>(((beg + blocks) * ctas - 1) / total);
    if (c0 == c1) continue;  // one CTA has done all of it
    // the piece is its CTA's first one unless the CTA's share begins before this sequence
    auto part = [&](int c) { return (static_cast<int64_t>(c) * 2 + (total * c / ctas < beg ? 1 : 0)) * p.group + head % p.group; };
    auto has = [&](int c) { return total * c / ctas < total * (c + 1) / ctas; };  // (more CTAs than blocks: some have none)
    float m = -INFINITY;
    for (int c = c0 + lane; c <= c1; c += 32)
      if (has(c)) m = fmaxf(m, p.part_lse[part(c)]);
    m = warp_max(m);
    float acc[kLaValueCols / 32] = {}, sum = 0.f;
    for (int c = c0; c <= c1; ++c) {
      if (!has(c)) continue;
      const int64_t at = part(c);
      const float w = exp2f(p.part_lse[at] - m);
      sum += w;
#pragma unroll
      for (int k = 0; k < kLaValueCols / 32; ++k)
        if (k * 32 + lane < cols) acc[k] += w * p.part_o[at * p.vcols + k * 32 + lane];
    }
    const float f = gate / sum;
#pragma unroll
    for (int k = 0; k < kLaValueCols / 32; ++k)
      if (k * 32 + lane < cols) stf<T>(dst + k * 32 + lane, acc[k] * f);
  }
}

struct LatentPlan {
  int kt, group, halves, vcols, slabs, stages;
  size_t smem;
};
// How the heads are grouped and how tall a key block is: blocks of 128 keys and as many heads as possible, at least two stages.
static bool latent_plan(int batch, int heads, int width, int rank, int page_size, LatentPlan* out) {
  if (batch < 1 || batch > kLaMaxBatch || heads < 1 || rank < 8 || rank > 2 * kLaValueCols || width < rank || ((width | rank) & 7)) return false;
  if (page_size < 8 || (page_size & (page_size - 1)) != 0) return false;
  LatentPlan pl;
  pl.slabs = (width + 63) / 64;
  pl.halves = rank > kLaValueCols ? 2 : 1;
  pl.vcols = rank > kLaValueCols ? kLaValueCols : rank;
  const int fixed = 1024 + (12 + 2 * kLaMaxStages) * 8 + 8 + (batch + 1) * 4;
  for (int groups = 1; groups <= heads; ++groups) {
    if (heads % groups || heads / groups > kLaMaxHeads) continue;
    pl.group = heads / groups;
    for (int kt = 128; kt >= 64; kt /= 2) {
      const int room = kLaSmem - fixed - 2 * pl.slabs * ((pl.group + 7) / 8 * 1024);
      int stages = room / (pl.slabs * kt * 128);
      if (stages < 2) continue;
      pl.kt = kt;
      pl.stages = stages < kLaMaxStages ? stages : kLaMaxStages;
      // (the 128-row view of the last slab of Q ends in the key stages behind it)
      pl.smem = fixed + 2 * pl.slabs * ((pl.group + 7) / 8 * 1024) + (size_t)pl.stages * pl.slabs * kt * 128;
      *out = pl;
      return true;
    }
  }
  return false;
}

}  // namespace blitz

extern "C" {
using namespace blitz;

int blitz_attn_latent_supported(int batch, int heads, int width, int rank, int page_size) {
  LatentPlan pl;
  return latent_plan(batch, heads, width, rank, page_size, &pl) ? 1 : 0;
}

// Bytes of fp32 scratch for the partial sums, whatever the batch is.
int64_t blitz_attn_latent_workspace_bytes(int heads, int rank) {
  const int group = heads < kLaMaxHeads ? heads : kLaMaxHeads, cols = rank < kLaValueCols ? rank : kLaValueCols;
  return (int64_t)device_sm_count() * 2 * group * (cols + 1) * (int64_t)sizeof(float);
}

// q [batch][q_stride]: heads of `width` columns; pool [max_pages][page_size][width], the first `rank` columns are the values;
// out [batch][out_stride]: heads of `rank` columns.  width, rank: multiples of 8, rank up to 512; page_size: a power of two >= 8;
// gate [batch][gate_stride] or null.  A row without pages gives zeros.
int blitz_attn_latent(const void* q, int64_t q_stride, const void* pool, const int32_t* indices, const int32_t* indptr,
                      const int32_t* last_page_len, void* out, int64_t out_stride, void* workspace, int batch, int heads, int width, int rank,
                      int page_size, int max_pages, float sm_scale, const void* gate, int64_t gate_stride, int* status, int dtype,
                      cudaStream_t stream) {
  if (batch <= 0) return 0;
  LatentPlan pl;
  if (!latent_plan(batch, heads, width, rank, page_size, &pl) || workspace == nullptr || max_pages < 1) return -1;
  if ((q_stride & 7) || (out_stride & 7) || (reinterpret_cast<uintptr_t>(out) & 15) || (reinterpret_cast<uintptr_t>(workspace) & 31)) return -1;
  const int bt = page_size < 64 ? page_size : 64;
  CUtensorMap tq, tk;
  if (!get_tmap_3d(&tq, q, (uint64_t)width, (uint64_t)heads, (uint64_t)batch, (uint64_t)width * 2, (uint64_t)q_stride * 2, 64,
                   (uint32_t)pl.group, 1))
    return -2;
  if (!get_tmap_2d(&tk, pool, (uint64_t)width, (uint64_t)max_pages * page_size, (uint64_t)width * 2, 64, (uint32_t)bt)) return -2;
  const int sms = device_sm_count();
  LatentParams p;
  p.indices = indices; p.indptr = indptr; p.last_page_len = last_page_len; p.out = out; p.gate = gate;
  p.out_stride = out_stride; p.gate_stride = gate_stride;
  p.batch = batch; p.heads = heads; p.group = pl.group; p.halves = pl.halves; p.subs = heads / pl.group * pl.halves; p.rank = rank;
  p.vcols = pl.vcols; p.slabs = pl.slabs; p.steps = (width + 15) / 16; p.stages = pl.stages; p.page_size = page_size; p.max_pages = max_pages; p.box_tokens = bt;
  p.oob_row = max_pages * page_size;
  p.part_o = reinterpret_cast<float*>(workspace);
  p.part_lse = p.part_o + (int64_t)sms * 2 * pl.group * pl.vcols;
  p.scale_log2 = sm_scale * 1.4426950408889634f; p.status = status;
  auto go = [&](auto type, auto keys) -> int {
    using T = decltype(type);
    constexpr int KT = decltype(keys)::value;
    static PerDeviceOnce once;
    cudaError_t e = once.run([] { return cudaFuncSetAttribute(attn_latent_kernel<T, KT>, cudaFuncAttributeMaxDynamicSharedMemorySize, kLaSmem); });
    if (e == cudaSuccess) e = launch_pdl(attn_latent_kernel<T, KT>, dim3(sms), dim3(kLaThreads), pl.smem, stream, tq, tk, p);
    if (e == cudaSuccess) e = launch_pdl(attn_latent_merge_kernel<T, KT>, dim3(batch, (heads + 7) / 8), dim3(256), 0, stream, p, sms);
    return (int)e;
  };
  auto tall = [&](auto type) {
    return pl.kt == 128 ? go(type, std::integral_constant<int, 128>{}) : go(type, std::integral_constant<int, 64>{});
  };
  return dtype == 1 ? tall(__nv_bfloat16{}) : tall(__half{});
}

}  // extern "C"
