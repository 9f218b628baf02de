// Decode attention over cached latent rows on tcgen05: one key and value for all heads, the value being the first `rank`
// columns of the key (queries and outputs are in the latent space, the projections on both sides are block-diagonal products).
//
//   out[b][h] = sigmoid(gate[b][h]) * sum_j softmax_j(scale * q[b][h] . row_j) row_j[0 .. rank)
//
// All heads of a token read the same rows, so both products have the keys on one side and the heads on the other.  The keys
// and the value columns take the 128 rows of an instruction, the heads its N columns, of which any 16, 32 or 64 cost about
// the same:
//
//   S = K Q^T       tcgen05.mma, A = K (keys x width, smem), B = Q (heads x width, smem), S in TMEM, two buffers
//   P = softmax     thread = key: one score per head; P goes to shared memory as [key][head], 16 bit, two buffers
//   O += V^T P      tcgen05.mma, A = the first columns of the same K tile, read transposed, B = P; O in TMEM, a row per value
//                   column, a column per head, 128 value columns per instruction
//
// A head's probabilities refer to the score of the sequence's first key here, and to the maximum so far once some score has
// exceeded that by more than 2^40 (bf16 probabilities and fp32 sums have the range; fp16: 2^8); one vote per block decides, and O
// and the row sums are rescaled then.  Row sums stay in the threads until the end.
// More than 64 heads run as groups that read the same keys.
//
// A load warp, a warp for each product and the softmax warps walk the blocks on their own, also across sequences.  An MMA
// warp stays converged and one elected lane issues, which keeps the operand descriptors in uniform registers: an instruction
// then costs about what the tensor core needs, not what its issue takes.
//
// The key blocks of all sequences, laid end to end, are dealt to the CTAs in equal contiguous shares whatever the lengths
// are: the work list follows from the page table on the device, so that the launch can be captured in a graph.  A CTA's
// share begins and ends anywhere in a sequence; it leaves at most two incomplete pieces (fp32 partial sums), which a second
// kernel merges.
//
// A sliding window leaves the blocks before it out (a sequence's blocks are counted from its first visible key's on); a sink is one
// more term of the row sum, added where a row's sum is complete.
//
// The tokens of prompts go through the same kernel, each as a row of its own that sees the keys up to its position (for models
// whose expanded heads the prompt kernel does not take).
#include "launch.cuh"
#include "ptx.cuh"
#include "scalar.cuh"
#include "tmap.cuh"

namespace blitz {

constexpr int kLaThreads = 224;       // softmax warps 0-3, S warp, load warp, O warp
constexpr int kLaMaxHeads = 64;       // heads of an item
constexpr int kLaMaxRank = 512;
constexpr int kLaMaxStages = 8;
constexpr int kLaMaxBatch = 4096;
constexpr int kLaMaxCtas = 160;
constexpr int kLaSmem = 227 * 1024;

struct LatentParams {
  const int32_t *indices, *indptr, *last_page_len;
  const int32_t *pos, *tok_indptr;  // rows are tokens of prompts: their positions, and the first tokens of `rows` sequences
  int rows, first_token;            // (else null: a row per sequence)
  void* out;                    // [batch][out_stride], head h's rank columns from h * rank on
  const void* gate;             // [batch][gate_stride], or null
  const void* sink;             // [heads] in the activation type, or null
  int window;                   // a row sees the last `window` positions (0: all)
  int64_t out_stride, gate_stride;
  float *part_o, *part_lse;     // [grid][2][group][rank], [grid][2][group]
  int* blocks_before;           // [batch + 1], for the merge
  int batch, heads, group, subs, rank, slabs, steps, stages, q_bufs, page_shift, max_pages, box_shift, oob_row, static_table;
  float scale_log2;
  int* status;
};

// A CTA's share of the blocks as pieces of sequences.  Blocks are numbered sequence by sequence, all blocks of one head group
// before the next one's; pref[b] counts the blocks of a head group before sequence b.
struct LaPiece {
  int b, sub, beg, end, blocks;  // blocks [beg, end) of the sequence's `blocks`
};
struct LaWalk {
  const int* pref;
  int subs, x, hi, b;
  // share: first block, end, sequence of the first block
  __device__ __forceinline__ LaWalk(const int* pref_, int subs_, const int* share)
      : pref(pref_), subs(subs_), x(share[0]), hi(share[1]), b(share[2]) {}
  __device__ __forceinline__ bool next(LaPiece& q) {
    if (x >= hi) return false;
    while (pref[b + 1] * subs <= x) ++b;
    const int n = pref[b + 1] - pref[b], rem = x - pref[b] * subs;
    q.b = b;
    q.blocks = n;
    q.sub = rem / n;
    q.beg = rem - q.sub * n;
    q.end = min(n, q.beg + (hi - x));
    x += q.end - q.beg;
    return true;
  }
};

// Blocks of the next piece, 0 at the end; the same in every lane, and known to be so.
__device__ __forceinline__ int la_next(LaWalk& w) {
  LaPiece q;
  const int n = w.next(q) ? q.end - q.beg : 0;
  return __shfl_sync(0xffffffffu, n, 0);
}

__device__ __forceinline__ void la_sync() { asm volatile("bar.sync 1, 128;" ::: "memory"); }
// Whether the predicate holds for any of the 128 softmax threads (a barrier).
__device__ __forceinline__ bool la_any(bool v) {
  uint32_t r;
  asm volatile(
      "{\n\t"
      ".reg .pred p, q;\n\t"
      "setp.ne.u32 p, %1, 0;\n\t"
      "barrier.cta.red.or.pred q, 1, 128, p;\n\t"
      "selp.b32 %0, 1, 0, q;\n\t"
      "}\n"
      : "=r"(r)
      : "r"(v ? 1u : 0u)
      : "memory");
  return r != 0;
}
// order-preserving map of a float to a signed integer, and back
__device__ __forceinline__ int la_key(float x) {
  const int i = __float_as_int(x);
  return i ^ ((i >> 31) & 0x7fffffff);
}
__device__ __forceinline__ float la_unkey(int k) { return __int_as_float(k ^ ((k >> 31) & 0x7fffffff)); }

// v[i] of every lane, i < 32: lane i receives the sum over the lanes.
__device__ __forceinline__ float la_transpose_sum(float (&v)[32], int lane) {
#pragma unroll
  for (int o = 16; o > 0; o >>= 1) {
    const bool up = lane & o;
#pragma unroll
    for (int i = 0; i < o; ++i) {
      const float give = up ? v[i] : v[i + o], keep = up ? v[i + o] : v[i];
      v[i] = keep + __shfl_xor_sync(0xffffffffu, give, o);
    }
  }
  return v[0];
}

template <typename T, int KT, int NH>
__global__ void __launch_bounds__(kLaThreads, 1)
attn_latent_kernel(const __grid_constant__ CUtensorMap tmap_q, const __grid_constant__ CUtensorMap tmap_k, const LatentParams p) {
  constexpr uint32_t kFmt = std::is_same<T, __nv_bfloat16>::value ? 1u : 0u;
  constexpr int KB = KT * 128;  // bytes of a slab of 64 columns of a key block
  constexpr int QB = NH * 128;  // the same of Q
  constexpr int PB = KT * 128;  // bytes of P: a row of up to 64 heads per key
  constexpr int kSoft = KT / 32;  // warps with keys
  constexpr float kRescaleAt = std::is_same<T, __nv_bfloat16>::value ? 40.f : 8.f;  // log2 units
  extern __shared__ uint8_t smem_raw[];
  const uint32_t raw_addr = ptx::smem_u32(smem_raw);
  uint8_t* smem = smem_raw + (((raw_addr + 1023u) & ~1023u) - raw_addr);
  uint8_t* sQ = smem;                                    // [q_bufs]
  uint8_t* sK = sQ + p.q_bufs * p.slabs * QB;            // [stages]; instructions read up to a slab behind a block's end
  uint8_t* sP = sK + p.stages * p.slabs * KB;            // [2]
  float* s_red = reinterpret_cast<float*>(sP + 2 * PB);  // [4][NH]
  float* s_ref = s_red + 4 * NH;                         // [NH] the maximum probabilities refer to, log2 units
  float* s_fac = s_ref + NH;                             // [NH] rescaling, or 1 / row sum
  uint64_t* bars = reinterpret_cast<uint64_t*>(s_fac + NH);
  uint64_t* q_full = bars;         // [q_bufs] per piece
  uint64_t* q_empty = bars + 2;    // [q_bufs]
  uint64_t* s_full = bars + 4;     // [2] per block
  uint64_t* p_ready = bars + 6;    // [2]
  uint64_t* pv_done = bars + 8;    // [2]
  uint64_t* o_full = bars + 10;    // per piece
  uint64_t* o_free = bars + 11;
  uint64_t* k_full = bars + 12;    // [stages]
  uint64_t* k_empty = k_full + kLaMaxStages;
  uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(k_empty + kLaMaxStages);
  volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
  int* s_share = reinterpret_cast<int*>(tmem_slot + 2);  // [4] this CTA's first block, end, sequence of the first
  int* s_sums = s_share + 4;                             // [128] blocks of 32 sequences
  int* s_pref = s_sums + kLaMaxBatch / 32;               // [batch + 1] blocks before a sequence
  int* s_page = s_pref + p.batch + 1;                   // [batch] its first page entry
  int* s_len = s_page + p.batch;                        // [batch]
  const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  constexpr int kWarps = kLaThreads / 32;

  if (threadIdx.x == 0) {
    for (int i = 0; i < 2; ++i) {
      ptx::mbar_init(&q_full[i], 1);
      ptx::mbar_init(&q_empty[i], 1);
      ptx::mbar_init(&s_full[i], 1);
      ptx::mbar_init(&p_ready[i], KT);
      ptx::mbar_init(&pv_done[i], 1);
    }
    ptx::mbar_init(o_full, 1);
    ptx::mbar_init(o_free, 128);
    for (int i = 0; i < p.stages; ++i) {
      ptx::mbar_init(&k_full[i], 1);
      ptx::mbar_init(&k_empty[i], 1);
    }
    *abort_flag = 0;
    ptx::fence_mbar_init();
    ptx::tma_prefetch_desc(&tmap_q);
    ptx::tma_prefetch_desc(&tmap_k);
  }
  // query rows behind the last head stay zero: their scores are zero and ask for no rescaling
  for (int i = threadIdx.x; i < p.q_bufs * p.slabs * QB / 16; i += kLaThreads) reinterpret_cast<uint4*>(sQ)[i] = make_uint4(0, 0, 0, 0);
  ptx::fence_proxy_async_smem();
  if (warp == 4) {
    ptx::tmem_alloc(tmem_slot, 512);
    ptx::tmem_relinquish();
  }
  // the work list; with a page table that no running kernel writes, while the previous kernel still runs
  if (!p.static_table) ptx::griddep_wait();
  auto first_key = [&](int len) { return p.window > 0 ? max(0, len - p.window) : 0; };
  auto first_block = [&](int len) { return first_key(len) / KT; };
  const int chunks32 = (p.batch + 31) / 32;
  for (int i = warp; i < chunks32; i += kWarps) {  // sums over 32 sequences
    const int b = i * 32 + lane;
    int v = 0;
    if (b < p.batch) {
      const int row = p.pos ? row_of_token(p.tok_indptr, p.rows, p.first_token + b) : b;
      const int first = p.indptr[row], npages = p.indptr[row + 1] - first;
      int len = 0;
      if (npages > 0) len = p.pos ? min(p.pos[b] + 1, npages << p.page_shift) : ((npages - 1) << p.page_shift) + p.last_page_len[b];
      s_page[b] = first;
      s_len[b] = len;
      v = (len + KT - 1) / KT - first_block(len);
    }
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
      const int u = __shfl_up_sync(0xffffffffu, v, o);
      if (lane >= o) v += u;
    }
    if (b < p.batch) s_pref[b + 1] = v;
    if (lane == 31) s_sums[i] = v;
  }
  if (threadIdx.x == 0) s_pref[0] = 0;
  __syncthreads();
  for (int i = warp; i < chunks32; i += kWarps) {
    int before = 0;
    for (int k = lane; k < i; k += 32) before += s_sums[k];
    before = __reduce_add_sync(0xffffffffu, before);
    if (i * 32 + lane < p.batch) s_pref[i * 32 + lane + 1] += before;
  }
  __syncthreads();
  {
    const int64_t total = s_pref[p.batch] * p.subs;
    const int x = static_cast<int>(total * blockIdx.x / gridDim.x), hi = static_cast<int>(total * (blockIdx.x + 1) / gridDim.x);
    if (threadIdx.x == 0) {
      s_share[0] = x;
      s_share[1] = hi;
    }
    for (int b = threadIdx.x; b < p.batch; b += kLaThreads)
      if (s_pref[b] * p.subs <= x && x < s_pref[b + 1] * p.subs) s_share[2] = b;
  }
  ptx::tc_fence_before_sync();
  __syncthreads();
  ptx::tc_fence_after_sync();
  ptx::griddep_launch_dependents();
  if (warp != 5) ptx::griddep_wait();  // (the load warp looks its first rows up before)
  if (blockIdx.x == 0 && warp < 4)
    for (int b = threadIdx.x; b <= p.batch; b += 128) p.blocks_before[b] = s_pref[b];
  const uint32_t tmem_base = __shfl_sync(0xffffffffu, *tmem_slot, 0);
  const int chunks = (p.rank + 127) / 128;     // of value columns
  const uint32_t tmem_O = tmem_base + 2 * NH;  // S buffers at + 0 and + NH; chunk c of O at tmem_O + c * NH
  auto wait = [&](uint64_t* bar, uint32_t parity) { return ptx::bounded_mbar_wait(bar, parity, abort_flag); };
  auto all_wait = [&](uint64_t* bar, uint32_t parity) { return __all_sync(0xffffffffu, wait(bar, parity)) != 0; };

  if (warp == 5) {
    // ------------------------------------------------------------ load warp
    const int bt = 1 << p.box_shift;
    const bool mine = lane < (KT >> p.box_shift);
    auto warp_wait = [&](uint64_t* bar, uint32_t parity) {
      int ok = 1;
      if (lane == 0) ok = wait(bar, parity) ? 1 : 0;
      return __shfl_sync(0xffffffffu, ok, 0) != 0;
    };
    auto box_row = [&](const LaPiece& q, int blk) {  // this lane's first row of a block in the pool
      const int tok = (first_block(s_len[q.b]) + blk) * KT + lane * bt, slot = tok >> p.page_shift;
      if (!mine || tok >= s_len[q.b]) return p.oob_row;  // past the pool: the box arrives as zeros
      int page = p.indices[s_page[q.b] + slot];
      if (page < 0 || page >= p.max_pages) {
        if (p.status) atomicCAS(p.status, 0, kStatusBadIndex);
        page = 0;
      }
      return (page << p.page_shift) + (tok & ((1 << p.page_shift) - 1));
    };
    LaWalk walk(s_pref, p.subs, s_share);
    LaPiece q, qn;
    bool ok = true, more = walk.next(q);
    int stage = 0, qb = 0;
    uint32_t phase = 1, q_phase = 1;  // a buffer's first round needs no wait (the other parity counts as passed)
    int row = more ? box_row(q, q.beg) : 0;
    ptx::griddep_wait();
    while (ok && more) {
      bool more_next = false;
      for (int blk = q.beg; blk < q.end && ok; ++blk) {
        ok = warp_wait(&k_empty[stage], phase);
        if (!ok) break;
        if (lane == 0) ptx::mbar_expect_tx(&k_full[stage], static_cast<uint32_t>(p.slabs) * KB);
        __syncwarp();
        if (mine)
          for (int s = 0; s < p.slabs; ++s)
            ptx::tma_load_2d(sK + (stage * p.slabs + s) * KB + lane * bt * 128, &tmap_k, &k_full[stage], s * 64, row);
        if (++stage == p.stages) {
          stage = 0;
          phase ^= 1u;
        }
        if (blk == q.beg) {
          ok = warp_wait(&q_empty[qb], q_phase);
          if (!ok) break;
          if (lane == 0) {
            ptx::mbar_expect_tx(&q_full[qb], static_cast<uint32_t>(p.slabs * p.group) * 128u);
            for (int s = 0; s < p.slabs; ++s)
              ptx::tma_load_3d(sQ + (qb * p.slabs + s) * QB, &tmap_q, &q_full[qb], s * 64, q.sub * p.group, q.b);
          }
          if (++qb == p.q_bufs) {
            qb = 0;
            q_phase ^= 1u;
          }
          more_next = walk.next(qn);
        }
        // the next block's rows are looked up a block ahead of their use
        row = blk + 1 < q.end ? box_row(q, blk + 1) : more_next ? box_row(qn, qn.beg) : 0;
      }
      q = qn;
      more = more_next;
    }
    if (!ok && lane == 0 && p.status) atomicCAS(p.status, 0, kStatusTimeoutProducer);
  } else if (warp == 4) {
    // ------------------------------------------------------------ S
    const bool leader = ptx::elect_one();
    constexpr uint32_t idesc = ptx::make_idesc_f16(kFmt, 0u, 0u, 128, NH);
    LaWalk walk(s_pref, p.subs, s_share);
    int stage = 0, qb = 0;
    uint32_t phase = 0, q_phase = 0, g = 0;
    bool ok = true;
    for (int n = la_next(walk); n > 0 && ok; n = la_next(walk)) {
      ok = all_wait(&q_full[qb], q_phase);
      for (int i = 0; i < n && ok; ++i, ++g) {
        ok = all_wait(&k_full[stage], phase);
        if (ok && g >= 2) ok = all_wait(&p_ready[g & 1], ((g >> 1) - 1) & 1);  // the scores of two blocks ago have been read
        if (!ok) break;
        ptx::tc_fence_after_sync();
        uint64_t a = ptx::make_smem_desc(ptx::smem_u32(sK + stage * p.slabs * KB), 16, 1024, ptx::kLayoutSw128);
        uint64_t b = ptx::make_smem_desc(ptx::smem_u32(sQ + qb * p.slabs * QB), 16, 1024, ptx::kLayoutSw128);
        const uint32_t d = tmem_base + (g & 1) * NH;
        for (int s = 0; s < p.steps / 4; ++s) {
#pragma unroll
          for (int k = 0; k < 4; ++k)
            if (leader) ptx::umma_f16_ss(d, a + k * 2, b + k * 2, idesc, (s | k) != 0 ? 1u : 0u);
          a += KB / 16;
          b += QB / 16;
        }
        for (int s = p.steps & ~3; s < p.steps; ++s) {
          if (leader) ptx::umma_f16_ss(d, a, b, idesc, s != 0 ? 1u : 0u);
          a += 2;
          b += 2;
        }
        if (leader) ptx::umma_commit(&s_full[g & 1]);
        if (++stage == p.stages) {
          stage = 0;
          phase ^= 1u;
        }
      }
      if (leader) ptx::umma_commit(&q_empty[qb]);
      if (++qb == p.q_bufs) {
        qb = 0;
        q_phase ^= 1u;
      }
    }
    if (!ok && leader && p.status) atomicCAS(p.status, 0, kStatusTimeoutMma);
  } else if (warp == 6) {
    // ------------------------------------------------------------ O += V^T P
    const bool leader = ptx::elect_one();
    constexpr uint32_t idesc = ptx::make_idesc_f16(kFmt, 1u, 1u, 128, NH);
    LaWalk walk(s_pref, p.subs, s_share);
    int stage = 0;
    uint32_t g = 0, o_phase = 1;  // (the first piece needs no wait)
    bool ok = true;
    for (int n = la_next(walk); n > 0 && ok; n = la_next(walk), o_phase ^= 1u) {
      ok = all_wait(o_free, o_phase);  // the last piece's O has been read
      for (int i = 0; i < n && ok; ++i, ++g) {
        ok = all_wait(&p_ready[g & 1], (g >> 1) & 1);
        if (!ok) break;
        ptx::tc_fence_after_sync();
        for (int c = 0; c < chunks; ++c) {
          // (value columns behind the last one are rows of O that nobody reads)
          const uint64_t a = ptx::make_smem_desc(ptx::smem_u32(sK + (stage * p.slabs + c * 2) * KB), KB, 1024, ptx::kLayoutSw128);
          const uint64_t b = ptx::make_smem_desc(ptx::smem_u32(sP + (g & 1) * PB), PB, 1024, ptx::kLayoutSw128);
#pragma unroll
          for (int k = 0; k < KT / 16; ++k)
            if (leader) ptx::umma_f16_ss(tmem_O + c * NH, a + k * 128, b + k * 128, idesc, (i | k) != 0 ? 1u : 0u);
        }
        if (leader) {
          ptx::umma_commit(&k_empty[stage]);
          ptx::umma_commit(&pv_done[g & 1]);
          if (i == n - 1) ptx::umma_commit(o_full);
        }
        if (++stage == p.stages) stage = 0;
      }
    }
    if (!ok && leader && p.status) atomicCAS(p.status, 0, kStatusTimeoutMma);
  } else {
    // ------------------------------------------------------------ softmax warps: thread = key, then thread = value column
    const int r = warp * 32 + lane;
    const uint32_t lane_addr = static_cast<uint32_t>(warp * 32) << 16;
    const bool soft = warp < kSoft;
    LaWalk walk(s_pref, p.subs, s_share);
    LaPiece q;
    bool ok = true;  // of this thread; the four warps keep meeting at the barriers
    uint32_t g = 0, n = 0;
    const uint32_t tO = tmem_O + lane_addr;
    // a piece's output: to the result, or where the partial sums of incomplete pieces go
    auto emit = [&](auto* row) {
      using U = std::remove_pointer_t<decltype(row)>;
#pragma unroll 1
      for (int c = 0; c < chunks; ++c) {
        const int d = c * 128 + r;
#pragma unroll 1
        for (int h0 = 0; h0 < NH; h0 += 16) {
          uint32_t o[16];
          ptx::tmem_ld_32x16(tO + c * NH + h0, o);
          ptx::tmem_ld_wait();
          if (c == chunks - 1 && h0 == NH - 16) {  // the next piece may overwrite O
            ptx::tc_fence_before_sync();
            ptx::mbar_arrive(o_free);
          }
          if (d >= p.rank || h0 >= p.group) continue;
          U* dst = row + h0 * p.rank + d;
          const bool all = h0 + 16 <= p.group;
#pragma unroll
          for (int i = 0; i < 16; i += 4) {
            const float4 f = *reinterpret_cast<const float4*>(s_fac + h0 + i);
            const float y[4] = {__uint_as_float(o[i]) * f.x, __uint_as_float(o[i + 1]) * f.y, __uint_as_float(o[i + 2]) * f.z,
                                __uint_as_float(o[i + 3]) * f.w};
#pragma unroll
            for (int k = 0; k < 4; ++k) {
              if (all || h0 + i + k < p.group) stf<U>(dst, y[k]);
              dst += p.rank;
            }
          }
        }
      }
    };
    for (; walk.next(q); ++n) {
      const int len = s_len[q.b], head0 = q.sub * p.group;
      const int key0 = first_block(len) * KT, lo = first_key(len) - key0;  // position of block 0's first key; first visible key there
      // of the thread's keys, per head: row sum, and the references (the same in all threads; for many heads in shared memory)
      constexpr bool kRefRegs = NH <= 32;
      float l[NH], ref[kRefRegs ? NH : 1] = {};
#pragma unroll
      for (int h = 0; h < NH; ++h) l[h] = 0.f;
      auto reference = [&](int h) { return kRefRegs ? ref[kRefRegs ? h : 0] : s_ref[h]; };
      for (int blk = q.beg; blk < q.end; ++blk, ++g) {
        float x[NH];  // scores relative to the references, log2 units
        const bool first = blk == q.beg;
        bool grow = false;
        if (soft) {
          if (ok) ok = wait(&s_full[g & 1], (g >> 1) & 1);
          ptx::tc_fence_after_sync();
          const uint32_t tS = tmem_base + (g & 1) * NH + lane_addr;
#pragma unroll
          for (int i = 0; i < NH; i += 16) {
            uint32_t v[16];
            ptx::tmem_ld_32x16(tS + i, v);
            ptx::tmem_ld_wait();
#pragma unroll
            for (int k = 0; k < 16; ++k) x[i + k] = fmaf(__uint_as_float(v[k]), p.scale_log2, first ? 0.f : -reference(i + k));
          }
          if ((key0 + blk * KT + KT > len && key0 + blk * KT + r >= len) || blk * KT + r < lo) {
#pragma unroll
            for (int h = 0; h < NH; ++h) x[h] = -INFINITY;
          }
          if (first) {  // the first visible key's scores are the references
            if (r == (blk == 0 ? lo : 0)) {
#pragma unroll
              for (int h = 0; h < NH; ++h) s_ref[h] = x[h];
            }
            asm volatile("bar.sync 2, %0;" ::"n"(KT) : "memory");
#pragma unroll
            for (int h = 0; h < NH; ++h) {
              if (kRefRegs) ref[kRefRegs ? h : 0] = s_ref[h];
              x[h] -= s_ref[h];
            }
          }
          float mx = -INFINITY;
#pragma unroll
          for (int h = 0; h < NH; h += 2) mx = ptx::fmax3(mx, x[h], x[h + 1]);
          grow = mx > kRescaleAt;
        }
        if (la_any(grow)) {
          // new references: the maximum over the block and over the old ones
          if (soft) {
            int mine = 0;
#pragma unroll
            for (int h = 0; h < NH; ++h) {
              const int k = __reduce_max_sync(0xffffffffu, la_key(x[h]));
              if ((h & 31) == lane) mine = k;
              if ((h & 31) == 31 || h == NH - 1)
                if (lane <= (h & 31)) s_red[warp * NH + (h & ~31) + lane] = la_unkey(mine);
            }
          }
          la_sync();
          if (r < NH) {
            float m = 0.f;
#pragma unroll
            for (int w = 0; w < kSoft; ++w) m = fmaxf(m, s_red[w * NH + r]);
            s_fac[r] = ptx::ex2_approx(-m);
            s_ref[r] += m;
            s_red[r] = m;  // (this thread has read the column)
          }
          la_sync();
#pragma unroll
          for (int h = 0; h < NH; ++h) {
            x[h] -= s_red[h];
            if (kRefRegs) ref[kRefRegs ? h : 0] = s_ref[h];
          }
          if (!first) {
            if (ok) ok = wait(&pv_done[(g - 1) & 1], ((g - 1) >> 1) & 1);  // O is settled
            ptx::tc_fence_after_sync();
#pragma unroll
            for (int h = 0; h < NH; ++h) l[h] *= s_fac[h];
#pragma unroll 1
            for (int c = 0; c < chunks * NH; c += 16) {
              uint32_t o[16];
              ptx::tmem_ld_32x16(tO + c, o);
              ptx::tmem_ld_wait();
#pragma unroll
              for (int i = 0; i < 16; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * s_fac[(c + i) % NH]);
              ptx::tmem_st_32x16(tO + c, o);
            }
            ptx::tmem_st_wait();
            ptx::tc_fence_before_sync();
            la_sync();
          }
        }
        if (soft) {
          if (g >= 2 && ok) ok = wait(&pv_done[g & 1], ((g >> 1) - 1) & 1);  // P of two blocks ago has been read
          uint8_t* prow = sP + (g & 1) * PB + r * 128;
#pragma unroll
          for (int h = 0; h < NH; h += 8) {
            float e[8];
#pragma unroll
            for (int i = 0; i < 8; ++i) {
              e[i] = ptx::ex2_approx(x[h + i]);
              l[h + i] += e[i];
            }
            *reinterpret_cast<uint4*>(prow + (((h >> 3) ^ (r & 7)) << 4)) = pack8<T>(e);
          }
          ptx::fence_proxy_async_smem();
          ptx::tc_fence_before_sync();
          ptx::mbar_arrive(&p_ready[g & 1]);
        }
      }
      // row sums: over a warp's keys, then over the warps
      if (soft) {
#pragma unroll
        for (int h0 = 0; h0 < NH; h0 += 32) {
          float t[32];
#pragma unroll
          for (int i = 0; i < 32; ++i) t[i] = h0 + i < NH ? l[(h0 + i) % NH] : 0.f;
          const float sum = la_transpose_sum(t, lane);
          if (h0 + lane < NH) s_red[warp * NH + h0 + lane] = sum;
        }
      }
      la_sync();
      const bool whole = q.beg == 0 && q.end == q.blocks;
      const int64_t part = (static_cast<int64_t>(blockIdx.x) * 2 + (n > 0)) * p.group;
      if (r < p.group) {
        float sum = 0.f;
#pragma unroll
        for (int w = 0; w < kSoft; ++w) sum += s_red[w * NH + r];
        if (whole && p.sink != nullptr)
          sum += exp2f(fminf(to_f<T>(reinterpret_cast<const T*>(p.sink)[head0 + r]) * 1.4426950408889634f - s_ref[r], 120.f));
        float f = sum > 0.f ? 1.f / sum : 0.f;
        if (whole && p.gate != nullptr) f *= sigmoid_f(to_f<T>(reinterpret_cast<const T*>(p.gate)[q.b * p.gate_stride + head0 + r]));
        s_fac[r] = f;
        if (!whole) p.part_lse[part + r] = s_ref[r] + log2f(sum);
      }
      la_sync();
      if (ok) ok = wait(o_full, n & 1);
      ptx::tc_fence_after_sync();
      if (whole) emit(reinterpret_cast<T*>(p.out) + q.b * p.out_stride + static_cast<int64_t>(head0) * p.rank);
      else emit(p.part_o + part * p.rank);
      if (la_any(!ok)) {  // (also: s_fac, s_red and s_ref have been read)
        ok = false;
        break;
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
// keys become zeros.  `per` warps per head (1, or all eight where there are few rows).
template <typename T>
__global__ void __launch_bounds__(256) attn_latent_merge_kernel(const LatentParams p, int ctas, int per) {
  ptx::griddep_launch_dependents();
  ptx::griddep_wait();
  extern __shared__ float s_acc[];  // [8][rank], several warps per head only
  const int b = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
  const int head = blockIdx.y * (8 / per) + warp / per, share = warp % per;
  if (head >= p.heads) return;  // (with several warps per head: all of a block or none)
  const int before = p.blocks_before[b], blocks = p.blocks_before[b + 1] - before, all = p.blocks_before[p.batch] * p.subs;
  const int64_t total = all;
  T* dst = reinterpret_cast<T*>(p.out) + b * p.out_stride + static_cast<int64_t>(head) * p.rank;
  if (blocks == 0) {
    if (share == 0)
      for (int c = lane; c < p.rank; c += 32) stf<T>(dst + c, 0.f);
    return;
  }
  const int beg = before * p.subs + head / p.group * blocks;
  auto cta_of = [&](int block) { return static_cast<int>(((block + 1) * static_cast<int64_t>(ctas) - 1) / total); };
  const int c0 = cta_of(beg), c1 = cta_of(beg + blocks - 1);
  if (c0 == c1) return;  // one CTA has done all of it
  constexpr int kRounds = kLaMaxCtas / 32;
  float w[kRounds];
  int at[kRounds];
  float m = -INFINITY, sum = 0.f;
#pragma unroll
  for (int i = 0; i < kRounds; ++i) {
    w[i] = -INFINITY;
    at[i] = -1;
    if (c0 + i * 32 > c1) continue;
    const int c = c0 + i * 32 + lane, lo = static_cast<int>(total * c / ctas);
    // the piece is its CTA's first one unless the CTA's share begins before this sequence; with more CTAs than blocks some
    // have none
    if (c <= c1 && lo < static_cast<int>(total * (c + 1) / ctas)) {
      at[i] = (c * 2 + (lo < beg ? 1 : 0)) * p.group + head % p.group;
      w[i] = p.part_lse[at[i]];
    }
    m = fmaxf(m, w[i]);
  }
  m = warp_max(m);
  const float sink = p.sink ? to_f<T>(reinterpret_cast<const T*>(p.sink)[head]) * 1.4426950408889634f : -INFINITY;
  m = fmaxf(m, sink);
#pragma unroll
  for (int i = 0; i < kRounds; ++i) {
    w[i] = exp2f(w[i] - m);
    sum += w[i];
  }
  sum = warp_sum(sum) + exp2f(sink - m);
  const float gate = p.gate ? sigmoid_f(to_f<T>(reinterpret_cast<const T*>(p.gate)[b * p.gate_stride + head])) : 1.f;
  float acc[kLaMaxRank / 32] = {};
#pragma unroll
  for (int i = 0; i < kRounds; ++i) {
    const int cnt = min(32, c1 - (c0 + i * 32) + 1);
#pragma unroll 2
    for (int j = share; j < cnt; j += per) {
      const int a = __shfl_sync(0xffffffffu, at[i], j);
      const float wj = __shfl_sync(0xffffffffu, w[i], j);
      if (a < 0) continue;
      const float* src = p.part_o + static_cast<int64_t>(a) * p.rank;
#pragma unroll
      for (int k = 0; k < kLaMaxRank / 32; ++k)
        if (k * 32 + lane < p.rank) acc[k] += wj * src[k * 32 + lane];
    }
  }
  const float f = gate / sum;
  if (per == 1) {
#pragma unroll
    for (int k = 0; k < kLaMaxRank / 32; ++k)
      if (k * 32 + lane < p.rank) stf<T>(dst + k * 32 + lane, acc[k] * f);
    return;
  }
#pragma unroll
  for (int k = 0; k < kLaMaxRank / 32; ++k)
    if (k * 32 + lane < p.rank) s_acc[warp * p.rank + k * 32 + lane] = acc[k];
  __syncthreads();
  for (int c = threadIdx.x; c < p.rank; c += blockDim.x) {
    float v = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) v += s_acc[i * p.rank + c];
    stf<T>(dst + c, v * f);
  }
}

struct LatentPlan {
  int kt, group, nh, slabs, stages, q_bufs;
  size_t smem;
};
// How the heads are grouped and how tall a key block is: as many heads as possible; blocks of 64 keys, whose stages are more, or,
// with few rows and heads, blocks of 128, which are through sooner; queries double buffered if that leaves room.
static bool latent_plan(int batch, int heads, int width, int rank, int page_size, int kt_hint, LatentPlan* out) {
  if (batch < 1 || batch > kLaMaxBatch || heads < 1 || rank < 8 || rank > kLaMaxRank || width < rank || ((width | rank) & 7)) return false;
  if (page_size < 8 || (page_size & (page_size - 1)) != 0) return false;
  LatentPlan pl;
  pl.slabs = (width + 63) / 64;
  for (int groups = 1; groups <= heads; ++groups) {
    if (heads % groups || heads / groups > kLaMaxHeads) continue;
    pl.group = heads / groups;
    pl.nh = pl.group <= 16 ? 16 : pl.group <= 32 ? 32 : 64;
    const int fixed = 1024 + 6 * pl.nh * 4 + (12 + 2 * kLaMaxStages) * 8 + 8 + 16 + kLaMaxBatch / 32 * 4 + (3 * batch + 1) * 4;
    const int tall_first = pl.nh <= 32 && batch < 64;
    for (int i = 0; i < 2; ++i) {
      const int kt = (i == 0) == (tall_first != 0) ? 128 : 64;
      if (kt_hint && kt != kt_hint) continue;
      for (int bufs = 2; bufs >= 1; --bufs) {
        const int rest = fixed + 2 * kt * 128 + bufs * pl.slabs * pl.nh * 128, stage = pl.slabs * kt * 128;
        const int stages = (kLaSmem - rest) / stage;
        if (rest > kLaSmem || stages < (bufs == 2 && kt == 64 ? 3 : 2)) continue;
        pl.kt = kt;
        pl.q_bufs = bufs;
        pl.stages = stages < kLaMaxStages ? stages : kLaMaxStages;
        pl.smem = rest + (size_t)pl.stages * stage;
        *out = pl;
        return true;
      }
    }
  }
  return false;
}

}  // namespace blitz

extern "C" {
using namespace blitz;

int blitz_attn_latent_supported(int batch, int heads, int width, int rank, int page_size) {
  LatentPlan pl;
  return latent_plan(batch, heads, width, rank, page_size, 0, &pl) ? 1 : 0;
}

// Bytes of fp32 scratch for the partial sums, whatever the batch is.
int64_t blitz_attn_latent_workspace_bytes(int heads, int rank) {
  const int group = heads < kLaMaxHeads ? heads : kLaMaxHeads;
  return (int64_t)device_sm_count() * 2 * group * (rank + 1) * (int64_t)sizeof(float) + (kLaMaxBatch + 1) * (int64_t)sizeof(int);
}

// q [batch][q_stride]: heads of `width` columns; pool [max_pages][page_size][width], the first `rank` columns are the values;
// out [batch][out_stride]: heads of `rank` columns.  width, rank: multiples of 8, rank up to 512; page_size: a power of two >= 8;
// gate [batch][gate_stride] or null; window (0 = none) and sink ([heads] or null): see the top of the file.  A row without pages gives zeros.  kt_hint: keys per block, 0 = choose, else 64 or 128.
// static_table: no kernel still running in the stream writes indices, indptr, last_page_len, pos or tok_indptr.
// pos [batch], tok_indptr [rows + 1] (both or none): the batch are tokens first_token .. of `rows` sequences, whose pages indptr
// [rows + 1] names; each sees the keys up to its position.  last_page_len is not read then.
int blitz_attn_latent(const void* q, int64_t q_stride, const void* pool, const int32_t* indices, const int32_t* indptr,
                      const int32_t* last_page_len, const int32_t* pos, const int32_t* tok_indptr, int rows, int first_token, void* out, int64_t out_stride, void* workspace, int batch, int heads, int width, int rank,
                      int page_size, int max_pages, float sm_scale, int window, const void* sink, const void* gate, int64_t gate_stride, int kt_hint, int static_table, int* status, int dtype,
                      cudaStream_t stream) {
  if (batch <= 0) return 0;
  LatentPlan pl;
  if (!latent_plan(batch, heads, width, rank, page_size, kt_hint, &pl) || workspace == nullptr || max_pages < 1 || window < 0) return -1;
  if ((pos == nullptr) != (tok_indptr == nullptr) || (pos && rows < 1)) return -1;
  if ((q_stride & 7) || (reinterpret_cast<uintptr_t>(workspace) & 15)) return -1;
  const int sms = device_sm_count() < kLaMaxCtas ? device_sm_count() : kLaMaxCtas;
  const int bt = page_size < 64 ? page_size : 64;
  CUtensorMap tq, tk;
  if (!get_tmap_3d(&tq, q, (uint64_t)width, (uint64_t)heads, (uint64_t)batch, (uint64_t)width * 2, (uint64_t)q_stride * 2, 64,
                   (uint32_t)pl.group, 1))
    return -2;
  if (!get_tmap_2d(&tk, pool, (uint64_t)width, (uint64_t)max_pages * page_size, (uint64_t)width * 2, 64, (uint32_t)bt)) return -2;
  LatentParams p;
  p.indices = indices; p.indptr = indptr; p.last_page_len = last_page_len;
  p.window = window; p.sink = sink;
  p.pos = pos; p.tok_indptr = tok_indptr; p.rows = rows; p.first_token = first_token; p.out = out; p.gate = gate;
  p.out_stride = out_stride; p.gate_stride = gate_stride;
  p.batch = batch; p.heads = heads; p.group = pl.group; p.subs = heads / pl.group; p.rank = rank;
  p.slabs = pl.slabs; p.steps = (width + 15) / 16; p.stages = pl.stages; p.q_bufs = pl.q_bufs;
  p.page_shift = __builtin_ctz(page_size); p.box_shift = __builtin_ctz(bt); p.static_table = static_table;
  p.max_pages = max_pages; p.oob_row = max_pages * page_size;
  p.part_o = reinterpret_cast<float*>(workspace);
  p.part_lse = p.part_o + (int64_t)sms * 2 * pl.group * rank;
  p.blocks_before = reinterpret_cast<int*>(p.part_lse + (int64_t)sms * 2 * pl.group);
  const int per = (int64_t)batch * heads >= 8 * (int64_t)sms ? 1 : 8;  // warps per head in the merge
  p.scale_log2 = sm_scale * 1.4426950408889634f; p.status = status;
  auto go = [&](auto type, auto keys, auto cols) -> int {
    using T = decltype(type);
    constexpr int KT = decltype(keys)::value, NH = decltype(cols)::value;
    static PerDeviceOnce once;
    cudaError_t e = once.run([] { return cudaFuncSetAttribute(attn_latent_kernel<T, KT, NH>, cudaFuncAttributeMaxDynamicSharedMemorySize, kLaSmem); });
    if (e == cudaSuccess) e = launch_pdl(attn_latent_kernel<T, KT, NH>, dim3(sms), dim3(kLaThreads), pl.smem, stream, tq, tk, p);
    if (e == cudaSuccess) e = launch_pdl(attn_latent_merge_kernel<T>, dim3(batch, (heads * per + 7) / 8), dim3(256),
                                          per > 1 ? (size_t)8 * rank * sizeof(float) : 0, stream, p, sms, per);
    return (int)e;
  };
  auto wide = [&](auto type, auto keys) {
    return pl.nh == 16 ? go(type, keys, std::integral_constant<int, 16>{}) : pl.nh == 32 ? go(type, keys, std::integral_constant<int, 32>{})
                                                                                           : go(type, keys, std::integral_constant<int, 64>{});
  };
  auto tall = [&](auto type) {
    return pl.kt == 128 ? wide(type, std::integral_constant<int, 128>{}) : wide(type, std::integral_constant<int, 64>{});
  };
  return dtype == 1 ? tall(__nv_bfloat16{}) : tall(__half{});
}

}  // extern "C"
