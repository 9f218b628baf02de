// Entry of a layer of a model whose residual stream is kept in fp32: whatever is added to the stream before the
// layer (nothing, the token's embedding as the start of the stream, the embedding once more and a step vector at the
// start of a pass of a looped block, the rows that a mixture of experts has left for the token), then the layer's
// RMSNorm, in one kernel: one read and at most one write of the stream.
//
//   x[t] = init ? embed[id[t]] : x[t] (+ embed[id[t]]) (+ step) (+ sum_k add[add_row[t][k]])
//   out[t] = x[src(t)] / sqrt(mean(x^2) + eps) * (w_offset + w)        src(t) = rows ? rows[t] + row_offset : t
//
// A block per token; the row stays in registers between the two passes up to 8192 columns.
#include "launch.cuh"
#include "ptx.cuh"
#include "scalar.cuh"

namespace blitz {

struct StreamNormParams {
  const int32_t* ids;
  const void* embed;
  const void* step;
  const int32_t* rows;
  float* x;
  const void* w;
  void* out;
  const void* add;          // rows of the activation type, or null
  const int32_t* add_row;   // [tokens][n_add]
  int n_add;
  int hidden, vocab, init, add_embed, row_offset;
  float eps, w_offset;
  int* status;
};

constexpr int kSnKeep = 8;  // float4 groups a thread keeps

template <typename T, int VEC, bool ADD>
__global__ void stream_norm_kernel(const StreamNormParams p) {
  ptx::griddep_launch_dependents();
  ptx::griddep_wait();
  __shared__ float red[33];
  const int t = blockIdx.x;
  const int src = p.rows ? p.rows[t] + p.row_offset : t;
  float* xr = p.x + static_cast<int64_t>(src) * p.hidden;
  const T* step = reinterpret_cast<const T*>(p.step);
  const bool change = p.init || p.add_embed || step != nullptr || ADD;
  const T* er = nullptr;
  if (p.init || p.add_embed) {
    const int id = p.ids[t];
    if (id >= 0 && id < p.vocab) {
      er = reinterpret_cast<const T*>(p.embed) + static_cast<int64_t>(id) * p.hidden;
    } else if (threadIdx.x == 0 && p.status) {
      atomicCAS(p.status, 0, kStatusBadIndex);
    }
  }
  const int n = p.hidden / VEC;
  // one group of VEC columns: VEC == 1 leaves y, z, w zero
  auto load = [&](const float* q) {
    return VEC == 4 ? *reinterpret_cast<const float4*>(q) : make_float4(*q, 0.f, 0.f, 0.f);
  };
  auto add = [&](float4& a, const T* q) {
    const float4 e = VEC == 4 ? ldf4<T>(q) : make_float4(ldf<T>(q), 0.f, 0.f, 0.f);
    a.x += e.x; a.y += e.y; a.z += e.z; a.w += e.w;
  };
  const int32_t* add_row = p.add_row + static_cast<int64_t>(t) * p.n_add;
  auto read = [&](int i) {
    float4 a = p.init ? make_float4(0.f, 0.f, 0.f, 0.f) : load(xr + i * VEC);
    if (er) add(a, er + i * VEC);
    if (step) add(a, step + i * VEC);
    if (ADD)
      for (int k = 0; k < p.n_add; ++k) add(a, reinterpret_cast<const T*>(p.add) + static_cast<int64_t>(add_row[k]) * p.hidden + i * VEC);
    if (change) {
      if (VEC == 4) *reinterpret_cast<float4*>(xr + i * VEC) = a;
      else xr[i] = a.x;
    }
    return a;
  };
  auto square = [](const float4& a) { return a.x * a.x + a.y * a.y + a.z * a.z + a.w * a.w; };
  float4 keep[kSnKeep];
  float ss = 0.f;
#pragma unroll
  for (int k = 0; k < kSnKeep; ++k) {
    const int i = threadIdx.x + k * blockDim.x;
    if (i < n) {
      keep[k] = read(i);
      ss += square(keep[k]);
    }
  }
  for (int i = threadIdx.x + kSnKeep * blockDim.x; i < n; i += blockDim.x) ss += square(read(i));
  if (p.out == nullptr) return;
  ss = block_sum(ss, red);
  const float scale = rsqrtf(ss / static_cast<float>(p.hidden) + p.eps);
  const T* w = reinterpret_cast<const T*>(p.w);
  T* out = reinterpret_cast<T*>(p.out) + static_cast<int64_t>(t) * p.hidden;
  auto write = [&](int i, const float4& v) {
    if (VEC == 4) {
      const float4 g = ldf4<T>(w + i * 4);
      stf4<T>(out + i * 4, make_float4(v.x * scale * (p.w_offset + g.x), v.y * scale * (p.w_offset + g.y),
                                       v.z * scale * (p.w_offset + g.z), v.w * scale * (p.w_offset + g.w)));
    } else {
      stf<T>(out + i, v.x * scale * (p.w_offset + ldf<T>(w + i)));
    }
  };
#pragma unroll
  for (int k = 0; k < kSnKeep; ++k) {
    const int i = threadIdx.x + k * blockDim.x;
    if (i < n) write(i, keep[k]);
  }
  for (int i = threadIdx.x + kSnKeep * blockDim.x; i < n; i += blockDim.x) write(i, load(xr + i * VEC));
}

}  // namespace blitz

extern "C" {
using namespace blitz;

// x [tokens, hidden] fp32; embed / step / w / out in the activation type (dtype 0 fp16, 1 bf16, 2 fp32).  init: the
// stream starts as the tokens' embeddings; add_embed: they are added to it; step: vector added to every token (may be
// null); add: rows [.., hidden] of which token t receives the n_add rows add_row[t] (not together with `rows`); out (may be null): the normalised rows.  rows: read row rows[t] + row_offset of x for output row t.
int blitz_stream_norm(const int32_t* ids, const void* embed, const void* step, const int32_t* rows, int row_offset,
                      float* x, const void* w, void* out, const void* add, const int32_t* add_row, int n_add, int num_tokens, int hidden, int vocab, int init, int add_embed, float eps,
                      float w_offset, int* status, int dtype, cudaStream_t stream) {
  if (num_tokens <= 0) return 0;
  if (hidden <= 0 || x == nullptr || n_add < 0 || (n_add > 0 && (add == nullptr || add_row == nullptr || rows != nullptr))) return -1;
  StreamNormParams p{ids, embed, step, rows, x, w, out, add, add_row, n_add, hidden, vocab, init, add_embed, row_offset, eps, w_offset, status};
  const int n = (hidden & 3) ? hidden : hidden / 4;
  int threads = 32;
  while (threads < n && threads < (n > 1024 ? 512 : 256)) threads <<= 1;
  auto go = [&](auto type, auto vec) {
    using T = decltype(type);
    constexpr int V = decltype(vec)::value;
    return n_add > 0 ? launch_pdl(stream_norm_kernel<T, V, true>, dim3(num_tokens), dim3(threads), 0, stream, p)
                     : launch_pdl(stream_norm_kernel<T, V, false>, dim3(num_tokens), dim3(threads), 0, stream, p);
  };
  cudaError_t e = cudaSuccess;
  BLITZ_DISPATCH_DTYPE3(dtype, (e = (hidden & 3) ? go(T{}, std::integral_constant<int, 1>{}) : go(T{}, std::integral_constant<int, 4>{})));
  return (int)e;
}

}  // extern "C"
