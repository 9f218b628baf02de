"""Python entry points of the hand-written sm_100a kernels.

Each function takes CUDA tensors, launches on the current stream and returns
the output tensor.  Shapes follow the serving data layouts: activations
``[tokens, features]`` row-major, weights ``[in, out]`` row-major (the layout
the reference loads, scripts/util/make_dangertensors.py:9-30), the paged KV
cache ``[page][K|V][token][kv_head][head_dim]`` per layer.
"""
from __future__ import annotations

import ctypes
from typing import NamedTuple, Optional, Sequence, Union

import torch

from ._lib import lib, available, KernelLibraryMissing  # noqa: F401

_DT = {torch.float16: 0, torch.bfloat16: 1}
_DT3 = {torch.float16: 0, torch.bfloat16: 1, torch.float32: 2}
_status = {}


def _dt(t: torch.Tensor) -> int:
    try:
        return _DT[t.dtype]
    except KeyError:
        raise TypeError(f"kernels take fp16/bf16 tensors, got {t.dtype}") from None


def _dt3(t: torch.Tensor) -> int:
    """Element type of kernels that also run in fp32."""
    try:
        return _DT3[t.dtype]
    except KeyError:
        raise TypeError(f"kernel takes fp16/bf16/fp32 tensors, got {t.dtype}") from None


def _stream() -> ctypes.c_void_p:
    return ctypes.c_void_p(torch.cuda.current_stream().cuda_stream)


def _p(t: Optional[torch.Tensor]) -> ctypes.c_void_p:
    return ctypes.c_void_p(0 if t is None else t.data_ptr())


def _check(rc: int, what: str) -> None:
    if rc != 0:
        raise RuntimeError(f"{what} failed with code {rc}" + (
            " (argument not supported by the kernel)" if rc == -1 else
            " (TMA descriptor encoder unavailable)" if rc == -2 else ""))


class KVPair(NamedTuple):
    """Paged cache of a layer whose keys and values differ in size: [pages, page, kv_heads, dim] and [.., vdim].  (Where they
    are equal, the cache is one tensor [pages, 2, page, kv_heads, dim].)"""
    k: torch.Tensor
    v: torch.Tensor


class LatentKV(NamedTuple):
    """Paged cache of a latent attention layer: [pages, page, 1, rank + rotated dimensions].  A row is the key of every head,
    its first ``rank`` columns the value of every head, before the heads' own projections."""
    pool: torch.Tensor
    rank: int


KVLayer = Union[torch.Tensor, KVPair, LatentKV]


def _kv(kv: KVLayer):
    """(key pool, value pool, rows per page in the pools, pages, value size)"""
    if isinstance(kv, LatentKV):
        assert kv.pool.is_contiguous()
        return _p(kv.pool), _p(kv.pool), kv.pool.shape[1], kv.pool.shape[0], kv.rank
    if isinstance(kv, KVPair):
        assert kv.k.is_contiguous() and kv.v.is_contiguous() and kv.k.shape[:3] == kv.v.shape[:3]
        return _p(kv.k), _p(kv.v), kv.k.shape[1], kv.k.shape[0], kv.v.shape[3]
    assert kv.is_contiguous()
    return _p(kv), ctypes.c_void_p(kv.data_ptr() + kv.stride(1) * kv.element_size()), 2 * kv.shape[2], kv.shape[0], kv.shape[4]


def _bias(bias: Optional[torch.Tensor], q_heads: int):
    assert bias is None or (bias.is_contiguous() and bias.dim() == 2 and bias.shape[0] == q_heads)
    return _p(bias), 0 if bias is None else bias.shape[1]


def _gate(gate: Optional[torch.Tensor]):
    assert gate is None or gate.stride(1) == 1
    return _p(gate), 0 if gate is None else gate.stride(0)


def status_word(device=None) -> torch.Tensor:
    """Per-device int32 word the kernels write a non-zero code into when a bounded wait or an index check fails."""
    dev = torch.device("cuda", torch.cuda.current_device()) if device is None else torch.device(device)
    key = (dev.type, dev.index)
    if key not in _status:
        _status[key] = torch.zeros(1, dtype=torch.int32, device=dev)
    return _status[key]


def check_status(device=None, reset: bool = True) -> int:
    """Read the status word (synchronises). Raises on a non-zero code."""
    w = status_word(device)
    code = int(w.item())
    if code != 0:
        if reset:
            w.zero_()
            for _, tickets in _gemm_ws.values():  # an aborted split-K GEMM may leave tickets behind
                tickets.zero_()
            for _, flags in _pair_ws.values():
                flags.zero_()
        names = {1: "TMA producer wait timed out", 2: "MMA wait timed out", 3: "epilogue wait timed out",
                 4: "flag wait timed out", 5: "index out of range", 6: "size beyond the supported maximum"}
        raise RuntimeError(f"kernel status {code}: {names.get(code, 'unknown')}")
    return code


# ---------------------------------------------------------------------------------------------- GEMM
_EPI = {"store": 0, "add": 1, "silu_mul": 2, "axpy": 5, "softcap": 6, "clamp_glu": 7}
_EPI_STORE_F32 = 4


_gemm_ws = {}
_pair_ws = {}
GEMM_TICKETS = 4096
PAIR_FLAGS = 65536
DECODE_GEMM_MAX_M = 128
PAIR_GEMM_MAX_M = 256


def gemm_workspace(device=None):
    """Per-device scratch of the split-K path: (fp32 partials as bytes, zeroed uint32 tickets)."""
    dev = torch.device("cuda", torch.cuda.current_device()) if device is None else torch.device(device)
    key = (dev.type, dev.index)
    if key not in _gemm_ws:
        n = int(lib().blitz_gemm_workspace_bytes(148))
        _gemm_ws[key] = (torch.empty(n, dtype=torch.uint8, device=dev),
                         torch.zeros(GEMM_TICKETS, dtype=torch.int32, device=dev))
    return _gemm_ws[key]


def pair_gemm_workspace(device=None):
    """Per-device scratch of the paired-SM GEMM: (fp32 partials as bytes, zeroed uint32 counters, eight per tile)."""
    dev = torch.device("cuda", torch.cuda.current_device()) if device is None else torch.device(device)
    key = (dev.type, dev.index)
    if key not in _pair_ws:
        sms = torch.cuda.get_device_properties(dev).multi_processor_count
        n = int(lib().blitz_gemm_pair_workspace_bytes(sms))
        _pair_ws[key] = (torch.empty(n, dtype=torch.uint8, device=dev),
                         torch.zeros(PAIR_FLAGS, dtype=torch.int32, device=dev))
    return _pair_ws[key]


def _tensor_core_operands(a: torch.Tensor, b: torch.Tensor, out: torch.Tensor, N: int, K: int) -> bool:
    """Sizes, pitches and base addresses the TMA-fed kernels need (16-byte rows and bases; fp32 outputs are accessed 32
    bytes at a time)."""
    return (N % 8 == 0 and K % 8 == 0 and a.stride(0) % 8 == 0 and b.stride(0) % 8 == 0 and out.stride(0) % 8 == 0
            and a.data_ptr() % 16 == 0 and b.data_ptr() % 16 == 0
            and out.data_ptr() % (32 if out.dtype == torch.float32 else 16) == 0)


def gemm(a: torch.Tensor, b: torch.Tensor, out: Optional[torch.Tensor] = None, *, residual=None,
         epilogue: str = "store", alpha: float = 1.0, beta: float = 1.0, bias: Optional[torch.Tensor] = None, groups: int = 1, a_step: int = 0, out_step: int = 0, b_layout: str = "kn", bn: int = 0, split_k: int = 0, static_b: bool = False,
         decode_path: Optional[bool] = None, decode_split: int = 0, pair_path: Optional[bool] = None,
         pair_bnf: int = 0, pair_upp: int = 0, pair_nacc: int = 0) -> torch.Tensor:
    """``out = a @ b`` on tcgen05 with a fused epilogue.

    a: [M, K].  b: [K, N] when ``b_layout == 'kn'`` (weights stored in,out) or [N, K] for ``'nk'``.
    epilogue 'add' adds ``residual`` ([M, N], same pitch as out); 'silu_mul' treats b as [gate | up] with
    N_out = b_cols / 2 and returns silu(a@gate) * (a@up).  ``split_k``: 0 lets the kernel split K when the
    GEMM is too skinny to fill the GPU, 1 forbids it, n > 1 forces n splits.

    Up to 256 rows of ``a`` with 'kn' weights go to the weight-streaming decode kernel (operands swapped on
    the tensor core, K split over a thread-block cluster with the reduction in distributed shared memory);
    ``decode_path`` forces (True) or forbids (False) that choice and ``decode_split`` caps its cluster size.  ``static_b=True`` promises that ``b`` is not written by kernels still
    running in this stream (model weights), so the decode kernel may start streaming it before its
    predecessor has finished.

    129..256 rows with 'kn' weights go to the paired-SM kernel (two CTAs issue one 256-row
    ``tcgen05.mma.cta_group::2``, stream-K over CTA pairs); ``pair_path`` forces (True) or forbids (False) it for
    any M, ``pair_bnf`` / ``pair_nacc`` / ``pair_upp`` override its tile width, tiles per pair and units per pair.

    ``out`` may be fp32 with 16-bit operands (the accumulator is stored unrounded); epilogue 'axpy' adds
    ``alpha * (a @ b)`` to an fp32 ``out`` (residual streams kept in 32 bits); 'softcap' stores
    ``alpha * tanh((a @ b) / alpha)`` in fp32 (logits); 'clamp_glu' is a clamped gated unit over [gate | up] columns with
    ``bias`` (as many as b's columns): g = min(gate, alpha), u = up within +- alpha, g * sigmoid(beta g) * (u + 1).  ``groups`` > 1: block-diagonal product,
    a [M, groups * K], b [groups * K, N] (the blocks stacked), out [M, groups * N]; ``a_step`` / ``out_step``: columns from a
    group to the next one in a and out, where the blocks' columns are parts of wider ones.  fp32 operands, and 16-bit ones
    whose sizes the tensor-core kernels do not take, run on the CUDA cores in fp32 arithmetic.
    """
    assert a.is_cuda and a.dim() == 2 and b.dim() == 2 and a.stride(1) == 1 and b.stride(1) == 1
    M, K = a.shape
    if groups > 1 or a_step or out_step:
        assert b.shape[0] % groups == 0 and epilogue == "store" and b_layout == "kn"
        K = b.shape[0] // groups
        a_step, out_step = a_step or K, out_step or b.shape[1]
        assert a_step * (groups - 1) + K <= a.shape[1] and out_step >= b.shape[1]
    if b_layout == "kn":
        assert b.shape[0] == K * groups
        bcols = b.shape[1]
    else:
        assert b.shape[1] == K
        bcols = b.shape[0]
    epi = _EPI[epilogue]
    gated = epi in (2, 7)
    N = bcols // 2 if gated else bcols
    if epi == 7:
        assert bias is not None and bias.is_contiguous() and bias.numel() == bcols and bias.dtype == a.dtype and alpha > 0
    if out is None:
        out = torch.empty((M, groups * N), dtype=a.dtype, device=a.device)
    assert out.stride(1) == 1 and out.shape[0] == M
    assert out.shape[1] >= out_step * (groups - 1) + N if out_step else out.shape[1] == N
    if epi in (5, 6):
        assert out.dtype == torch.float32
    elif out.dtype != a.dtype:
        assert epi == 0 and out.dtype == torch.float32
        epi = _EPI_STORE_F32
    if M == 0:
        return out
    if a.dtype == torch.float32 or (a_step | out_step) % 8 or not _tensor_core_operands(a, b, out, N, K):
        if epi == 1 or b_layout != "kn":
            raise TypeError("gemm: epilogue 'add' and 'nk' weights need the tensor-core kernels")
        assert b.dtype == a.dtype
        _check(lib().blitz_gemm_simt(_p(a), a.stride(0), _p(b), b.stride(0), _p(out), out.stride(0), M, N, K, epi,
                                     N if gated else 0, _p(bias), alpha, beta, groups, a_step, out_step, _dt3(a), _stream()), "blitz_gemm_simt")
        return out
    if epi == 1:
        assert residual is not None and residual.shape == (M, N) and residual.stride(0) == out.stride(0)
    extra = bias if epi == 7 else residual
    ws, tickets = gemm_workspace(a.device)
    # the decode kernel re-reads the activation tile with every weight tile, which the SM's load path cannot keep up
    # with beyond ~128 rows; from there on the tiled kernel is faster
    use_dec = groups == 1 and M <= DECODE_GEMM_MAX_M and bn == 0 and split_k == 0 and \
        bool(lib().blitz_gemm_decode_supported(M, N, K, 0 if b_layout == "kn" else 1, epi))
    if decode_path is not None:
        assert not decode_path or lib().blitz_gemm_decode_supported(M, N, K, 0 if b_layout == "kn" else 1, epi)
        use_dec = decode_path
    pair_ok = bool(lib().blitz_gemm_pair_supported(M, N, K, 0 if b_layout == "kn" else 1, epi))
    use_pair = (groups == 1 and not use_dec and DECODE_GEMM_MAX_M < M <= PAIR_GEMM_MAX_M and bn == 0 and split_k == 0 and pair_ok)
    if pair_path is not None:
        assert not pair_path or pair_ok
        use_pair = pair_path
    if use_pair:
        pws, pflags = pair_gemm_workspace(a.device)
        rc = lib().blitz_gemm_pair(_p(a), a.stride(0), _p(b), b.stride(0), _p(out), out.stride(0), _p(extra), M, N,
                                   K, epi, N if gated else 0, _dt(a), int(static_b), pair_bnf, pair_nacc, pair_upp,
                                   _p(pws), pws.numel(), _p(pflags), pflags.numel(), _p(status_word(a.device)),
                                   alpha, beta, _stream())
        _check(rc, "blitz_gemm_pair")
        return out
    if use_dec:
        rc = lib().blitz_gemm_decode(_p(a), a.stride(0), _p(b), b.stride(0), _p(out), out.stride(0), _p(extra), M, N,
                                     K, epi, N if gated else 0, _dt(a), int(static_b), decode_split,
                                     _p(status_word(a.device)), alpha, beta, _stream())
        _check(rc, "blitz_gemm_decode")
        return out
    rc = lib().blitz_gemm(_p(a), a.stride(0), _p(b), b.stride(0), _p(out), out.stride(0), _p(extra), M, N, K,
                          0 if b_layout == "kn" else 1, epi, N if gated else 0, _dt(a), bn, split_k,
                          _p(ws), ws.numel(), _p(tickets), tickets.numel(), _p(status_word(a.device)), alpha, beta,
                          groups, a_step, out_step, _stream())
    _check(rc, "blitz_gemm")
    return out


# ---------------------------------------------------------------------------------------------- elementwise
def embedding(ids: torch.Tensor, table: torch.Tensor, out: Optional[torch.Tensor] = None, *, vocab_start: int = 0,
              zero_missing: bool = True, dst_rows: Optional[torch.Tensor] = None) -> torch.Tensor:
    assert ids.dtype == torch.int32
    T, H = ids.numel(), table.shape[1]
    if out is None:
        out = torch.empty((T, H), dtype=table.dtype, device=table.device)
    _check(lib().blitz_embedding(_p(ids), _p(table), _p(out), T, H, vocab_start, table.shape[0], int(zero_missing),
                                 _p(dst_rows), _dt(table), _stream()), "blitz_embedding")
    return out


def rms_norm(x: torch.Tensor, w: torch.Tensor, eps: float = 1e-5, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    T, H = x.shape
    if out is None:
        out = torch.empty_like(x)
    _check(lib().blitz_rms_norm(_p(x), _p(w), _p(out), T, H, eps, _dt(x), _stream()), "blitz_rms_norm")
    return out


def add_rms_norm(x: torch.Tensor, residual: torch.Tensor, w: torch.Tensor, eps: float = 1e-5,
                 out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """residual += x; returns RMSNorm(residual) * w (written to ``out``, which may be ``x``)."""
    T, H = x.shape
    if out is None:
        out = torch.empty_like(x)
    _check(lib().blitz_add_rms_norm(_p(x), _p(residual), _p(w), _p(out), T, H, eps, _dt(x), _stream()),
           "blitz_add_rms_norm")
    return out


def silu_mul(x: torch.Tensor, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    T, two_i = x.shape
    inter = two_i // 2
    if out is None:
        out = torch.empty((T, inter), dtype=x.dtype, device=x.device)
    _check(lib().blitz_silu_mul(_p(x), _p(out), T, inter, x.stride(0), _dt(x), _stream()), "blitz_silu_mul")
    return out


def add_residual(residual: torch.Tensor, x: torch.Tensor) -> torch.Tensor:
    assert residual.is_contiguous() and x.is_contiguous() and residual.numel() == x.numel()
    _check(lib().blitz_add_residual(_p(residual), _p(x), residual.numel(), _dt(x), _stream()), "blitz_add_residual")
    return residual


def gather_last(x: torch.Tensor, indptr: torch.Tensor, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    B, H = indptr.numel() - 1, x.shape[1]
    if out is None:
        out = torch.empty((B, H), dtype=x.dtype, device=x.device)
    _check(lib().blitz_gather_last(_p(x), _p(indptr), _p(out), B, H, _dt(x), _stream()), "blitz_gather_last")
    return out


def argmax(logits: torch.Tensor, out: Optional[torch.Tensor] = None, out_val: Optional[torch.Tensor] = None,
           idx_offset: int = 0) -> torch.Tensor:
    B, V = logits.shape
    if out is None:
        out = torch.empty(B, dtype=torch.int32, device=logits.device)
    _check(lib().blitz_argmax(_p(logits), B, V, logits.stride(0), _p(out), _p(out_val), idx_offset, _dt3(logits),
                              _stream()), "blitz_argmax")
    return out


def sample(logits: torch.Tensor, temperature: torch.Tensor, top_k: torch.Tensor, top_p: torch.Tensor,
           seeds: torch.Tensor, step: int, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    B, V = logits.shape
    if out is None:
        out = torch.empty(B, dtype=torch.int32, device=logits.device)
    assert temperature.dtype == torch.float32 and top_k.dtype == torch.int32 and top_p.dtype == torch.float32
    assert seeds.dtype in (torch.int64, torch.uint64)
    _check(lib().blitz_sample(_p(logits), B, V, logits.stride(0), _p(temperature), _p(top_k), _p(top_p), _p(seeds),
                              step, _p(out), _dt3(logits), _stream()), "blitz_sample")
    return out


def rope_kv_store(qkv: torch.Tensor, pos: torch.Tensor, slot: torch.Tensor, kv_layer: torch.Tensor, *, q_heads: int,
                  kv_heads: int, head_dim: int, page_size: int, rope_theta: float) -> None:
    """Rotate q and k of ``qkv`` in place and write rotated k and v to ``kv_layer`` ([pages, 2, page, kvh, hd])."""
    T = qkv.shape[0]
    assert qkv.is_contiguous() and qkv.shape[1] == (q_heads + 2 * kv_heads) * head_dim
    assert pos.dtype == torch.int32 and slot.dtype == torch.int32
    max_pages = kv_layer.shape[0]
    _check(lib().blitz_rope_kv_store(_p(qkv), _p(pos), _p(slot), _p(kv_layer), T, q_heads, kv_heads, head_dim,
                                     page_size, max_pages, rope_theta, _p(status_word(qkv.device)), _dt(qkv),
                                     _stream()), "blitz_rope_kv_store")


# ---------------------------------------------------------------------------------------------- attention
def attn_decode_workspace_bytes(batch: int, q_heads: int, value_dim: int, num_splits: int) -> int:
    return int(lib().blitz_attn_decode_workspace_bytes(batch, q_heads, value_dim, num_splits))


def attn_decode(q: torch.Tensor, kv_layer: KVLayer, indices: torch.Tensor, indptr: torch.Tensor,
                last_page_len: torch.Tensor, *, q_heads: int, kv_heads: int, head_dim: int, page_size: int,
                num_splits: int = 1, workspace: Optional[torch.Tensor] = None, out: Optional[torch.Tensor] = None,
                sm_scale: Optional[float] = None, window: int = 0, keep_first: int = 0, softcap: float = 0.0,
                sink: Optional[torch.Tensor] = None, gate: Optional[torch.Tensor] = None,
                bias: Optional[torch.Tensor] = None, chunked: bool = False, sigmoid: bool = False) -> torch.Tensor:
    """q: [batch, >= q_heads*head_dim] (row pitch free, e.g. a view of the fused qkv buffer).  ``window`` > 0: only the
    last that many positions and the first ``keep_first`` are visible (and read); ``softcap`` > 0:
    scores are cap * tanh(score / cap); ``sink`` [q_heads]: a term e^sink in the softmax denominator; ``gate``
    [batch, q_heads]: a head's output is multiplied by its sigmoid; ``bias`` [q_heads, n]: added to the scaled scores by the
    key's distance, the last column for all longer ones.  ``chunked``: the window is a chunk counted from position 0, of which
    the keys up to the position are visible; ``sigmoid``: the weights are sigmoids of the scores, not normalised.  Values may have a size of their own (KVPair)."""
    B = indptr.numel() - 1
    kp, vp, page_rows, pages, vdim = _kv(kv_layer)
    if out is None:
        out = torch.empty((B, q_heads * vdim), dtype=q.dtype, device=q.device)
    if num_splits > 1 and workspace is None:
        workspace = torch.empty(attn_decode_workspace_bytes(B, q_heads, vdim, num_splits), dtype=torch.uint8,
                                device=q.device)
    if sm_scale is None:
        sm_scale = head_dim ** -0.5
    _check(lib().blitz_attn_decode(_p(q), q.stride(0), kp, vp, _p(indices), _p(indptr), _p(last_page_len),
                                   _p(out), out.stride(0), _p(workspace), B, q_heads, kv_heads, head_dim, vdim, page_size,
                                   page_rows, pages, num_splits, sm_scale, window, keep_first, int(chunked), int(sigmoid), softcap, _p(sink), *_bias(bias, q_heads), *_gate(gate),
                                   _p(status_word(q.device)), _dt(q), _stream()), "blitz_attn_decode")
    return out


def attn_tensor_core(q: torch.Tensor, q_heads: int, kv_heads: int, head_dim: int, page_size: int, value_dim: int = 0) -> bool:
    """Whether attn_decode and attn_prefill_paged take these head sizes (attn_ragged takes every one)."""
    return (q.dtype in _DT and attn_head_sizes(head_dim, value_dim or head_dim, page_size) and q.stride(0) % 8 == 0
            and q.data_ptr() % 16 == 0)


def attn_head_sizes(head_dim: int, value_dim: int, page_size: int) -> bool:
    return all(8 <= d <= 128 and d % 8 == 0 for d in (head_dim, value_dim)) and page_size >= 8 and page_size & (page_size - 1) == 0


def prefill_work_list(q_lens, kv_lens, page_size: int, device, skip: int = 0) -> torch.Tensor:
    """Work records of `attn_prefill_paged`, one per (sequence, 256 rows of it): first row of the sequence in the
    activation, its rows in this pass, index of its first page id, number of its pages, tokens cached for it (this
    pass included), which 256-row pair.  Ordered by the number of key blocks the pair walks, heaviest first; the kernel
    deals the list back and forth over its CTAs.  The first `skip` sequences get no record."""
    items = []
    row0 = pg0 = 0
    for s, (n, kv) in enumerate(zip(q_lens, kv_lens)):
        n, kv = int(n), int(kv)
        npages = (kv + page_size - 1) // page_size
        for pair in range((n + 255) // 256 if s >= skip else 0):
            items.append((min(kv, kv - n + 256 * (pair + 1)), row0, n, pg0, npages, kv, pair))
        row0 += n
        pg0 += npages
    items.sort(key=lambda x: -x[0])
    rec = [[r0, n, p0, np_, kv, pair, 0, 0] for _, r0, n, p0, np_, kv, pair in items]
    return torch.tensor(rec, dtype=torch.int32).reshape(-1, 8).to(device, non_blocking=True)


PREFILL_KEY_BLOCK = 128     # keys that attn_prefill_paged walks at a time


def attn_prefill_paged(q: torch.Tensor, kv_layer: KVLayer, page_indices: torch.Tensor, work: torch.Tensor, *,
                       q_heads: int, kv_heads: int, head_dim: int, page_size: int, out: Optional[torch.Tensor] = None,
                       sm_scale: Optional[float] = None, poly_exp: bool = False, window: int = 0, keep_first: int = 0,
                       softcap: float = 0.0, sink: Optional[torch.Tensor] = None,
                       gate: Optional[torch.Tensor] = None, bias: Optional[torch.Tensor] = None, chunked: bool = False,
                       sigmoid: bool = False) -> torch.Tensor:
    """Causal attention of the pass's rows over the paged cache (which already holds the rows' own keys and values,
    after whatever earlier passes stored).  ``q``: rotated query columns, e.g. the fused qkv buffer (rope_kv_store);
    ``page_indices``: the sequences' page ids back to back, covering prefix + rows; ``work`` from `prefill_work_list`
    for the same sequences.  ``window`` / ``keep_first`` / ``softcap`` / ``sink`` / ``gate`` / ``bias`` / ``chunked`` / ``sigmoid``
    as for `attn_decode` (no bias beside a window, cap or sink; with sigmoid weights a bias of one column)."""
    T = q.shape[0]
    kp, vp, page_rows, pages, vdim = _kv(kv_layer)
    if out is None:
        out = torch.empty((T, q_heads * vdim), dtype=q.dtype, device=q.device)
    if sm_scale is None:
        sm_scale = head_dim ** -0.5
    assert work.dtype == torch.int32 and work.dim() == 2 and work.shape[1] == 8 and work.is_contiguous()
    _check(lib().blitz_attn_prefill_paged(_p(q), q.stride(0), kp, vp, _p(out), out.stride(0), _p(page_indices),
                                          _p(work), work.shape[0], T, q_heads, kv_heads, head_dim, vdim, page_size, page_rows,
                                          pages, sm_scale, 1 if poly_exp else 0, window, keep_first, int(chunked), int(sigmoid), softcap, _p(sink),
                                          *_bias(bias, q_heads), *_gate(gate), _p(status_word(q.device)), _dt(q), _stream()), "blitz_attn_prefill_paged")
    return out


# ---------------------------------------------------------------------------------------------- fp32-stream models
def stream_norm(x: torch.Tensor, w: Optional[torch.Tensor], eps: float, out: Optional[torch.Tensor], *,
                w_offset: float = 0.0, ids: Optional[torch.Tensor] = None, embed: Optional[torch.Tensor] = None,
                init: bool = False, add_embed: bool = False, step: Optional[torch.Tensor] = None,
                rows: Optional[torch.Tensor] = None, row_offset: int = 0, num_tokens: Optional[int] = None,
                add: Optional[torch.Tensor] = None, add_rows: Optional[torch.Tensor] = None) -> Optional[torch.Tensor]:
    """Additions to the fp32 residual stream ``x`` ([T, hidden], in place) and the RMSNorm that follows, in one kernel.

    ``init``: x starts as ``embed[ids]``; ``add_embed``: the embeddings are added to it; ``step``: a vector added to
    every row; ``add``: row t receives the rows ``add_rows[t]`` ([T, n] int32) of it.  ``out`` (None: no norm) = x / rms(x) * (w_offset + w).  ``rows``: output row t takes row
    ``rows[t] + row_offset`` of x."""
    n = num_tokens if num_tokens is not None else (rows.numel() if rows is not None else x.shape[0])
    assert x.dtype == torch.float32 and x.is_contiguous()
    ref = out if out is not None else embed if embed is not None else add
    assert out is None or out.is_contiguous()
    n_add = 0
    if add is not None:
        n_add = add_rows.shape[1]
        assert add.is_contiguous() and add.shape[1] == x.shape[1] and add_rows.is_contiguous() and add_rows.dtype == torch.int32
        assert add_rows.shape[0] >= n and add.dtype == ref.dtype
    _check(lib().blitz_stream_norm(_p(ids), _p(embed), _p(step), _p(rows), row_offset, _p(x), _p(w), _p(out), _p(add), _p(add_rows),
                                   n_add, n,
                                   x.shape[1], embed.shape[0] if embed is not None else 0, int(init), int(add_embed),
                                   eps, w_offset, _p(status_word(x.device)), _dt3(ref), _stream()), "blitz_stream_norm")
    return out


def rope_freqs(dims: int, base: float, device, stretch: Optional[Sequence[float]] = None) -> torch.Tensor:
    """[dims / 2, 2]: base^(-2 i / dims) (times ``stretch[i]``) as an unevaluated sum of two fp32 numbers."""
    i = torch.arange(0, dims // 2, dtype=torch.float64)
    f = torch.pow(torch.tensor(base, dtype=torch.float64), -2.0 * i / max(1, dims))
    if stretch is not None:
        f = f * torch.tensor(stretch, dtype=torch.float64)
    hi = f.to(torch.float32)
    lo = (f - hi.to(torch.float64)).to(torch.float32)
    return torch.stack([hi, lo], 1).contiguous().to(device)


def rope_store(q: torch.Tensor, k: Optional[torch.Tensor], v: Optional[torch.Tensor], pos: torch.Tensor, slot: torch.Tensor,
               kv_layer: KVLayer, freqs: torch.Tensor, *, q_heads: int, kv_heads: int, dim: int, rot_dims: int,
               page_size: int, interleaved: bool, gain: float = 1.0, q_b: Optional[torch.Tensor] = None,
               k_b: Optional[torch.Tensor] = None, v_b: Optional[torch.Tensor] = None, q_w: Optional[torch.Tensor] = None,
               k_w: Optional[torch.Tensor] = None, eps: float = 0.0) -> None:
    """Rotate q in place and write rotated keys and the values to the paged cache.  q, k, v: column ranges of one
    projection ([T, ...] views with a common row pitch); ``v`` None: the values are the keys before rotation; ``k`` None:
    nothing is written.  ``q_b``, ``k_b``, ``v_b``: biases, added first.  ``gain`` multiplies the rotated dimensions.  ``q_w``,
    ``k_w``: before the rotation the rows of queries and keys get an RMS norm over all heads together, with these weights."""
    assert (q_w is None or q_w.numel() == q_heads * dim) and (k_w is None or k_w.numel() == kv_heads * dim)
    T = q.shape[0]
    assert q.stride(1) == 1 and all(x is None or (x.stride(0) == q.stride(0) and x.stride(1) == 1) for x in (k, v))
    kp, vp, page_rows, pages, vdim = _kv(kv_layer)
    _check(lib().blitz_rope_store(_p(q), _p(k), _p(v), _p(q_b), _p(k_b), _p(v_b), q.stride(0), _p(q_w), _p(k_w), eps, _p(pos), _p(slot), kp, vp, _p(freqs),
                                  gain, T, q_heads, kv_heads, dim, vdim, rot_dims, int(interleaved), page_size, page_rows, pages,
                                  _p(status_word(q.device)), _dt3(q), _stream()), "blitz_rope_store")


def attn_ragged(q: torch.Tensor, kv_layer: KVLayer, pos: torch.Tensor, tok_indptr: Optional[torch.Tensor],
                page_indptr: torch.Tensor, page_indices: torch.Tensor, out: torch.Tensor, *, q_heads: int, kv_heads: int,
                dim: int, page_size: int, scale: float, window: int = 0, keep_first: int = 0, softcap: float = 0.0,
                sink: Optional[torch.Tensor] = None, gate: Optional[torch.Tensor] = None,
                bias: Optional[torch.Tensor] = None, chunked: bool = False, sigmoid: bool = False) -> torch.Tensor:
    """General paged attention (CUDA cores, any head sizes, any element type); see csrc/kernels/attn_ragged.cu.  ``gate``
    [T, q_heads]: a head's output is multiplied by its sigmoid; ``bias``, ``chunked`` and ``sigmoid`` as for `attn_decode`."""
    T = q.shape[0]
    rows = page_indptr.numel() - 1
    assert q.stride(1) == 1 and out.stride(1) == 1
    kp, vp, page_rows, pages, vdim = _kv(kv_layer)
    _check(lib().blitz_attn_ragged(_p(q), q.stride(0), kp, vp, _p(out), out.stride(0), _p(pos), _p(tok_indptr),
                                   _p(page_indptr), _p(page_indices), _p(sink), *_bias(bias, q_heads),
                                   kv_layer.pool.shape[3] if isinstance(kv_layer, LatentKV) else vdim, *_gate(gate), T, rows,
                                   q_heads, kv_heads, dim, vdim,
                                   page_size, page_rows, pages, window, keep_first, int(chunked), int(sigmoid), scale, softcap, _p(status_word(q.device)),
                                   _dt3(q), _stream()), "blitz_attn_ragged")
    return out


def stream_mix(x: torch.Tensor, *, n: Optional[int] = None, ids: Optional[torch.Tensor] = None, embed: Optional[torch.Tensor] = None,
               pending: Optional["Pending"] = None, read: Optional[torch.Tensor] = None, norm: Optional[Sequence[torch.Tensor]] = None,
               out: Optional[torch.Tensor] = None, total: Optional[torch.Tensor] = None, write: bool = False,
               rows: Optional[torch.Tensor] = None, row_offset: int = 0) -> None:
    """Between two sublayers of a model with several residual streams (``x`` [T, streams, hidden] fp32), in one kernel.

    ``embed`` (with ``ids``): every stream is the token's embedding, x is not read.  ``pending``: the last sublayer's output,
    which the streams take up first (``write``: and keep).  Then u = sum_s read[s] x_s (None: the plain sum); ``total``
    receives u (fp32), ``out`` receives tanh(alpha u) w + b with ``norm`` = (w, alpha, b).  ``rows``: result t comes from
    token rows[t] + row_offset."""
    T, S, H = x.shape
    n = n if n is not None else (rows.numel() if rows is not None else T)
    assert x.dtype == torch.float32 and x.is_contiguous() and (out is None or (norm is not None and out.is_contiguous()))
    assert total is None or (total.dtype == torch.float32 and total.is_contiguous())
    w, alpha, b = norm if out is not None else (None, None, None)
    ref = embed if embed is not None else out if out is not None else pending.y if pending is not None else read
    if ref is None:
        ref = torch.empty(0, dtype=torch.bfloat16)        # a plain sum of fp32 streams
    pd = pending if pending is not None else Pending(None, None, None)
    assert pd.y is None or (pd.y.stride(1) == 1 and pd.y.stride(0) == H)
    _check(lib().blitz_stream_mix(_p(ids), _p(embed), embed.shape[0] if embed is not None else 0, int(embed is not None), _p(x), _p(pd.y),
                                  _p(pd.place), pd.place.shape[1] if pd.place is not None else 0, _p(pd.ident), _p(pd.prev), _p(pd.mix),
                                  _p(pd.out), _p(read), _p(alpha), _p(w), _p(b), _p(rows), row_offset, _p(out), _p(total), int(write),
                                  n, H, S, _p(status_word(x.device)), _dt3(ref), _stream()), "blitz_stream_mix")


class Pending(NamedTuple):
    """Output of a sublayer that the streams have not taken up: ``y`` [T, hidden], or rows that ``place`` [T, n] names (-1: none),
    with ``ident`` [T] times ``prev`` [T, hidden] on top; the coefficients ``mix`` [streams, streams] and ``out`` [streams].  For
    `stream_rms` also: ``bias`` [hidden] on top of y, or ``norms`` = (w0, w1): y has two outputs side by side, [T, 2 hidden], of which
    half the sum of the RMS-normed ones counts."""
    y: Optional[torch.Tensor]
    mix: Optional[torch.Tensor]
    out: Optional[torch.Tensor]
    place: Optional[torch.Tensor] = None
    ident: Optional[torch.Tensor] = None
    prev: Optional[torch.Tensor] = None
    bias: Optional[torch.Tensor] = None
    norms: Optional[tuple] = None


class TokenState(NamedTuple):
    """What a causal convolution of a token's row reads beside it: ``conv`` [taps, width], the last inputs by slot ``hist`` [slots,
    taps - 1, width], and for mixes with the row before it ``mu`` [mixes, width] and that row by slot, ``shift`` [slots, width].  Both
    histories are fp32."""
    conv: torch.Tensor
    hist: torch.Tensor
    mu: Optional[torch.Tensor] = None
    shift: Optional[torch.Tensor] = None


def stream_rms(x: torch.Tensor, *, eps: float, n: Optional[int] = None, ids: Optional[torch.Tensor] = None,
               embed: Optional[torch.Tensor] = None, pending: Optional[Pending] = None, read: Optional[torch.Tensor] = None,
               w: Optional[torch.Tensor] = None, w_offset: float = 0.0, out: Optional[torch.Tensor] = None, total: Optional[torch.Tensor] = None,
               write: bool = False, rows: Optional[torch.Tensor] = None, row_offset: int = 0, tokens: Optional[TokenState] = None,
               pos: Optional[torch.Tensor] = None, seq_slot: Optional[torch.Tensor] = None) -> None:
    """`stream_mix` with an RMS norm: ``out`` receives u / sqrt(mean(u^2) + eps) * (w_offset + w), w one number or one per column
    (``out`` may be fp32 beside shorter weights).
    ``tokens`` (decode: a token per row, ``pos`` and ``seq_slot`` say which): out is that plus its causal convolution, or with mixes
    [n, mixes * hidden]; see `token_conv`, which does the same for rows of any length."""
    T, S, H = x.shape
    n = n if n is not None else (rows.numel() if rows is not None else T)
    assert x.dtype == torch.float32 and x.is_contiguous() and (out is None or (w is not None and out.is_contiguous()))
    assert total is None or (total.dtype == torch.float32 and total.is_contiguous())
    ref = embed if embed is not None else w if w is not None else pending.y if pending is not None else read
    if ref is None:
        ref = torch.empty(0, dtype=torch.bfloat16)        # a plain sum of fp32 streams
    h32 = out is not None and out.dtype != ref.dtype
    pd = pending if pending is not None else Pending(None, None, None)
    assert pd.y is None or (pd.y.stride(1) == 1 and pd.place is None)
    assert not h32 or (out.dtype == torch.float32 and tokens is None)
    w0, w1 = pd.norms or (None, None)
    y1 = ctypes.c_void_p(pd.y.data_ptr() + H * pd.y.element_size()) if pd.norms else None
    ts = tokens if tokens is not None else TokenState(None, None)
    taps, mixes = (0 if ts.conv is None else ts.conv.shape[0]), (0 if ts.mu is None else ts.mu.shape[0])
    assert all(t is None or (t.dtype == torch.float32 and t.is_contiguous()) for t in (ts.hist, ts.shift))
    assert tokens is None or (n == seq_slot.numel() and out is not None and out.numel() == n * max(1, mixes) * H)
    _check(lib().blitz_stream_rms(_p(ids), _p(embed), embed.shape[0] if embed is not None else 0, int(embed is not None), _p(x), _p(pd.y), y1,
                                  pd.y.stride(0) if pd.y is not None else H, _p(pd.bias), _p(w0), _p(w1), _p(pd.mix), _p(pd.out), _p(read),
                                  _p(w), int(w is not None and w.numel() > 1), w_offset, eps, _p(rows), row_offset, _p(out), int(h32), _p(total),
                                  int(write), _p(ts.conv), taps, _p(ts.hist), _p(ts.mu), mixes, _p(ts.shift), _p(pos), _p(seq_slot),
                                  0 if ts.hist is None else ts.hist.shape[0], n, H, S, _p(status_word(x.device)), _dt3(ref), _stream()),
           "blitz_stream_rms")


def token_conv(x: torch.Tensor, conv: torch.Tensor, hist: torch.Tensor, out: torch.Tensor, pos, tok_indptr, seq_slot, *,
               bias: Optional[torch.Tensor] = None, silu: bool = False, residual: bool = False, mu: Optional[torch.Tensor] = None,
               shift: Optional[torch.Tensor] = None, last: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Causal convolution of every column of ``x`` [T, width] over the rows of a step, with the history [slots, taps - 1, width] it
    reads and brings up to date: silu of it, or x plus it (``residual``).  ``mu`` [mixes, width]: out [T, mixes * width] are the
    mixes with the token before, which ``shift`` [slots, width] holds between steps (``last`` [rows, width]: scratch).
    ``tok_indptr`` None: one token per row.  x, hist, shift and last may be fp32 beside shorter weights and outputs."""
    slots, keep, width = hist.shape
    assert all(t is None or t.dtype == x.dtype for t in (hist, shift, last)) and (x.dtype == out.dtype or x.dtype == torch.float32)
    mixes = 0 if mu is None else mu.shape[0]
    assert x.stride(1) == 1 and out.stride(1) == 1 and x.shape[1] == width and conv.shape == (keep + 1, width)
    assert conv.is_contiguous() and hist.is_contiguous() and out.shape[1] >= max(1, mixes) * width
    _check(lib().blitz_token_conv(_p(x), x.stride(0), _p(conv), _p(bias), _p(hist), _p(out), out.stride(0), int(silu), int(residual), int(x.dtype != out.dtype), _p(mu),
                                  mixes, _p(shift), _p(last), _p(pos), _p(tok_indptr), _p(seq_slot), x.shape[0], seq_slot.numel(), width,
                                  keep + 1, slots, _p(status_word(x.device)), _dt3(out), _stream()), "blitz_token_conv")
    return out


def norm_store(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, pos: torch.Tensor, slot: torch.Tensor, kv_layer: KVLayer,
               q_w: torch.Tensor, k_w: torch.Tensor, *, q_heads: int, kv_heads: int, dim: int, page_size: int, eps: float,
               temp_coef: float = 0.0, temp_every: int = 0) -> None:
    """RMSNorm of every query head (in place, times a temperature that grows with the position) and key head; keys and values go
    to the paged cache.  q, k, v: column ranges of one projection."""
    T = q.shape[0]
    assert all(x.stride(0) == q.stride(0) and x.stride(1) == 1 for x in (q, k, v))
    kp, vp, page_rows, pages, vdim = _kv(kv_layer)
    _check(lib().blitz_norm_store(_p(q), _p(k), _p(v), q.stride(0), _p(q_w), _p(k_w), eps, temp_coef, temp_every, _p(pos), _p(slot),
                                  kp, vp, T, q_heads, kv_heads, dim, vdim, page_size, page_rows, pages, _p(status_word(q.device)),
                                  _dt3(q), _stream()), "blitz_norm_store")


# ---------------------------------------------------------------------------------------------- latent attention
def latent_store(cq: Optional[torch.Tensor], ckv: torch.Tensor, pos: torch.Tensor, slot: torch.Tensor, kv: LatentKV,
                 cq_w: Optional[torch.Tensor], ckv_w: torch.Tensor, freqs: torch.Tensor, *, eps: float, interleaved: bool = False) -> None:
    """RMSNorm of the queries' latent (in place) and of the keys' latent (to the cache), and the rotated key part (to the
    cache).  cq, ckv: column ranges of one projection."""
    T = ckv.shape[0]
    pages, page, _, width = kv.pool.shape
    assert ckv.shape[1] == width and ckv.stride(1) == 1 and (cq is None or (cq.stride(0) == ckv.stride(0) and cq.stride(1) == 1))
    _check(lib().blitz_latent_store(_p(cq), _p(ckv), ckv.stride(0), _p(cq_w), _p(ckv_w), _p(pos), _p(slot), _p(kv.pool), _p(freqs), eps,
                                    T, cq.shape[1] if cq is not None else 0, kv.rank, width - kv.rank, int(interleaved), page, pages,
                                    _p(status_word(ckv.device)), _dt3(ckv), _stream()), "blitz_latent_store")


def latent_rotate(q: torch.Tensor, out: torch.Tensor, pos: torch.Tensor, freqs: torch.Tensor, *, heads: int, dim: int, rot: int,
                  out_step: int, interleaved: bool = False) -> None:
    """Rotate the last ``rot`` dimensions of every head of q [T, heads * (dim + rot)]; head h's go to columns h * out_step on of
    ``out`` (which may be a view of q: in place)."""
    assert q.stride(1) == 1 and out.stride(1) == 1 and q.shape[1] == heads * (dim + rot)
    _check(lib().blitz_latent_rotate(_p(q), q.stride(0), _p(out), out.stride(0), out_step, _p(pos), _p(freqs), q.shape[0], heads, dim,
                                     rot, int(interleaved), _dt3(q), _stream()), "blitz_latent_rotate")


def latent_gather(kv: LatentKV, pages: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
    """The rows of the named pages, back to back: out [pages * page, width]."""
    n, page, width = pages.numel(), kv.pool.shape[1], kv.pool.shape[3]
    assert out.is_contiguous() and out.shape == (n * page, width) and pages.dtype == torch.int32
    _check(lib().blitz_latent_gather(_p(kv.pool), _p(pages), _p(out), n, page * width * out.element_size(), kv.pool.shape[0],
                                     _p(status_word(out.device)), _stream()), "blitz_latent_gather")
    return out


def attn_latent_supported(q: torch.Tensor, batch: int, heads: int, kv: LatentKV) -> bool:
    """Whether attn_latent takes these sizes (attn_ragged takes every one)."""
    _, page, _, width = kv.pool.shape
    return q.dtype in _DT and bool(lib().blitz_attn_latent_supported(batch, heads, width, kv.rank, page))


def attn_latent_workspace(heads: int, rank: int, device) -> torch.Tensor:
    return torch.empty(int(lib().blitz_attn_latent_workspace_bytes(heads, rank)), dtype=torch.uint8, device=device)


ATTN_LATENT_ROWS = 1024     # tokens of prompts in one launch


def attn_latent(q: torch.Tensor, kv: LatentKV, indices: torch.Tensor, indptr: torch.Tensor, last_page_len: torch.Tensor, *, heads: int,
                scale: float, workspace: torch.Tensor, out: torch.Tensor, gate: Optional[torch.Tensor] = None,
                keys: int = 0, static_table: bool = False, pos: Optional[torch.Tensor] = None,
                tok_indptr: Optional[torch.Tensor] = None, window: int = 0, sink: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Decode attention over latent rows: q [batch, heads * width] against every cached row as it is, out [batch, heads * rank] =
    the weighted sums of the rows' first ``rank`` columns, times the sigmoid of ``gate`` [batch, heads].  With ``pos`` and
    ``tok_indptr`` the batch are the tokens of a ragged step (as for `attn_ragged`), each sees the keys up to its position.  ``window`` > 0: only the
    last that many positions; ``sink`` [heads]: a term e^sink in the softmax denominator.  ``keys``: per block, 64 or 128 (0: chosen).
    ``static_table`` promises that no kernel still running in this stream writes the page table (indices, indptr,
    last_page_len), so that the work list can be made before the predecessor has finished."""
    assert (pos is None) == (tok_indptr is None)
    B = q.shape[0]
    if pos is not None and B > ATTN_LATENT_ROWS:
        for t in range(0, B, ATTN_LATENT_ROWS):
            part = slice(t, min(B, t + ATTN_LATENT_ROWS))
            _attn_latent(q[part], kv, indices, indptr, last_page_len, heads, scale, workspace, out[part], None if gate is None else gate[part],
                         keys, static_table, pos[part], tok_indptr, t, window, sink)
        return out
    _attn_latent(q, kv, indices, indptr, last_page_len, heads, scale, workspace, out, gate, keys, static_table, pos, tok_indptr, 0, window, sink)
    return out


def _attn_latent(q, kv, indices, indptr, last_page_len, heads, scale, workspace, out, gate, keys, static_table, pos, tok_indptr, first, window, sink) -> None:
    rows = indptr.numel() - 1
    B = rows if pos is None else q.shape[0]
    pages, page, _, width = kv.pool.shape
    assert q.shape == (B, heads * width) and out.shape == (B, heads * kv.rank) and q.stride(1) == 1 and out.stride(1) == 1
    assert workspace.numel() >= int(lib().blitz_attn_latent_workspace_bytes(heads, kv.rank))
    _check(lib().blitz_attn_latent(_p(q), q.stride(0), _p(kv.pool), _p(indices), _p(indptr), _p(last_page_len), _p(pos),
                                   _p(tok_indptr), rows, first, _p(out), out.stride(0), _p(workspace), B, heads, width, kv.rank, page, pages, scale, window, _p(sink), *_gate(gate), keys, int(static_table), _p(status_word(q.device)),
                                   _dt(q), _stream()), "blitz_attn_latent")


# ---------------------------------------------------------------------------------------------- mixture of experts
class ExpertPlan:
    """Work list of the grouped products of a step, in buffers for up to ``max_tokens`` tokens (see csrc/kernels/moe_route.cu):
    filled by `moe_route` on the device, read by `gemm_grouped` and by `stream_norm` or `stream_mix` (``place``: -1 where a
    token chose an identity expert, whose weights are summed in ``ident``)."""

    def __init__(self, max_tokens: int, experts: int, top: int, shared: bool, device, identity: int = 0):
        i32 = lambda *shape: torch.zeros(*shape, dtype=torch.int32, device=device)
        self.experts, self.top, self.shared, self.max_tokens = experts, top, int(shared), max_tokens
        rows = max_tokens * (top + self.shared)
        self.pairs, self.counters, self.num_tiles = i32(max_tokens * top, 2), i32(2 * experts + 1), i32(1)
        self.src, self.factors = i32(rows), torch.zeros(rows, 2, dtype=torch.float32, device=device)
        self._place, self._tiles = i32(rows), i32(self.tiles_at_most(max_tokens, 64), 4)
        self.identity, self._ident = identity, torch.zeros(max_tokens, dtype=torch.float32, device=device) if identity else None
        self.tokens, self.tile_rows = 0, 128

    @property
    def ident(self) -> Optional[torch.Tensor]:
        return None if self._ident is None else self._ident[:self.tokens]

    def tiles_at_most(self, tokens: int, tile_rows: int) -> int:
        pairs = tokens * self.top
        return min(pairs, self.experts) + pairs // tile_rows

    @property
    def rows(self) -> int:
        return self.tokens * (self.top + self.shared)

    @property
    def place(self) -> torch.Tensor:
        return self._place[:self.rows].view(self.tokens, self.top + self.shared)

    def tiles_usually(self):
        """(tiles, rows of one) of an even spread over the experts."""
        pairs = self.tokens * self.top * self.experts // (self.experts + self.identity)
        used = max(1, round(self.experts * (1.0 - (1.0 - 1.0 / self.experts) ** pairs)))
        return used + max(0, pairs - used * self.tile_rows // 2) // self.tile_rows, min(self.tile_rows, max(1, -(-pairs // used)))


def moe_route(logits: torch.Tensor, plan: ExpertPlan, *, weight_on_input: bool = True, renormalize: bool = False,
              softmax: bool = False, correction: Optional[torch.Tensor] = None, groups: int = 0, keep: int = 0,
              tile_rows: int = 128) -> ExpertPlan:
    """Choose experts from fp32 router logits [T, experts (+ identity experts, or + 1: gate of the shared expert)] and sort the
    rows by expert.  ``softmax``: scores are a softmax over all outputs (else sigmoids); ``correction``: added to the scores
    the choice is made by; ``groups``: only experts of the best ``keep`` of so many equal groups can be chosen."""
    T = logits.shape[0]
    assert logits.dtype == torch.float32 and logits.stride(1) == 1 and logits.shape[1] >= plan.experts + plan.identity + plan.shared
    assert correction is None or (correction.is_contiguous() and correction.numel() == plan.experts + plan.identity)
    assert T <= plan.max_tokens and tile_rows >= 64
    plan.tokens, plan.tile_rows = T, tile_rows
    _check(lib().blitz_moe_route(_p(logits), logits.stride(0), T, plan.experts, plan.top, plan.shared, int(weight_on_input),
                                 int(renormalize), plan.identity, int(softmax), groups, keep, _p(correction),
                                 0 if correction is None else _dt3(correction), _p(plan._ident), tile_rows, plan.tiles_at_most(T, tile_rows), _p(plan.pairs), _p(plan.counters),
                                 _p(plan.src), _p(plan.factors), _p(plan._place), _p(plan._tiles), _p(plan.num_tiles),
                                 _p(status_word(logits.device)), _stream()), "blitz_moe_route")
    return plan


_ACT = {"none": 0, "relu2": 1, "silu_gate": 2}


def grouped_tensor_core(a: torch.Tensor, *matrices: Optional[torch.Tensor]) -> bool:
    """Whether `gemm_grouped` runs these operands on the tensor cores (else on the CUDA cores, with tile_rows 64)."""
    return (a.dtype in _DT and a.stride(0) % 8 == 0 and a.data_ptr() % 16 == 0
            and all(m is None or (m.shape[-1] % 8 == 0 and m.shape[-2] % 8 == 0 and m.data_ptr() % 16 == 0) for m in matrices))


def gemm_grouped(a: torch.Tensor, b: torch.Tensor, plan: ExpertPlan, out: torch.Tensor, *, shared: Optional[torch.Tensor] = None,
                 gather: bool = False, act: str = "none", factors: bool = False, bn: int = 0, fetch: int = 0) -> torch.Tensor:
    """out[r] = after_r * act(before_r * (a[row] @ b[expert of r])) for the plan's sorted rows r; ``b`` [experts, K, N];
    ``shared`` [K', N']: the shared expert's matrix for the rows behind (K' and N' columns of a and out).  ``gather``: row r
    reads the activation of its token, else sorted row r.  ``act`` "silu_gate": b has 32 gate columns, the 32 up columns they
    gate, and so on (`interleave_gate`), out half as many.  ``factors``: apply the plan's factors (else both are 1).  ``bn``
    forces the tile width, ``fetch`` how rows are gathered (1 TMA, 2 copying warps)."""
    E, K, N = b.shape
    assert E == plan.experts and b.is_contiguous() and a.stride(1) == 1 and out.stride(1) == 1 and a.dtype == b.dtype == out.dtype
    assert (shared is not None) == bool(plan.shared) and out.shape[0] >= plan.rows
    Ks, Ns = (K, N) if shared is None else shared.shape
    assert act != "silu_gate" or (shared is None and N % 64 == 0)
    assert a.shape[1] >= max(K, Ks) and out.shape[1] >= (N // 2 if act == "silu_gate" else max(N, Ns)) and (shared is None or shared.is_contiguous())
    src, fac = plan.src if gather else None, plan.factors if factors else None
    row0, shared_rows = plan.tokens * plan.top, plan.tokens * plan.shared
    most = plan.tiles_at_most(plan.tokens, plan.tile_rows)
    if plan.tile_rows == 64:
        _check(lib().blitz_gemm_grouped_simt(_p(a), a.stride(0), _p(src), _p(b), N, K, _p(shared), Ns, Ks, _p(out), out.stride(0),
                                             _p(fac), _p(plan._tiles), _p(plan.num_tiles), most, row0, shared_rows, _ACT[act],
                                             _dt3(a), _stream()), "blitz_gemm_grouped_simt")
        return out
    assert plan.tile_rows == 128 and grouped_tensor_core(a, b, shared) and out.stride(0) % 8 == 0
    _check(lib().blitz_gemm_grouped(_p(a), a.stride(0), plan.tokens if gather else plan.rows, _p(src), _p(b), E, N, K, _p(shared), Ns,
                                    Ks, _p(out), out.stride(0), _p(fac), _p(plan._tiles), _p(plan.num_tiles), most,
                                    *plan.tiles_usually(), row0, shared_rows, plan.tokens, _ACT[act], bn, fetch,
                                    _p(status_word(a.device)), _dt(a), _stream()), "blitz_gemm_grouped")
    return out


def interleave_gate(gate: torch.Tensor, up: torch.Tensor) -> torch.Tensor:
    """[K, n] gate and up matrices (n a multiple of 32) -> [K, 2 n], 32 columns of one and of the other in turn."""
    K, n = gate.shape
    return torch.stack([gate.reshape(K, n // 32, 32), up.reshape(K, n // 32, 32)], 2).reshape(K, 2 * n)


def gla_recurrent(q, k, v, g, low, a2, a2_b, norm, state: torch.Tensor, out: torch.Tensor, pos, tok_indptr, seq_slot, *,
                  rank: int, tau: float, eps: float) -> torch.Tensor:
    """Gated linear attention token by token over the rows of a step; ``state`` [slots, heads, dim, vdim] fp32.
    ``tok_indptr`` None: one token per row (decode)."""
    slots, heads, dim, vdim = state.shape
    assert state.dtype == torch.float32 and state.is_contiguous() and out.stride(1) == 1
    _check(lib().blitz_gla_recurrent(_p(q), _p(k), _p(v), _p(g), _p(low), q.stride(0), _p(a2), _p(a2_b), _p(norm),
                                     _p(state), _p(out), out.stride(0), _p(pos), _p(tok_indptr), _p(seq_slot),
                                     seq_slot.numel(), heads, dim, vdim, rank, slots, dim ** -0.5, tau, eps,
                                     int(tok_indptr is not None), _p(status_word(q.device)), _dt3(q), _stream()),
           "blitz_gla_recurrent")
    return out


def conv_causal(x, x_b, conv, conv_b, hist: torch.Tensor, u: torch.Tensor, pos, tok_indptr, seq_slot) -> torch.Tensor:
    """Causal short convolution per channel over the rows of a step; ``hist`` [slots, taps - 1, width], only read."""
    slots, keep, width = hist.shape
    _check(lib().blitz_conv_causal(_p(x), x.stride(0), _p(x_b), _p(conv), _p(conv_b), _p(hist), _p(u), u.stride(0), _p(pos),
                                   _p(tok_indptr), _p(seq_slot), x.shape[0], seq_slot.numel(), width, keep + 1, slots,
                                   _p(status_word(x.device)), _dt3(x), _stream()), "blitz_conv_causal")
    return u


def rglru_scan(u, gates: torch.Tensor, gate_b, lam, y, x, y_b, state: torch.Tensor, hist: torch.Tensor, out, pos,
               tok_indptr, seq_slot, *, block: int) -> torch.Tensor:
    """Real-gated linear recurrent unit over the rows of a step, times gelu(y); updates ``state`` [slots, width] and the
    convolution's history."""
    slots, width = state.shape
    assert gates.dtype == torch.float32 and gates.is_contiguous() and y.stride(0) == x.stride(0)
    _check(lib().blitz_rglru_scan(_p(u), u.stride(0), _p(gates), _p(gate_b), _p(lam), _p(y), _p(x), y.stride(0), _p(y_b),
                                  _p(state), _p(hist), _p(out), out.stride(0), _p(pos), _p(tok_indptr), _p(seq_slot),
                                  seq_slot.numel(), width, block, hist.shape[1] + 1, slots, int(tok_indptr is None),
                                  _p(status_word(u.device)), _dt3(u), _stream()), "blitz_rglru_scan")
    return out


GLA_CHUNK_MIN_LEN = 16      # rows shorter than this are faster token by token


def gla(q, k, v, g, low, a2, a2_b, norm, state: torch.Tensor, out: torch.Tensor, pos, tok_indptr, seq_slot, *, rank: int,
        tau: float, eps: float, row_lens=None, cum: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Gated linear attention over the rows of a step; ``row_lens``: tokens per row (host), needed where rows are longer
    than one token.  Prompts in bf16 go through the chunked tensor-core kernel, everything else token by token.
    ``cum``: fp32 scratch of the chunked kernel, tokens x heads x dim elements (allocated when missing)."""
    slots, heads, dim, vdim = state.shape
    longest = 1 if tok_indptr is None else max(row_lens)
    aligned = all(t.data_ptr() % 16 == 0 for t in (q, k, v)) and q.stride(0) % 8 == 0 and g.data_ptr() % 4 == 0
    if (longest < GLA_CHUNK_MIN_LEN or q.dtype != torch.bfloat16 or not aligned or out.stride(0) % 2 or out.data_ptr() % 4
            or not lib().blitz_gla_chunk_supported(dim, vdim, rank)):
        return gla_recurrent(q, k, v, g, low, a2, a2_b, norm, state, out, pos, tok_indptr, seq_slot, rank=rank, tau=tau, eps=eps)
    n = q.shape[0] * heads * dim
    if cum is None:
        cum = torch.empty(n, dtype=torch.float32, device=q.device)
    assert cum.dtype == torch.float32 and cum.numel() >= n and state.dtype == torch.float32 and state.is_contiguous()
    _check(lib().blitz_gla_chunk(_p(q), _p(k), _p(v), _p(g), _p(low), q.stride(0), _p(a2), _p(a2_b), _p(norm), _p(cum),
                                 _p(state), _p(out), out.stride(0), _p(pos), _p(tok_indptr), _p(seq_slot), seq_slot.numel(),
                                 longest, heads, dim, vdim, rank, slots, dim ** -0.5, tau, eps, _p(status_word(q.device)),
                                 _stream()), "blitz_gla_chunk")
    return out


def wkv(r, k, v, g, low: torch.Tensor, a2, a2_b, bonus, norm, state: torch.Tensor, out: torch.Tensor, pos, tok_indptr, seq_slot, *,
        rank: int, eps: float, row_lens=None, cum: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Linear attention that sees the state before the token plus the token itself with a bonus, with decays exp(-exp(tanh(low) a2 +
    a2_b)) from ``low`` [T, >= rank] fp32; then the norm of every head (``norm`` [heads * vdim]) and silu(g).  Otherwise as `gla`."""
    slots, heads, dim, vdim = state.shape
    assert low.dtype == torch.float32 and low.stride(1) == 1 and state.dtype == torch.float32 and state.is_contiguous() and out.stride(1) == 1
    assert all(t.stride(0) == r.stride(0) and t.stride(1) == 1 for t in (k, v, g))
    longest = 1 if tok_indptr is None else max(row_lens)
    aligned = all(t.data_ptr() % 16 == 0 for t in (r, k, v, bonus)) and r.stride(0) % 8 == 0 and g.data_ptr() % 4 == 0
    args = [_p(r), _p(k), _p(v), _p(g), r.stride(0), _p(low), low.stride(0), _p(a2), _p(a2_b), _p(bonus), _p(norm)]
    if (longest < GLA_CHUNK_MIN_LEN or r.dtype != torch.bfloat16 or not aligned or out.stride(0) % 2 or out.data_ptr() % 4
            or not lib().blitz_gla_chunk_supported(dim, vdim, rank)):
        _check(lib().blitz_wkv_recurrent(*args, _p(state), _p(out), out.stride(0), _p(pos), _p(tok_indptr), _p(seq_slot), seq_slot.numel(),
                                         heads, dim, vdim, rank, slots, eps, int(tok_indptr is not None), _p(status_word(r.device)),
                                         _dt3(r), _stream()), "blitz_wkv_recurrent")
        return out
    n = r.shape[0] * heads * dim
    if cum is None:
        cum = torch.empty(n, dtype=torch.float32, device=r.device)
    assert cum.dtype == torch.float32 and cum.numel() >= n
    _check(lib().blitz_wkv_chunk(*args, _p(cum), _p(state), _p(out), out.stride(0), _p(pos), _p(tok_indptr), _p(seq_slot), seq_slot.numel(),
                                 longest, heads, dim, vdim, rank, slots, eps, _p(status_word(r.device)), _stream()), "blitz_wkv_chunk")
    return out


SSD_CHUNK_MIN_LEN = 16


def ssd(x, B, C, z, dt, dt_bias, A_log, D, state: torch.Tensor, out: torch.Tensor, pos, tok_indptr, seq_slot, *, groups: int,
        row_lens=None) -> torch.Tensor:
    """State-space recurrence with a decay per head over the rows of a step, gated by silu(z); ``state`` [slots, heads, state, vdim]
    fp32.  x, B, C: column ranges of one buffer; z, dt: of another.  Prompts in bf16 go through the chunked tensor-core kernel."""
    slots, heads, dim, vdim = state.shape
    assert state.dtype == torch.float32 and state.is_contiguous() and out.stride(1) == 1
    assert B.stride(0) == x.stride(0) == C.stride(0) and z.stride(0) == dt.stride(0)
    args = [_p(x), _p(B), _p(C), x.stride(0), _p(z), _p(dt), z.stride(0), _p(dt_bias), _p(A_log), _p(D), _p(state), _p(out), out.stride(0),
            _p(pos), _p(tok_indptr), _p(seq_slot), seq_slot.numel(), heads, groups, dim, vdim, slots, _p(status_word(x.device))]
    longest = 1 if tok_indptr is None else max(row_lens)
    aligned = all(t.data_ptr() % 16 == 0 for t in (x, B, C)) and x.stride(0) % 8 == 0 and all(t.data_ptr() % 4 == 0 and t.stride(0) % 2 == 0 for t in (z, out))
    if longest < SSD_CHUNK_MIN_LEN or x.dtype != torch.bfloat16 or not aligned or not lib().blitz_ssd_chunk_supported(dim, vdim):
        _check(lib().blitz_ssd_recurrent(*args, _dt3(x), _stream()), "blitz_ssd_recurrent")
    else:
        _check(lib().blitz_ssd_chunk(*args, _stream()), "blitz_ssd_chunk")
    return out


def part_norm(x: torch.Tensor, w: torch.Tensor, parts: int, eps: float) -> torch.Tensor:
    """RMS norm of the rows of ``x`` [T, width] in equal parts, each by its own root mean square, in place, times ``w`` [width]."""
    T, width = x.shape
    assert x.stride(1) == 1 and w.numel() == width and width % parts == 0
    for t in range(0, T, 65535):
        rows = x[t:t + 65535]
        _check(lib().blitz_part_norm(_p(rows), x.stride(0), _p(w), eps, rows.shape[0], parts, width // parts, _dt3(x), _stream()), "blitz_part_norm")
    return x
