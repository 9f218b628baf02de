"""Per-GPU serving engine: weight segment + paged KV pool + batches + the fused forward.

This is the counterpart of the reference's engine facade (src/blitz/stub.h:68-291 constructor,
:1283-1364 `forward`): it owns the model memory, the page allocator and the cached batches, stages
the per-step page table through pinned memory, and runs prefill / decode steps.  Differences that
matter for speed: the decode step is replayed from a CUDA graph per padded batch size (the
reference relaunches ~9 kernels per layer per token on the default stream and synchronises after
every prefill layer, src/model/llama.h:345-355), attention needs no host-side plan, and there is
exactly one H2D copy (inputs + page table) and one D2H copy (sampled tokens) per step.
"""
from __future__ import annotations

import time
from typing import Dict, List, Optional, Sequence

import numpy as np
import torch

from .. import ops
from ..models.config import ModelConfig, get_config
from ..models.llama import LlamaRunner, StepMeta, TPComm
from ..models.weights import WeightSegment
from ..utils.tracing import nvtx_range
from . import core

_BUCKETS = [1, 2, 4, 8, 16, 24, 32, 48, 64, 96, 128, 192, 256, 384, 512, 768, 1024]


def _bucket(n: int) -> int:
    for b in _BUCKETS:
        if n <= b:
            return b
    return n


class Engine:
    def __init__(self, model: str | ModelConfig, *, num_pages: int, page_size: int = 64, max_batch: int = 256,
                 max_batch_tokens: int = 8192, tp: int = 1, tp_rank: int = 0, dtype=torch.bfloat16,
                 device: Optional[torch.device] = None, comm: Optional[TPComm] = None, use_graphs: bool = True,
                 seg_buffer: Optional[torch.Tensor] = None, kv_buffer: Optional[torch.Tensor] = None,
                 ready: bool = True, seed: int = 0, fused_tp: bool = True, oneshot_max_rows: int = 1024,
                 tp_contexts: int = 1, use_switch: bool = True, state_slots: Optional[int] = None):
        self.cfg = get_config(model) if isinstance(model, str) else model
        self.device = device or torch.device("cuda", torch.cuda.current_device())
        self.dtype, self.tp, self.tp_rank = dtype, tp, tp_rank
        self.page_size, self.num_pages = page_size, num_pages
        self.max_batch, self.max_batch_tokens = max_batch, max_batch_tokens
        c = self.cfg
        self.seg = WeightSegment(c, tp, tp_rank, dtype, device=self.device, buffer=seg_buffer)
        self.fused = None
        self.slots = None           # state slots of models with recurrent layers
        if c.family == "hybrid":
            if tp > 1 or kv_buffer is not None:
                raise ValueError(f"{c.name}: a hybrid model runs on one GPU, with its own cache memory")
            from ..models.hybrid import HybridRunner
            from .hybrid_cache import HybridCache
            self.cache = HybridCache(c, num_pages, page_size, state_slots or max_batch, dtype, self.device)
            if c.recurrent:
                self.slots = core.SlotPool(self.cache.num_slots)
        else:
            if dtype == torch.float32:
                raise ValueError(f"{c.name}: the kernels of this model take 16-bit types")
            kvh = c.kv_heads // tp
            kv_shape = (c.layers, num_pages, 2, page_size, kvh, c.head_dim)
            if kv_buffer is None:
                # zero-filled: the attention kernels require finite values in every slot of an allocated page
                self.kv = torch.zeros(kv_shape, dtype=dtype, device=self.device)
            else:
                self.kv = kv_buffer.view(dtype)[:int(np.prod(kv_shape))].view(kv_shape)
        if c.family == "hybrid":
            self.runner = HybridRunner(self.seg, self.cache, max(max_batch_tokens, max_batch), max_batch)
        elif tp > 1 and comm is not None and fused_tp:
            # tensor-parallel layers through the fused peer-memory kernels (GEMM -> reduce-scatter push, reduce + norm +
            # all-gather push, flag-gated GEMM); the NCCL all-reduce runner is the baseline (`fused_tp=False`)
            from ..parallel.tp import FusedTP, LlamaRunnerTP
            self.fused = FusedTP(comm.group, c.hidden, max(max_batch_tokens, max_batch), dtype=dtype,
                                 contexts=tp_contexts)
            self.runner = LlamaRunnerTP(self.seg, self.kv, max(max_batch_tokens, max_batch), max_batch, comm, self.fused,
                                        oneshot_max_rows=oneshot_max_rows)
            self.runner.use_switch = use_switch
        else:
            self.runner = LlamaRunner(self.seg, self.kv, max_tokens=max(max_batch_tokens, max_batch), max_batch=max_batch,
                                      comm=comm)
        self.pool = core.PagePool(num_pages, page_size)
        self.layout = core.MetaLayout.make(max(max_batch_tokens, max_batch), max_batch, num_pages)
        self.host = torch.zeros(self.layout.total, dtype=torch.int32, pin_memory=True)
        self.host_np = self.host.numpy()
        self.dev = torch.zeros(self.layout.total, dtype=torch.int32, device=self.device)
        self.tok_host = torch.zeros(max_batch, dtype=torch.int32, pin_memory=True)
        self.status = core.ModelStatus(c.layers)
        if ready:
            self.seg.random_init_fast_(seed)
            self.status.set_ready()
        self.batches: Dict[int, "core.Batch"] = {}
        self.use_graphs = use_graphs
        self._graphs: Dict[tuple, torch.cuda.CUDAGraph] = {}
        self.stream = torch.cuda.Stream(device=self.device)
        self.h2d_bytes = 0
        self.d2h_bytes = 0
        self.launches_per_decode_step = 0

    # ------------------------------------------------------------------ meta views
    def _views(self, T: int, B: int, P: int, prefill: bool, seq_lens: Sequence[int] = (), splits: int = 1,
               kv_lens: Sequence[int] = (), work: Optional[torch.Tensor] = None, singles: int = 0) -> StepMeta:
        L, d = self.layout, self.dev
        kv_lens = list(kv_lens) if kv_lens else list(seq_lens)
        if prefill and work is None:
            # the hybrid runner takes the leading single tokens of a ragged step through its decode kernels
            work = ops.prefill_work_list(seq_lens, kv_lens, self.page_size, self.device,
                                         skip=singles if self.cfg.family == "hybrid" else 0)
        return StepMeta(kv_lens_host=kv_lens, prefill_work=work,
                        ids=d[L.ids:L.ids + T], pos=d[L.pos:L.pos + T], slot=d[L.slot:L.slot + T],
                        page_indices=d[L.page_indices:L.page_indices + max(P, 1)],
                        page_indptr=d[L.page_indptr:L.page_indptr + B + 1],
                        last_page_len=d[L.last_page_len:L.last_page_len + B],
                        tok_indptr=d[L.tok_indptr:L.tok_indptr + B + 1] if prefill else None,
                        seq_slot=d[L.seq_slot:L.seq_slot + B], singles=singles,
                        seq_lens_host=list(seq_lens), is_prefill=prefill, batch=B, num_tokens=T, num_splits=splits)

    def _h2d(self, hi: int) -> None:
        self.dev[:hi].copy_(self.host[:hi], non_blocking=True)
        self.h2d_bytes = hi * 4

    def _tokens_to_host(self, toks: torch.Tensor, B: int) -> List[int]:
        self.tok_host[:B].copy_(toks[:B], non_blocking=True)
        torch.cuda.current_stream().synchronize()
        self.d2h_bytes = B * 4
        return self.tok_host[:B].tolist()

    # ------------------------------------------------------------------ batches
    def new_batch(self, batch_id: int, specs) -> Optional["core.Batch"]:
        b = core.Batch(batch_id, self.pool, self.slots)
        if not b.add_prompts(specs):
            return None
        return b

    def choose_splits(self, B: int, max_len: int) -> int:
        if self.cfg.family == "hybrid":
            kv_heads, max_len = self.cfg.attention_work(max_len)
            if kv_heads == 0:
                return 1
        else:
            kv_heads = self.cfg.kv_heads // self.tp
        ctas = B * kv_heads
        if ctas >= 2 * 148 or max_len <= 256:
            return 1
        want = (2 * 148 + ctas - 1) // ctas
        cap = max(1, max_len // 256)
        s = 1
        while s * 2 <= min(want, cap, 32):
            s *= 2
        return s

    # ------------------------------------------------------------------ steps
    @torch.no_grad()
    def prefill(self, batch: "core.Batch", after_layer=None) -> List[int]:
        """Run the prompt of every request in `batch`, cache its K/V and return the first token of each.

        `after_layer(l)` is called when every K/V row of layer l is in the stream that runs the pass (in a prefill of
        several windows: during the last window), so that a caller can send the layer away while the next ones run."""
        if not self.status.fully_loaded():
            raise RuntimeError("model parameters are not loaded")
        if batch.size > self.max_batch:
            raise ValueError(f"prefill batch of {batch.size} sequences exceeds max_batch={self.max_batch}")
        if batch.num_prompt_tokens() > self.max_batch_tokens:
            toks = self._prefill_in_chunks(batch, after_layer)
            toks = self._sample_rows(batch, batch.size, toks)
            out = self._tokens_to_host(toks, batch.size)
            batch.mark_prefilled()
            batch.append_tokens(out, False)
            batch.decode = True
            return out
        T, P = batch.fill_prefill(self.host_np, self.layout)
        self._h2d(self.layout.page_indices + P)
        lens = batch.prompt_lens()
        m = self._views(T, batch.size, P, True, lens)
        with nvtx_range("prefill"):
            toks = self.runner.forward(m, after_layer=after_layer)
        toks = self._sample_rows(batch, batch.size, toks)
        out = self._tokens_to_host(toks, batch.size)
        batch.mark_prefilled()
        batch.append_tokens(out, False)
        batch.decode = True
        return out

    def _prefill_in_chunks(self, batch: "core.Batch", after_layer=None) -> torch.Tensor:
        """Prompts that together exceed `max_batch_tokens` (one prompt alone may): passes over windows of that many
        tokens of the prompts laid end to end.  A window's rows attend to the cache, which holds what earlier windows
        stored for the same sequence; the state of every sequence's last token is kept when its prompt ends, and the
        head runs once over all of them.  The reference stops packing at the token budget and cannot split a prompt
        (router_v2/src/queue.rs:279-286)."""
        total, B = batch.num_prompt_tokens(), batch.size
        runner = self.runner
        forced = getattr(runner, "force_switch", None)
        if forced is not None:
            runner.force_switch = True          # tensor parallel: keep the residual stream replicated in every pass
        try:
            states = torch.empty(B, self.cfg.hidden, dtype=runner.res.dtype, device=self.device)
            tok0 = 0
            while tok0 < total:
                T, P, rows, s0, q_lens, kv_lens, ended = batch.fill_prefill_chunk(self.host_np, self.layout, tok0,
                                                                                  self.max_batch_tokens)
                self._h2d(self.layout.page_indices + P)
                m = self._views(T, rows, P, True, q_lens, kv_lens=kv_lens)
                with nvtx_range("prefill_chunk"):
                    runner.forward(m, with_head=False, after_layer=after_layer if tok0 + T >= total else None)
                    if any(ended):
                        last = runner.last_rows(m)
                        for r, e in enumerate(ended):
                            if e:
                                states[s0 + r].copy_(last[r])
                # the staging arrays are reused by the next window
                torch.cuda.current_stream().synchronize()
                tok0 += T
            return runner.head_from_rows(states)
        finally:
            if forced is not None:
                runner.force_switch = forced

    @torch.no_grad()
    def decode(self, batch: "core.Batch") -> List[int]:
        """One decode step for every request in `batch` (already extended if several were merged).  Requests that
        have already finished stay in their rows as padding (no cache write; their returned token is meaningless and
        is not recorded): callers normally filter them out between steps."""
        if not self.status.fully_loaded():
            raise RuntimeError("model parameters are not loaded")
        B = batch.size
        if B > self.max_batch:
            raise ValueError(f"decode batch of {B} sequences exceeds max_batch={self.max_batch}")
        Bp = _bucket(B) if self.use_graphs else B
        Bp = min(Bp, self.max_batch)
        splits = self.choose_splits(Bp, batch.max_seq_len())
        P = batch.fill_decode(self.host_np, self.layout, Bp)
        self._h2d(self.layout.page_indices + P)
        if self.use_graphs:
            key = (Bp, splits)
            g = self._graphs.get(key)
            if g is None:
                g = self._capture(Bp, splits)
            g.replay()
            toks = self.runner.tokens
        else:
            toks = self.runner.forward(self._views(Bp, Bp, self.num_pages, False, splits=splits))
        toks = self._sample_rows(batch, B, toks)
        out = self._tokens_to_host(toks, B)
        batch.append_tokens(out, True)
        return out

    @torch.no_grad()
    def step(self, batch: "core.Batch", counts: Sequence[int], want: Sequence[Sequence[int]] = ()) -> Optional[torch.Tensor]:
        """One step over any mixture of the batch's requests: `counts[i]` tokens of request i, from the first one that is
        not cached yet (0: it sits this step out); portions of prompts and single tokens run together.  `want[i]`: places
        among these tokens whose logits are returned, [total, vocab] fp32, in the order of the requests (None if there
        are none).  Nothing is sampled.  Steps beyond `max_batch_tokens` are cut into several passes."""
        if not self.status.fully_loaded():
            raise RuntimeError("model parameters are not loaded")
        if self.tp > 1:
            raise RuntimeError("steps of given tokens run on one GPU")
        if batch.size > self.max_batch:
            raise ValueError(f"step over {batch.size} sequences exceeds max_batch={self.max_batch}")
        counts = list(counts)
        want = [list(w) for w in want] if len(want) else [[] for _ in counts]
        first = [sum(len(w) for w in want[:i]) for i in range(len(want))]
        total = sum(len(w) for w in want)
        out = torch.empty(total, self.cfg.vocab, dtype=torch.float32, device=self.device) if total else None
        done = [0] * len(counts)
        while any(d < c for d, c in zip(done, counts)):
            room, take = self.max_batch_tokens, []
            for d, c in zip(done, counts):
                take.append(min(room, c - d))
                room -= take[-1]
            dest, src = [], []           # rows of `out` this pass fills, and where they come from
            for i, w in enumerate(want):
                for j, p in enumerate(w):
                    if done[i] <= p < done[i] + take[i]:
                        dest.append(first[i] + j)
                        src.append((i, p - done[i]))
            rows = self._step_pass(batch, take, src)
            if dest:
                out[torch.tensor(dest, device=self.device)] = rows
            done = [d + t for d, t in zip(done, take)]
        return out

    def _step_pass(self, batch: "core.Batch", counts: List[int], src: List[tuple]) -> Optional[torch.Tensor]:
        """One forward pass of `step`: logits of the (request, place) pairs in `src`."""
        single = all(c <= 1 for c in counts)
        rows_max = sum(1 for c in counts if c)
        pad = min(_bucket(rows_max), self.max_batch) if self.use_graphs else rows_max
        T, P, rows, singles, order, q_lens, kv_lens = batch.fill_step(self.host_np, self.layout, counts, pad)
        self._h2d(self.layout.page_indices + P)
        row_of = {b: r for r, b in enumerate(order)}
        if single:
            splits = self.choose_splits(pad, max(kv_lens))
            if self.use_graphs:
                (self._graphs.get((pad, splits)) or self._capture(pad, splits)).replay()
            else:
                self.runner.forward(self._views(pad, pad, self.num_pages, False, splits=splits))
            got = None
            if src:
                got = self.runner.logits[torch.tensor([row_of[b] for b, _ in src], device=self.device)].float()
        else:
            splits = self.choose_splits(singles, max(kv_lens[:singles])) if singles else 1
            m = self._views(T, rows, P, True, q_lens, splits=splits, kv_lens=kv_lens, singles=singles)
            with nvtx_range("step"):
                self.runner.forward(m, with_head=False)
                starts = [sum(q_lens[:r]) for r in range(rows)]
                flat = [starts[row_of[b]] + p for b, p in src]
                parts = []
                for i in range(0, len(flat), self.max_batch):
                    idx = torch.tensor(flat[i:i + self.max_batch], dtype=torch.int32, device=self.device)
                    parts.append(self.runner.logits_of(idx.numel(), idx).float().clone())
                got = torch.cat(parts) if parts else None
        torch.cuda.current_stream().synchronize()       # the staging arrays are reused by the next pass
        batch.advance(counts)
        return got

    def _sample_rows(self, batch: "core.Batch", B: int, toks: torch.Tensor) -> torch.Tensor:
        """Rows whose request asked for sampling (`do_sample` with temperature / top-k / top-p / seed) draw their token
        from this step's logits with the sampling kernel; all other rows keep the arg-max.  One extra small launch,
        outside the CUDA graph, and only when such a row exists.  With tp > 1 every rank holds a vocabulary shard of
        the logits; the shards of the sampled rows are gathered first (the reference serves greedily only)."""
        rows, temp, top_k, top_p, seeds = batch.sampling_rows()
        if not rows:
            return toks
        dev = self.device
        idx = torch.tensor(rows, dtype=torch.long, device=dev)
        logits = self.runner.logits[:B].index_select(0, idx)
        if self.tp > 1:
            # every rank holds a vocabulary shard of the rows: gather the shards of the (few) sampled rows, so that
            # every rank draws from the same full distribution with the same seed and gets the same token
            logits = self._gather_vocab_shards(logits)
        drawn = ops.sample(logits, torch.tensor(temp, dtype=torch.float32, device=dev),
                           torch.tensor(top_k, dtype=torch.int32, device=dev),
                           torch.tensor(top_p, dtype=torch.float32, device=dev),
                           torch.tensor(seeds, dtype=torch.int64, device=dev), 0)
        toks = toks[:B].clone()
        toks[idx] = drawn.to(toks.dtype)
        return toks

    def _gather_vocab_shards(self, shard_rows: torch.Tensor) -> torch.Tensor:
        """[n, vocab / tp] on every rank -> [n, vocab] on every rank, through the peer-memory all-gather of the fused
        runner (a few rows per call, bounded by its slot size) or the collective library of the comparison runner."""
        n, vs = shard_rows.shape
        if self.fused is None:
            full = self.runner.comm.all_gather(shard_rows)                       # [tp, n, vs]
            return full.permute(1, 0, 2).reshape(n, self.tp * vs).contiguous()
        per_call = max(1, self.fused.gather_bytes // (vs * shard_rows.element_size()))
        parts = []
        for r0 in range(0, n, per_call):
            g = self.fused.all_gather(shard_rows[r0:r0 + per_call])             # [tp, k, vs]
            parts.append(g.permute(1, 0, 2).reshape(g.shape[1], self.tp * vs))
        return torch.cat(parts, 0).contiguous()

    def _capture(self, Bp: int, splits: int) -> torch.cuda.CUDAGraph:
        m = self._views(Bp, Bp, self.num_pages, False, splits=splits)
        # warm up outside capture: first-use work (attribute setup, descriptor cache, workspace allocation)
        # (its rows carry no state slot: a K/V write repeats itself, a recurrence would advance the state twice)
        slots = m.seq_slot.clone()
        m.seq_slot.fill_(-1)
        self.runner.forward(m)
        m.seq_slot.copy_(slots)
        torch.cuda.current_stream().synchronize()
        g = torch.cuda.CUDAGraph()
        # thread-local capture: transfer and RPC threads of a worker keep making CUDA calls (small copies, flag reads)
        # on their own streams while this thread captures; under the default global mode those calls invalidate
        # the capture ("operation not permitted when stream is capturing")
        with torch.cuda.graph(g, capture_error_mode="thread_local"):
            self.runner.forward(m)
        self._graphs[(Bp, splits)] = g
        return g

    def precapture(self, max_batch: Optional[int] = None, contexts: Sequence[int] = (64, 1024, 4096, 16384)) -> int:
        """Capture the decode graphs of every batch bucket up to `max_batch` (default: the engine's) and of the
        split-KV choices that contexts of the given lengths select, so that no request pays for a capture later.
        The captures run on padded rows only (an empty batch): graph topology and buffer addresses do not depend
        on the parameters' values, so this also works on a replica whose parameters have not arrived.  With tp > 1
        every rank of the replica must call it (the captures contain the collectives).  Returns the number captured."""
        if not self.use_graphs:
            return 0
        limit = min(max_batch or self.max_batch, self.max_batch)
        empty = core.Batch((1 << 62), self.pool)
        n = 0
        for Bp in _BUCKETS:
            if Bp > limit:
                break
            for ctx in contexts:
                splits = self.choose_splits(Bp, ctx)
                if (Bp, splits) in self._graphs:
                    continue
                P = empty.fill_decode(self.host_np, self.layout, Bp)      # Bp padded rows: no page, no cache write
                self._h2d(self.layout.page_indices + P)
                self._capture(Bp, splits)
                n += 1
        torch.cuda.current_stream().synchronize()
        return n

    def release_graphs(self) -> None:
        """Drop every captured decode graph (first step of an orderly exit: the graphs hold kernel arguments that
        name peer memory and, with the NCCL runner, collectives of its communicator)."""
        self._graphs.clear()

    def close_regions(self) -> None:
        """Drop the symmetric regions this engine owns (the fused tensor-parallel state); see parallel/teardown.py."""
        if self.fused is not None:
            self.fused.close_regions()

    def decode_launch_count(self) -> int:
        """Kernels of this library launched by one decode step at tp = 1 (for the bench's launch accounting)."""
        if self.cfg.family == "hybrid":
            return self.runner.decode_launches()
        per_layer = 8  # rms_norm, qkv gemm, rope_kv_store, attention, o gemm, rms_norm, gate_up gemm, down gemm
        return 1 + per_layer * self.cfg.layers + 3  # embedding + layers + final norm, lm_head gemm, argmax

    # ------------------------------------------------------------------ parameters
    def load_checkpoint(self, directory) -> None:
        """Weights straight from a checkpoint folder (.safetensors), without a segment file in between (one GPU)."""
        from ..models.convert import CheckpointReader, checkpoint_to_segment
        if self.tp > 1:
            raise ValueError("sharded replicas load segment files (see models/convert.py)")
        seg = checkpoint_to_segment(CheckpointReader(directory), self.cfg, self.dtype)
        n = self.seg.layout.total_bytes
        self.seg.buffer[:n].copy_(seg.buffer[:n])
        torch.cuda.synchronize()
        self.status.set_ready()

    def set_status_ready(self) -> None:
        self.status.set_ready()

    def reset_status(self) -> None:
        self.status.reset()

    def load_params_from_host(self, host_mirror: torch.Tensor, chunk_bytes: int = 256 << 20) -> float:
        """Chunked H2D of a pinned host mirror on two streams; returns seconds."""
        n = self.seg.layout.total_bytes
        assert host_mirror.numel() >= n and host_mirror.dtype == torch.uint8
        t0 = time.perf_counter()
        streams = [torch.cuda.Stream(device=self.device) for _ in range(2)]
        for i, off in enumerate(range(0, n, chunk_bytes)):
            hi = min(n, off + chunk_bytes)
            with torch.cuda.stream(streams[i % 2]):
                self.seg.buffer[off:hi].copy_(host_mirror[off:hi], non_blocking=True)
        for s in streams:
            s.synchronize()
        self.status.set_ready()
        return time.perf_counter() - t0

    def load_params_from_disk(self, directory, host_mirror: Optional[torch.Tensor] = None) -> dict:
        """Disk -> pinned host (O_DIRECT, threaded) -> device.  Returns timings."""
        path = WeightSegment.check_sidecar(directory, self.cfg, self.tp, self.tp_rank, self.dtype)
        n = self.seg.layout.total_bytes
        if host_mirror is None:
            host_mirror = torch.empty(n, dtype=torch.uint8, pin_memory=True)
        res = core.load_file_to_host(str(path), host_mirror.data_ptr(), n)
        h2d = self.load_params_from_host(host_mirror)
        return {"disk_s": res.seconds, "h2d_s": h2d, "bytes": n, "direct_io": res.direct_io, "host_mirror": host_mirror}
