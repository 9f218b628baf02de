"""Per-sequence memory of a hybrid model: a paged KV pool per attention run and a state slot per recurrent run.

A page id addresses the same page in the pool of every attention run, and a slot id the same slot in the state arrays
of every recurrent run, so the host bookkeeping (native PagePool, SlotPool and Batch) does not know how many runs there
are or what shape each has.  A layer that runs several times in one forward pass has one entry per run; a layer that
reads another layer's keys and values has that layer's pool as its entry.

A mixer that consists of two has the pool of one and the state of the other in its entry.

A pool is one tensor with a key and a value plane per page, or a pair of tensors where keys and values differ in size, or one
tensor of latent rows.

Slots are not cleared when they change hands: the kernels start from zero at position 0.  KV pools are zero-filled once
(the attention kernels require finite values in every slot of an allocated page)."""
from __future__ import annotations

from dataclasses import dataclass
from typing import List, Optional, Union

import torch

from ..models.hybrid_config import HybridConfig, mixer_parts
from ..ops import KVPair, LatentKV


@dataclass
class RunCache:
    # [pages, 2, page, kv_heads, dim], or two [pages, page, kv_heads, size], or latent rows [pages, page, 1, width]
    kv: Optional[Union[torch.Tensor, KVPair, LatentKV]] = None
    state: Optional[torch.Tensor] = None   # fp32: [slots, heads, dim, vdim] (keys or state by values) or [slots, width]
    hist: Optional[torch.Tensor] = None    # last inputs of a short convolution: [slots, taps - 1, width]
    mix_hist: Optional[torch.Tensor] = None  # the same of the convolution of a mixer's input, fp32
    shift: Optional[torch.Tensor] = None   # a mixer's last input: [slots, width], fp32


class HybridCache:
    def __init__(self, cfg: HybridConfig, num_pages: int, page_size: int, num_slots: int, dtype, device):
        self.cfg, self.num_pages, self.page_size, self.num_slots = cfg, num_pages, page_size, num_slots
        self.runs: List[RunCache] = []
        zeros = lambda *shape: torch.zeros(*shape, dtype=dtype, device=device)
        for r, (m, source) in enumerate(zip(cfg.run_mixers(), cfg.kv_runs())):
            rc = RunCache()
            self.runs.append(rc)
            if cfg.mix_taps:
                rc.mix_hist = torch.zeros(num_slots, cfg.mix_taps - 1, cfg.hidden, device=device)
            for m in mixer_parts(m):
                if m.kind == "attention" and source != r:
                    rc.kv = self.runs[source].kv
                elif m.kind == "latent":
                    rc.kv = LatentKV(zeros(num_pages, page_size, 1, m.width), m.kv_rank)
                elif m.kind == "attention" and m.vdim != m.dim:
                    rc.kv = KVPair(*(zeros(num_pages, page_size, m.kv_heads, n) for n in (m.dim, m.vdim)))
                elif m.kind == "attention":
                    rc.kv = zeros(num_pages, 2, page_size, m.kv_heads, m.dim)
                elif m.kind in ("gla", "wkv"):
                    rc.state = torch.zeros(num_slots, m.heads, m.dim, m.vdim, device=device)
                    if m.kind == "wkv":
                        rc.shift = torch.zeros(num_slots, m.hidden, device=device)
                elif m.kind == "ssd":
                    rc.state = torch.zeros(num_slots, m.heads, m.state, m.vdim, device=device)
                    rc.hist = zeros(num_slots, m.taps - 1, m.channels)
                else:
                    rc.state = torch.zeros(num_slots, m.width, device=device)
                    rc.hist = zeros(num_slots, m.taps - 1, m.width)

    def bytes(self) -> int:
        held = {}
        for r in self.runs:
            pools = r.kv if isinstance(r.kv, KVPair) else (r.kv.pool,) if isinstance(r.kv, LatentKV) else (r.kv,)
            for t in (*pools, r.state, r.hist, r.mix_hist, r.shift):
                if t is not None:
                    held[t.data_ptr()] = t.numel() * t.element_size()
        return sum(held.values())
