"""Forward pass of hybrid models (hybrid_config.py) over the weight segment, the paged KV pools and the state slots.

A layer run with its feed-forward beside the mixer is: one norm (with whatever is added to the stream before it), one product for all projections of the
mixer, the mixer's own kernels, one product for gate and up with SiLU * mul in its epilogue, and one product that adds
``m * (mixer + feed-forward)`` to the fp32 stream in its epilogue::

    stream_norm -> GEMM (in) -> mixer -> GEMM (gate||up, SiLU*mul) -> GEMM (out, fp32 axpy)

A layer run with experts behind the mixer::

    stream_norm -> GEMM (in) -> mixer -> GEMM (out, fp32 axpy)
    -> stream_norm -> GEMM (router, fp32) -> moe_route -> grouped GEMM (up, act) -> grouped GEMM (down)

The experts' output rows stay where the last product leaves them: the next layer's norm kernel adds them to the stream
(`flush` does where a pass ends).

A model with several residual streams: every sublayer starts with one kernel that lets the streams take up the output of the
sublayer before it, joins them and norms the result::

    stream_mix -> GEMM (in) -> mixer -> GEMM (out)
    -> stream_mix -> GEMM (gate||up, SiLU*mul) -> GEMM (down)     or router, moe_route and the grouped products as above

With RMS norms that kernel is stream_rms.  Mixers may read their input plus a causal convolution of it (and the mixes of a token
shift): stream_rms does that too where every row is one token, token_conv behind it where there are longer rows.

    attention: rope_store (biases, rotation, paged write) or norm_store (norm of every head, paged write)
               -> attention over the pages (window, cap, sink, gate per head, bias by distance)
    latent:    latent_store (norms, shared rotated key, paged write) -> GEMM (queries), then
               single tokens: block-diagonal GEMM (queries into the latent space) -> rotation -> attention over the cached
               rows, one key and value for all heads -> block-diagonal GEMM (values out of the latent space);
               prompts: rotation -> gather of the cached rows -> GEMMs (keys, values of all heads) -> attention
               (heads that the prompt kernel does not take: as single tokens)
    gla:       one kernel (decay projection, recurrence, output norm, gate), or the chunked kernels for prompts
    rglru:     conv_causal -> block-diagonal GEMM (gates, fp32 out) -> rglru_scan
    wkv:       one block-diagonal GEMM over the mixes (receptance, keys, values, gates), GEMM (decay, fp32 out) -> recurrence with
               output norm and gate, or the chunked kernels for prompts
    parallel:  attention as above (norm over whole rows with the rotation; chunks, sigmoid weights), and
               token_conv (SiLU) -> state-space recurrence with gate, or the chunked kernel for prompts -> norm in parts;
               an output product each, side by side: the next stream_rms norms and adds them

A step may hold rows of any length (StepMeta.singles of one token first): single tokens go to the decode kernels, the
others to the prefill kernels, everything else runs over all tokens at once.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from .. import ops
from ..runtime.hybrid_cache import HybridCache
from .hybrid_config import (AttentionMixer, ExpertsSpec, GLAMixer, HybridConfig, LatentAttentionMixer, LayerSpec, ParallelMixer, RGLRUMixer,
                            SSDMixer, WKVMixer)
from .llama import StepMeta
from .weights import WeightSegment


class HybridRunner:
    def __init__(self, seg: WeightSegment, cache: HybridCache, max_tokens: int, max_batch: int):
        cfg: HybridConfig = seg.cfg
        self.cfg, self.seg, self.cache = cfg, seg, cache
        self.runs = cfg.runs()
        self.page_size = cache.page_size
        self.max_tokens, self.max_batch = max_tokens, max_batch
        dev, dt = seg.buffer.device, seg.dtype
        H = cfg.hidden
        # residual stream, or streams
        self.res = torch.empty(*(max_tokens, cfg.streams, H) if cfg.streams else (max_tokens, H), dtype=torch.float32, device=dev)
        self.normed = torch.empty(max_tokens, H, dtype=dt, device=dev)
        self._proj = torch.empty(max_tokens * max(s.in_columns()[1] for s in cfg.layer_specs), dtype=dt, device=dev)
        # mixer output and feed-forward activation side by side, one buffer per column layout: its padding columns stay
        # zero because nothing ever writes them
        self._mid: Dict[tuple, torch.Tensor] = {}
        for s in cfg.layer_specs:
            key = self._mid_key(s)
            if key not in self._mid:
                self._mid[key] = torch.zeros(max_tokens, s.out_rows, dtype=dt, device=dev)
        rw = max((m.width for m in cfg.run_mixers() if m.kind == "rglru"), default=0)
        cw = max([rw] + [m.channels for m in cfg.run_parts() if m.kind == "ssd"])
        self._conv = torch.empty(max_tokens * cw, dtype=dt, device=dev) if cw else None
        self._gates = torch.empty(max_tokens * 2 * rw, dtype=torch.float32, device=dev) if rw else None
        ck = max((m.heads * m.dim for m in cfg.run_mixers() if m.kind in ("gla", "wkv")), default=0)
        self._cum = torch.empty(max_tokens * ck, dtype=torch.float32, device=dev) if ck and dt == torch.bfloat16 else None
        self._init_experts(max_tokens, dev, dt)
        self._init_streams(max_tokens, max_batch, dev, dt)
        self._init_latent(max_tokens, max_batch, dev, dt)
        self._init_shift(max_tokens, max_batch, dev, dt)
        self.last = torch.empty(max_batch, H, dtype=torch.float32, device=dev)
        self._logits_pad = torch.zeros(max_batch, cfg.vocab_pad, dtype=torch.float32, device=dev)
        self.logits = self._logits_pad[:, :cfg.vocab]
        self.tokens = torch.empty(max_batch, dtype=torch.int32, device=dev)
        self._freqs = {}
        for m in cfg.run_parts():
            if m.kind == "attention" and self._rot_key(m) not in self._freqs:
                stretch = m.yarn.stretch(m.rot_dims, m.rot_base) if m.yarn else None
                self._freqs[self._rot_key(m)] = ops.rope_freqs(m.rot_dims, m.rot_base, dev, stretch)
            elif m.kind == "latent":
                self._freqs[(m.rot_dim, m.rot_base, None)] = ops.rope_freqs(m.rot_dim, m.rot_base, dev)
        self._ws: Optional[torch.Tensor] = None
        self._ws_old: List[Optional[torch.Tensor]] = []

    @staticmethod
    def _mid_key(s: LayerSpec) -> tuple:
        return (s.mixer.out_width, s.ff)

    @staticmethod
    def _rot_key(m: AttentionMixer) -> tuple:
        return (m.rot_dims, m.rot_base, m.yarn)

    def _w(self, l: int, name: str) -> torch.Tensor:
        return self.seg[f"layers.{l}.{name}"]

    def _init_experts(self, max_tokens: int, dev, dt) -> None:
        """Buffers of the layers with experts: router logits, work lists (one per shape of router), activations of the sorted
        rows, and output rows."""
        moes = [s.moe for s in self.cfg.layer_specs if s.moe]
        self._pending: Optional[tuple] = None        # output rows of experts that are not in the stream yet, and where they go
        self._plans: Dict[tuple, ops.ExpertPlan] = {}
        if not moes:
            return
        for e in moes:
            key = self._plan_key(e)
            if key not in self._plans:
                self._plans[key] = ops.ExpertPlan(max_tokens, e.experts, e.top, bool(e.shared_ff), dev, e.identity)
        rows = max_tokens * max(e.per_token for e in moes)
        self._router = torch.empty(max_tokens * max(e.router_cols for e in moes), dtype=torch.float32, device=dev)
        self._act = torch.empty(rows * max(max(e.ff_pad, e.shared_pad) for e in moes), dtype=dt, device=dev)
        self._expert_out = torch.empty(rows, self.cfg.hidden, dtype=dt, device=dev)

    @staticmethod
    def _plan_key(e: ExpertsSpec) -> tuple:
        return (e.experts, e.top, bool(e.shared_ff), e.identity)

    def _init_streams(self, max_tokens: int, max_batch: int, dev, dt) -> None:
        """Buffers of a model with several streams: the last sublayer's output, a feed-forward's activations, the head's input."""
        c = self.cfg
        self._fresh = False          # the streams are still the embeddings (of self._ids) and not in memory
        self._ids: Optional[torch.Tensor] = None
        if not c.streams:
            return
        pair = any(m.kind == "parallel" for m in c.run_mixers())
        self._y = torch.empty(max_tokens * (2 if pair else 1), c.hidden, dtype=dt, device=dev)
        self._head_in = torch.empty(max_batch, c.hidden, dtype=dt, device=dev)
        ff = max(s.ff_after_pad for s in c.layer_specs)
        self._ff = torch.empty(max_tokens * ff, dtype=dt, device=dev) if ff else None

    def _init_latent(self, max_tokens: int, max_batch: int, dev, dt) -> None:
        """Buffers of latent attention: queries, and queries and outputs in the latent space (of single tokens where the prompts'
        keys and values are expanded, else of all tokens)."""
        ms = [m for m in self.cfg.run_mixers() if m.kind == "latent"]
        self._scratch: Dict[str, torch.Tensor] = {}
        if not ms:
            return
        self._latent_ws = max((ops.attn_latent_workspace(m.heads, m.kv_rank, dev) for m in ms), key=torch.Tensor.numel)
        rows = lambda m: max_batch if self._expands(m, dt) else max_tokens
        self._q = torch.empty(max_tokens * max(m.heads * m.qdim for m in ms), dtype=dt, device=dev)
        self._q_latent = torch.empty(max(rows(m) * m.heads * m.width for m in ms), dtype=dt, device=dev)
        self._o_latent = torch.empty(max(rows(m) * m.heads * m.kv_rank for m in ms), dtype=dt, device=dev)

    def _init_shift(self, max_tokens: int, max_batch: int, dev, dt) -> None:
        """Buffers of convolved mixer inputs, token shifts and mixers side by side."""
        c = self.cfg
        wkv = [m for m in c.run_mixers() if m.kind == "wkv"]
        mixes = max([1 if c.mix_taps else 0] + [len(m.MIXES) for m in wkv])
        self._mixed = torch.empty(max_tokens * mixes * c.hidden, dtype=dt, device=dev) if mixes else None
        # what the convolution reads is not rounded
        self._unmixed = torch.empty(max_tokens, c.hidden, dtype=torch.float32, device=dev) if mixes else None
        if wkv:
            self._last_h = torch.empty(max_batch, c.hidden, dtype=torch.float32, device=dev)
            self._rkvg = torch.empty(max_tokens * 4 * max(m.out_width for m in wkv), dtype=dt, device=dev)
            self._low = torch.empty(max_tokens * max(m.rank + 7 for m in wkv), dtype=torch.float32, device=dev)
        # (padding columns stay zero because nothing ever writes them)
        self._mid_right = {m.right.out_width: torch.zeros(max_tokens, m.right_rows, dtype=dt, device=dev)
                           for m in c.run_mixers() if m.kind == "parallel"}

    def _expands(self, m: LatentAttentionMixer, dt) -> bool:
        """Whether prompts run over expanded keys and values on the tensor cores (else over the latent rows)."""
        return dt != torch.float32 and ops.attn_head_sizes(m.qdim, m.vdim, self.page_size) and m.width % 8 == 0

    # ------------------------------------------------------------------ pieces
    def embed(self, m: StepMeta) -> None:
        """Nothing: the first layer run's norm kernel starts the stream from the embedding table."""

    def run_layer(self, r: int, m: StepMeta) -> None:
        """Layer run `r` (an index into the executions of a pass, not a layer number)."""
        run, T, c = self.runs[r], m.num_tokens, self.cfg
        l = run.layer
        spec = c.layer_specs[l]
        if c.streams:
            return self._run_layer_streams(r, l, spec, m)
        step = self.seg["loop_step"][run.step] if run.step >= 0 else None
        h = self.normed[:T]
        needs_ids = r == 0 or run.add_embed
        if r == 0:
            self._pending = None
        ops.stream_norm(self.res[:T], self._w(l, "norm1"), c.rms_eps, h, w_offset=c.norm_offset, ids=m.ids if needs_ids else None,
                        embed=self.seg["embed"] if needs_ids else None, init=r == 0, add_embed=run.add_embed, step=step,
                        **self._take_pending())
        cols, width = spec.in_columns()
        proj = self._proj[:T * width].view(T, width)
        ops.gemm(h, self._w(l, "in"), out=proj, static_b=True)
        mid = self._mid[self._mid_key(spec)][:T]
        parts = {n: proj[:, at:at + w] for n, (at, w) in cols.items()}
        getattr(self, "_" + spec.mixer.kind)(r, l, spec.mixer, parts, mid, m)
        if spec.ff:
            ops.gemm(h, self._w(l, "gate_up"), out=mid[:, spec.mix_rows:], epilogue="silu_mul", static_b=True)
        ops.gemm(mid, self._w(l, "out"), out=self.res[:T], epilogue="axpy", alpha=c.residual_mult, static_b=True)
        if spec.moe:
            ops.stream_norm(self.res[:T], self._w(l, "norm2"), c.rms_eps, h, w_offset=c.norm_offset)
            out, plan = self._experts(l, spec.moe, h)
            self._pending = (out, plan.place)

    def _streams(self, norm: Optional[str] = None, **what) -> None:
        """The streams take up what is pending (``write``: and keep it) and are joined; ``norm``: name of the norm of ``out``."""
        what.update(self._embeddings(), pending=self._pending)
        if self.cfg.norm == "tanh":
            weights = dict(norm=(self.seg[norm], self.seg[norm + "_alpha"], self.seg[norm + "_b"])) if norm else {}
            ops.stream_mix(self.res, **what, **weights)
        else:
            ops.stream_rms(self.res, eps=self.cfg.rms_eps, w=self.seg[norm] if norm else None, w_offset=self.cfg.norm_offset, **what)

    def _join(self, l: int, q: int, T: int, **more) -> torch.Tensor:
        """Input of sublayer q of layer l; the streams take up what is pending."""
        take, h = self._pending is not None, more.pop("out", self.normed[:T])
        self._streams(f"layers.{l}.norm{q}", n=T, read=self._w(l, f"hc{q}_in"), out=h, write=take, **more)
        self._fresh = self._fresh and not take
        return h

    def _join_convolved(self, r: int, l: int, mx, m: StepMeta) -> torch.Tensor:
        """Input of the mixer of layer l: the norm's output plus its causal convolution, or with a token shift its mixes [T, mixes *
        hidden]."""
        T, H, rc = m.num_tokens, self.cfg.hidden, self.cache.runs[r]
        mu = self._w(l, "mu") if mx.kind == "wkv" else None
        width = H * (mu.shape[0] if mu is not None else 1)
        out = self._mixed[:T * width].view(T, width)
        conv = self._w(l, "mix_conv")
        if not m.is_prefill:
            return self._join(l, 1, T, out=out, tokens=ops.TokenState(conv, rc.mix_hist, mu, rc.shift), pos=m.pos, seq_slot=m.seq_slot)
        h = self._join(l, 1, T, out=self._unmixed[:T])
        shift = dict(mu=mu, shift=rc.shift, last=self._last_h) if mu is not None else {}
        return ops.token_conv(h, conv, rc.mix_hist, out, m.pos, m.tok_indptr, m.seq_slot, residual=True, **shift)

    def _embeddings(self) -> dict:
        return dict(ids=self._ids, embed=self.seg["embed"]) if self._fresh else {}

    def _leave(self, l: int, q: int, y: torch.Tensor, **rows) -> None:
        self._pending = ops.Pending(y, self._w(l, f"hc{q}_mix"), self._w(l, f"hc{q}_out"), **rows)

    def _run_layer_streams(self, r: int, l: int, spec: LayerSpec, m: StepMeta) -> None:
        T, c = m.num_tokens, self.cfg
        if r == 0:
            self._pending, self._fresh, self._ids = None, True, m.ids
        h, y = self._join_convolved(r, l, spec.mixer, m) if c.mix_taps else self._join(l, 1, T), self._y[:T]
        cols, width = spec.in_columns()
        mid = self._mid[self._mid_key(spec)][:T]
        if spec.mixer.kind == "wkv":                 # its projections have an input each
            self._wkv(r, l, spec.mixer, h, mid, m)
        else:
            proj = self._proj[:T * width].view(T, width)
            ops.gemm(h, self._w(l, "in"), out=proj, static_b=True)
            getattr(self, "_" + spec.mixer.kind)(r, l, spec.mixer, {n: proj[:, at:at + w] for n, (at, w) in cols.items()}, mid, m)
        if spec.mixer.kind == "parallel":
            both, H = self._y[:2 * T].view(T, 2 * c.hidden), c.hidden
            ops.gemm(mid, self._w(l, "out"), out=both[:, :H], static_b=True)
            ops.gemm(self._mid_right[spec.mixer.right.out_width][:T], self._w(l, "r_out"), out=both[:, H:], static_b=True)
            self._leave(l, 1, both, norms=(self._w(l, "l_out_norm"), self._w(l, "r_out_norm")))
        else:
            ops.gemm(mid, self._w(l, "out"), out=y, static_b=True)
            self._leave(l, 1, y)
        if spec.ff_after:
            h = self._join(l, 2, T)
            act = self._ff[:T * spec.ff_after_pad].view(T, spec.ff_after_pad)
            unit = (dict(epilogue="clamp_glu", alpha=spec.unit.limit, beta=spec.unit.beta, bias=self._w(l, "gate_up_b")) if spec.unit
                    else dict(epilogue="silu_mul"))
            ops.gemm(h, self._w(l, "gate_up"), out=act, static_b=True, **unit)
            ops.gemm(act, self._w(l, "down"), out=y, static_b=True)
            self._leave(l, 2, y, **(dict(bias=self._w(l, "down_b")) if spec.unit else {}))
        elif spec.moe:
            h = self._join(l, 2, T)
            out, plan = self._experts(l, spec.moe, h)
            self._leave(l, 2, out, place=plan.place, ident=plan.ident, prev=h if spec.moe.identity else None)

    def _take_pending(self) -> dict:
        p, self._pending = self._pending, None
        return dict(add=p[0], add_rows=p[1]) if p else {}

    def flush(self, T: int) -> None:
        """Everything the layers so far have produced is in the stream (several streams: what reads them takes it up)."""
        if self._pending and not self.cfg.streams:
            ops.stream_norm(self.res[:T], None, 0.0, None, **self._take_pending())

    def _experts(self, l: int, e: ExpertsSpec, h: torch.Tensor) -> tuple:
        """Output rows of the chosen experts, and the plan that says whose they are."""
        T, H = h.shape
        plan = self._plans[self._plan_key(e)]
        z = self._router[:T * e.router_cols].view(T, e.router_cols)
        # few columns: beyond a decode batch, narrow tiles with K split keep more SMs loading
        narrow = dict(bn=64, split_k=4 if T <= 2048 else 1) if T > ops.DECODE_GEMM_MAX_M else {}
        ops.gemm(h, self._w(l, "router"), out=z, static_b=True, **narrow)
        up, down = self._w(l, "up").view(e.experts, H, e.up_cols), self._w(l, "down").view(e.experts, e.ff_pad, H)
        s_up, s_down = (self._w(l, "shared_up"), self._w(l, "shared_down")) if e.shared_ff else (None, None)
        tc = ops.grouped_tensor_core(h, up, down, s_up, s_down)
        ops.moe_route(z, plan, weight_on_input=e.weight_on_input, renormalize=e.renormalize, softmax=e.softmax,
                      correction=self._w(l, "correction") if e.correction else None, groups=e.groups, keep=e.keep,
                      tile_rows=128 if tc else 64)
        width = max(e.ff_pad, e.shared_pad)
        act, out = self._act[:plan.rows * width].view(plan.rows, width), self._expert_out[:plan.rows]
        ops.gemm_grouped(h, up, plan, act, shared=s_up, gather=True, act="silu_gate" if e.gated else "relu2", factors=True)
        ops.gemm_grouped(act, down, plan, out, shared=s_down)
        return out, plan

    def _attention(self, r: int, l: int, mx: AttentionMixer, p: Dict[str, torch.Tensor], mid: torch.Tensor, m: StepMeta,
                   prefix: str = "") -> None:
        T, kv = m.num_tokens, self.cache.runs[r].kv
        w = lambda n: self._w(l, prefix + n)
        if mx.qk_norm:
            temp = dict(temp_coef=mx.q_temp.coef, temp_every=mx.q_temp.every) if mx.q_temp else {}
            ops.norm_store(p["q"], p["k"], p["v"], m.pos, m.slot, kv, w("q_norm"), w("k_norm"), q_heads=mx.heads,
                           kv_heads=mx.kv_heads, dim=mx.dim, page_size=self.page_size, eps=self.cfg.rms_eps, **temp)
        else:
            biases = {n + "_b": w(n + "_b") for n in ("q", "k", "v") if mx.bias and n in p}
            if mx.whole_norm:
                biases = dict(q_w=w("q_norm"), k_w=w("k_norm"), eps=self.cfg.rms_eps)
            ops.rope_store(p["q"], p.get("k"), p.get("v"), m.pos, m.slot, kv, self._freqs[self._rot_key(mx)], q_heads=mx.heads,
                           kv_heads=mx.kv_heads, dim=mx.dim, rot_dims=mx.rot_dims, page_size=self.page_size,
                           interleaved=mx.interleaved, gain=mx.yarn.gain if mx.yarn else 1.0, **biases)
        extra = dict(window=mx.window, keep_first=mx.keep_first, softcap=mx.softcap, sink=w("sink") if mx.sink else None,
                     bias=w("rel_by_distance") if mx.rel else w("weight_b") if mx.sigmoid else None, chunked=mx.chunked, sigmoid=mx.sigmoid)
        gate = p.get("g")
        if not ops.attn_tensor_core(p["q"], mx.heads, mx.kv_heads, mx.dim, self.page_size, mx.vdim):
            ops.attn_ragged(p["q"], kv, m.pos, m.tok_indptr if m.is_prefill else None, m.page_indptr, m.page_indices, mid,
                            q_heads=mx.heads, kv_heads=mx.kv_heads, dim=mx.dim, page_size=self.page_size, scale=mx.scale, gate=gate, **extra)
            return
        args = dict(q_heads=mx.heads, kv_heads=mx.kv_heads, head_dim=mx.dim, page_size=self.page_size, sm_scale=mx.scale, **extra)
        ns = m.singles if m.is_prefill else m.batch
        if ns:
            ops.attn_decode(p["q"][:ns], kv, m.page_indices, m.page_indptr[:ns + 1], m.last_page_len[:ns],
                            num_splits=m.num_splits, workspace=self._workspace(ns, mx, m.num_splits), out=mid[:ns],
                            gate=gate[:ns] if gate is not None else None, **args)
        if m.batch > ns:
            ops.attn_prefill_paged(p["q"], kv, m.page_indices, m.prefill_work, out=mid, gate=gate, **args)

    def _workspace(self, B: int, mx: AttentionMixer, splits: int) -> Optional[torch.Tensor]:
        if splits <= 1:
            return None
        n = ops.attn_decode_workspace_bytes(B, mx.heads, mx.vdim, splits)
        if self._ws is None or self._ws.numel() < n:
            # an earlier buffer may be named by captured graphs: keep it
            self._ws_old.append(self._ws)
            self._ws = torch.empty(n, dtype=torch.uint8, device=self.res.device)
        return self._ws

    def _latent(self, r: int, l: int, mx: LatentAttentionMixer, p: Dict[str, torch.Tensor], mid: torch.Tensor, m: StepMeta) -> None:
        T, H, R, W, kv = m.num_tokens, mx.heads, mx.kv_rank, mx.width, self.cache.runs[r].kv
        freqs, gate = self._freqs[(mx.rot_dim, mx.rot_base, None)], p.get("g")
        ops.latent_store(p["dq"], p["dkv"], m.pos, m.slot, kv, self._w(l, "dq_norm"), self._w(l, "dkv_norm"), freqs, eps=self.cfg.rms_eps,
                         interleaved=mx.interleaved)
        q = self._q[:T * H * mx.qdim].view(T, H * mx.qdim)
        ops.gemm(p["dq"], self._w(l, "uq"), out=q, static_b=True)
        rotate = dict(heads=H, dim=mx.dim, rot=mx.rot_dim, interleaved=mx.interleaved)
        extra = dict(window=mx.window, sink=self._w(l, "sink") if mx.sink else None)
        n = m.batch if not m.is_prefill else m.singles if self._expands(mx, q.dtype) else T    # rows that go through the latent space
        if n:
            ql, ol = self._q_latent[:n * H * W].view(n, H * W), self._o_latent[:n * H * R].view(n, H * R)
            ops.gemm(q[:n], self._w(l, "uk"), out=ql, groups=H, a_step=mx.qdim, out_step=W, static_b=True)
            ops.latent_rotate(q[:n], ql[:, R:], m.pos[:n], freqs, out_step=W, **rotate)
            single = not m.is_prefill or n == m.singles
            g = gate[:n] if gate is not None else None
            if ops.attn_latent_supported(ql, n if single else min(n, ops.ATTN_LATENT_ROWS), H, kv):
                rows = m.batch if not single else n
                ops.attn_latent(ql, kv, m.page_indices, m.page_indptr[:rows + 1], m.last_page_len[:rows], heads=H, scale=mx.scale,
                                workspace=self._latent_ws, out=ol, gate=g, static_table=True, **extra,
                                **({} if single else dict(pos=m.pos[:n], tok_indptr=m.tok_indptr)))
            else:
                ops.attn_ragged(ql, kv, m.pos, None if single else m.tok_indptr, m.page_indptr[:n + 1] if single else m.page_indptr,
                                m.page_indices, ol, q_heads=H, kv_heads=1, dim=W, page_size=self.page_size, scale=mx.scale, gate=g, **extra)
            # few rows: a tile per head is enough, and an exchange of K splits would cost more than it saves
            narrow = dict(bn=64, split_k=1) if n <= ops.PAIR_GEMM_MAX_M else {}
            ops.gemm(ol, self._w(l, "uv"), out=mid[:n, :H * mx.vdim], groups=H, a_step=R, out_step=mx.vdim, static_b=True, **narrow)
        if n < T:
            self._latent_prompts(l, mx, q, gate, kv, mid, m, n, freqs, rotate, extra)

    def _latent_prompts(self, l: int, mx: LatentAttentionMixer, q, gate, kv: ops.LatentKV, mid, m: StepMeta, n: int, freqs, rotate, extra) -> None:
        """Rows from n on: keys and values of all their sequences' cached rows are expanded into a pool of their own, some heads
        at a time where that would be large.  With a window only the pages that one of a sequence's rows sees."""
        ops.latent_rotate(q[n:], q[n:, mx.dim:], m.pos[n:], freqs, out_step=mx.qdim, **rotate)
        ps = self.page_size
        index, pages, np_ = self._expanded_pages(m, n, mx.window, q.device)
        rows = ops.latent_gather(kv, pages, self._room("rows", (np_ * ps, mx.width), q.dtype))
        H = mx.heads
        heads = max(1, min(H, self.EXPANDED_BYTES // (np_ * ps * (mx.qdim + mx.vdim) * 2)))
        for h0 in range(0, H, heads):
            hn = min(heads, H - h0)
            k = self._room("keys", (np_, ps, hn, mx.qdim), q.dtype)
            v = self._room("values", (np_, ps, hn, mx.vdim), q.dtype)
            ops.gemm(rows, self._w(l, "k_up")[:, h0 * mx.qdim:(h0 + hn) * mx.qdim], out=k.view(np_ * ps, -1), static_b=True)
            ops.gemm(rows[:, :mx.kv_rank], self._w(l, "v_up")[:, h0 * mx.vdim:(h0 + hn) * mx.vdim], out=v.view(np_ * ps, -1), static_b=True)
            ops.attn_prefill_paged(q[:, h0 * mx.qdim:(h0 + hn) * mx.qdim], ops.KVPair(k, v), index, m.prefill_work, q_heads=hn, kv_heads=hn,
                                   head_dim=mx.qdim, page_size=ps, sm_scale=mx.scale, out=mid[:, h0 * mx.vdim:(h0 + hn) * mx.vdim],
                                   gate=gate[:, h0:h0 + hn] if gate is not None else None, window=extra["window"],
                                   sink=extra["sink"][h0:h0 + hn] if extra["sink"] is not None else None)

    def _expanded_pages(self, m: StepMeta, n: int, window: int, dev) -> tuple:
        """For the sequences from n on: where their page entries are in the expanded pool, the pages it holds, and how many."""
        ps = self.page_size
        pages = [-(-kv_len // ps) for kv_len in m.kv_lens_host]
        first, total = sum(pages[:n]), sum(pages)
        if not window:       # page i of the expanded pool is the i-th page of these sequences
            return torch.arange(-first, total - first, dtype=torch.int32, device=dev), m.page_indices[first:total], total - first
        key = (n, window)
        if self._expanded is None or self._expanded[0] is not m or key not in self._expanded[1]:
            index, need, at = [0] * first, [], first
            for s in range(n, len(pages)):
                # (the attention kernel walks whole blocks of keys)
                lo = max(0, m.kv_lens_host[s] - m.seq_lens_host[s] - window + 1) // ops.PREFILL_KEY_BLOCK * ops.PREFILL_KEY_BLOCK // ps
                index += [0] * lo + list(range(len(need), len(need) + pages[s] - lo))
                need += range(at + lo, at + pages[s])
                at += pages[s]
            both = torch.tensor(index + need, dtype=torch.int32).to(dev, non_blocking=True)
            if self._expanded is None or self._expanded[0] is not m:
                self._expanded = (m, {})
            self._expanded[1][key] = (both[:len(index)], m.page_indices.index_select(0, both[len(index):]), len(need))
        return self._expanded[1][key]

    _expanded: Optional[tuple] = None       # (step, tables) of the last prefill pass
    EXPANDED_BYTES = 1 << 30      # of expanded keys and values at a time

    def _room(self, name: str, shape: tuple, dt) -> torch.Tensor:
        """Scratch of a prefill pass (grows with the longest one)."""
        n = 1
        for s in shape:
            n *= s
        have = self._scratch.get(name)
        if have is None or have.numel() < n:
            have = self._scratch[name] = torch.empty(n, dtype=dt, device=self.res.device)
        return have[:n].view(shape)

    def _gla(self, r: int, l: int, mx: GLAMixer, p: Dict[str, torch.Tensor], mid: torch.Tensor, m: StepMeta) -> None:
        ns = m.batch if not m.is_prefill else m.singles
        args = dict(rank=mx.rank, tau=mx.tau, eps=self.cfg.rms_eps)
        w = [self._w(l, n) for n in ("a2", "a2_b", "o_norm")]
        parts = [p[n] for n in ("q", "k", "v", "g", "low")]
        state = self.cache.runs[r].state
        if ns:
            ops.gla_recurrent(*parts, *w, state, mid, m.pos, None, m.seq_slot[:ns], **args)
        if m.batch > ns:
            ops.gla(*parts, *w, state, mid, m.pos, m.tok_indptr[ns:], m.seq_slot[ns:], row_lens=m.seq_lens_host[ns:],
                    cum=self._cum, **args)

    def _rglru(self, r: int, l: int, mx: RGLRUMixer, p: Dict[str, torch.Tensor], mid: torch.Tensor, m: StepMeta) -> None:
        T, rc = m.num_tokens, self.cache.runs[r]
        u = self._conv[:T * mx.width].view(T, mx.width)
        gates = self._gates[:T * 2 * mx.width].view(T, 2 * mx.width)
        indptr = m.tok_indptr if m.is_prefill else None
        ops.conv_causal(p["x"], self._w(l, "x_b"), self._w(l, "conv"), self._w(l, "conv_b"), rc.hist, u, m.pos, indptr, m.seq_slot)
        ops.gemm(u, self._w(l, "gates"), out=gates, groups=mx.blocks, static_b=True)
        ops.rglru_scan(u, gates, self._w(l, "gate_b"), self._w(l, "lam"), p["y"], p["x"], self._w(l, "y_b"), rc.state, rc.hist,
                       mid, m.pos, indptr, m.seq_slot, block=mx.block)

    def _wkv(self, r: int, l: int, mx: WKVMixer, h: torch.Tensor, mid: torch.Tensor, m: StepMeta) -> None:
        """h: the mixes, [T, 5 * hidden]."""
        T, H, N, rc = m.num_tokens, self.cfg.hidden, mx.out_width, self.cache.runs[r]
        out = self._rkvg[:T * 4 * N].view(T, 4 * N)
        ops.gemm(h[:, :4 * H], self._w(l, "rkvg"), out=out, groups=4, static_b=True)
        w1 = self._w(l, "w1")
        low = self._low[:T * w1.shape[1]].view(T, w1.shape[1])
        narrow = dict(bn=64, split_k=4 if T <= 2048 else 1) if T > ops.DECODE_GEMM_MAX_M else {}     # as for a router's columns
        ops.gemm(h[:, 4 * H:], w1, out=low, static_b=True, **narrow)
        parts = [out[:, i * N:(i + 1) * N] for i in range(4)]
        weights = [self._w(l, n) for n in ("w2", "w0", "bonus", "o_norm")]
        args = dict(rank=mx.rank, eps=self.cfg.rms_eps)
        ns = m.batch if not m.is_prefill else m.singles
        if ns:
            ops.wkv(*parts, low, *weights, rc.state, mid, m.pos, None, m.seq_slot[:ns], **args)
        if m.batch > ns:
            ops.wkv(*parts, low, *weights, rc.state, mid, m.pos, m.tok_indptr[ns:], m.seq_slot[ns:], row_lens=m.seq_lens_host[ns:],
                    cum=self._cum, **args)

    def _parallel(self, r: int, l: int, mx: ParallelMixer, p: Dict[str, torch.Tensor], mid: torch.Tensor, m: StepMeta) -> None:
        left = {n[2:]: v for n, v in p.items() if n.startswith("l_")}
        self._attention(r, l, mx.left, left, mid, m, prefix="l_")
        self._ssd(r, l, mx.right, p["r_z"], p["r_xbc"], p["r_dt"], self._mid_right[mx.right.out_width][:m.num_tokens], m, "r_")

    def _ssd(self, r: int, l: int, mx: SSDMixer, z, xbc, dt, mid: torch.Tensor, m: StepMeta, prefix: str) -> None:
        T, rc = m.num_tokens, self.cache.runs[r]
        w = lambda n: self._w(l, prefix + n)
        u = self._conv[:T * mx.channels].view(T, mx.channels)
        ops.token_conv(xbc, w("conv"), rc.hist, u, m.pos, m.tok_indptr if m.is_prefill else None, m.seq_slot, bias=w("conv_b"), silu=True)
        n = mx.groups * mx.state
        parts = [u[:, :mx.out_width], u[:, mx.out_width:mx.out_width + n], u[:, mx.out_width + n:], z, dt, w("dt_bias"), w("A_log"), w("D")]
        ns = m.batch if not m.is_prefill else m.singles
        if ns:
            ops.ssd(*parts, rc.state, mid, m.pos, None, m.seq_slot[:ns], groups=mx.groups)
        if m.batch > ns:
            ops.ssd(*parts, rc.state, mid, m.pos, m.tok_indptr[ns:], m.seq_slot[ns:], groups=mx.groups, row_lens=m.seq_lens_host[ns:])
        ops.part_norm(mid[:, :mx.out_width], w("o_norm"), mx.norm_groups, self.cfg.rms_eps)

    # ------------------------------------------------------------------ head
    def logits_of(self, n: int, rows: Optional[torch.Tensor] = None, row_offset: int = 0) -> torch.Tensor:
        """fp32 logits of `n` rows of the stream: rows 0 .. n - 1, or `rows` (+ row_offset)."""
        c = self.cfg
        cap = dict(epilogue="softcap", alpha=c.logit_softcap) if c.logit_softcap else {}
        if c.streams:
            h = self._head_in[:n]
            self._streams("final_norm", n=n, out=h, rows=rows, row_offset=row_offset)
            ops.gemm(h, self.seg["lm_head"], out=self._logits_pad[:n], static_b=True, **cap)
            return self.logits[:n]
        add = {} if rows is not None else self._take_pending()
        ops.stream_norm(self.res, self.seg["final_norm"], c.rms_eps, self.normed[:n], w_offset=c.norm_offset, rows=rows,
                        row_offset=row_offset, num_tokens=n, **add)
        ops.gemm(self.normed[:n], self.seg["lm_head"], out=self._logits_pad[:n], static_b=True, **cap)
        return self.logits[:n]

    def head(self, m: StepMeta) -> torch.Tensor:
        B = m.batch
        if m.is_prefill:
            self.logits_of(B, m.tok_indptr[1:], -1)
        else:
            self.logits_of(B)
        ops.argmax(self.logits[:B], out=self.tokens[:B])
        return self.tokens[:B]

    def last_rows(self, m: StepMeta) -> torch.Tensor:
        """[batch, hidden]: the stream (or the sum of the streams) at the last row of every sequence of a prefill pass."""
        if self.cfg.streams:
            last = self.last[:m.batch]
            self._streams(n=m.batch, total=last, rows=m.tok_indptr[1:], row_offset=-1)
            return last
        return torch.index_select(self.res, 0, m.tok_indptr[1:] - 1, out=self.last[:m.batch])

    def head_from_rows(self, rows: torch.Tensor) -> torch.Tensor:
        """First tokens from rows collected with `last_rows` over several passes."""
        B = rows.shape[0]
        if self.cfg.streams:
            self.res[:B].zero_()
            self.res[:B, 0].copy_(rows)
            self._pending, self._fresh = None, False
        else:
            self.res[:B].copy_(rows)
        return self.head(StepMeta(ids=None, pos=None, slot=None, page_indices=None, page_indptr=None, last_page_len=None,
                                  is_prefill=False, batch=B, num_tokens=B))

    def forward(self, m: StepMeta, lo: int = 0, hi: Optional[int] = None, with_embed: bool = True, with_head: bool = True,
                after_layer=None) -> Optional[torch.Tensor]:
        """Layer runs lo .. hi - 1; `after_layer(r)` is called once run r's kernels are in the stream."""
        for r in range(lo, len(self.runs) if hi is None else hi):
            self.run_layer(r, m)
            if after_layer is not None:
                after_layer(r)
        if m.is_prefill or not with_head:
            self.flush(m.num_tokens)             # (in a decode step the final norm adds them)
        return self.head(m) if with_head else None

    def decode_launches(self) -> int:
        """Kernels of this library in one decode step."""
        per = {"attention": 2, "latent": 7, "gla": 1, "rglru": 3, "wkv": 2, "parallel": 6}
        specs = [self.cfg.layer_specs[r.layer] for r in self.runs]
        n = sum(3 + per[s.mixer.kind] + bool(s.ff) + 3 * bool(s.ff_after) + 5 * bool(s.moe) for s in specs)
        return n + 3      # final norm, head product, arg-max
