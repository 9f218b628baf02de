"""Hybrid models (per-layer mixers over an fp32 stream) beside the uniform Llama-type model of equal size: prefill and
decode throughput of whole forward passes, and every kernel of the design against its roofline beside the like kernel
of the uniform model.  One GPU, bf16, random weights.

    python bench.py --hybrid [--hybrid-part models|kernels|all]

Timing: CUDA events around captured CUDA graphs (kernels, decode steps) or around the launches themselves (prefill
passes, milliseconds long), at least three warm-up runs, median.  Working sets exceed the 126 MB L2: a pass walks
several layers' weights, kernels rotate over copies of their operands."""
from __future__ import annotations

import dataclasses
import json
import os
import sys

import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
from kernels_bench import n_copies, peaks, timeit  # noqa: E402
from blitz_scale_b200 import ops  # noqa: E402

# hidden, ff, q heads, kv heads, head dim, GLA heads x (dim, vdim), recurrence width / blocks
SIZES = {"h4096": (4096, 14336, 32, 8, 128, 16, 128, 256, 4096, 16), "h2048": (2048, 8192, 16, 4, 128, 8, 128, 256, 2048, 8)}
LAYERS, VOCAB, WINDOW = 8, 32000, 2048


def configs(size: str):
    from blitz_scale_b200.models.config import ModelConfig
    from blitz_scale_b200.models.fafudra import shape_config
    H, ff, qh, kvh, hd, gh, gd, gv, w, nb = SIZES[size]
    hybrid = shape_config(f"fafudra_{size}", VOCAB, H, ("gla", "attention", "rglru", "gla") * (LAYERS // 4), ff, heads=qh, kv_heads=kvh,
                          dim=hd, window=WINDOW, gla_heads=gh, gla_dim=gd, gla_vdim=gv, width=w, blocks=nb)
    return {"fafudra": hybrid, "llama": ModelConfig(f"llama_{size}", VOCAB, H, LAYERS, qh, kvh, hd, ff)}


def _median(fn, n=7, warmup=3):
    for _ in range(warmup):
        fn()
    torch.cuda.synchronize()
    times = []
    for _ in range(n):
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        fn()
        b.record()
        torch.cuda.synchronize()
        times.append(a.elapsed_time(b))
    return sorted(times)[n // 2] * 1e-3


def bench_models(out, sizes=("h4096", "h2048"), configs=configs):
    from blitz_scale_b200.runtime import core
    from blitz_scale_b200.runtime.engine import Engine, _bucket
    for size in sizes:
        for name, cfg in configs(size).items():
            eng = Engine(cfg, num_pages=4224, page_size=64, max_batch=256, max_batch_tokens=8192, seed=0, state_slots=256)
            g = torch.Generator().manual_seed(1)
            for lens in ([8192], [2048] * 4, [256] * 32):
                b = eng.new_batch(0, [core.SeqSpec(i, torch.randint(0, VOCAB, (n,), generator=g).tolist(), 4) for i, n in enumerate(lens)])
                T, P = b.fill_prefill(eng.host_np, eng.layout)
                eng._h2d(eng.layout.page_indices + P)
                m = eng._views(T, b.size, P, True, b.prompt_lens())
                t = _median(lambda: eng.runner.forward(m))
                ops.check_status()
                b.clear()
                row = dict(kind="prefill", size=size, model=name, sequences=len(lens), length=lens[0], ms=t * 1e3, tokens_per_s=T / t)
                out.append(row)
                print(json.dumps(row), flush=True)
            for B, ctx in ((256, 1000), (64, 4000), (16, 1000), (1, 4000)):
                b = eng.new_batch(1, [core.SeqSpec(i, [1] * ctx, 4) for i in range(B)])
                assert b is not None
                b.mark_prefilled()                      # contents do not matter for the time
                b.append_tokens(torch.randint(0, VOCAB, (B,), generator=g).tolist(), False)   # (they choose experts)
                P = b.fill_decode(eng.host_np, eng.layout, _bucket(B))
                eng._h2d(eng.layout.page_indices + P)
                graph = eng._capture(_bucket(B), eng.choose_splits(_bucket(B), b.max_seq_len()))
                t = _median(graph.replay, n=15)
                ops.check_status()
                b.clear()
                eng._graphs.clear()
                weights = eng.seg.layout.total_bytes - 2 * VOCAB * cfg.hidden       # (of the embedding table only rows)
                if cfg.family == "hybrid":
                    for e in (s.moe for s in cfg.layer_specs if s.moe):
                        # experts that no token of the step chooses are not read (expected number, choices being random)
                        weights -= e.experts * (1 - e.top / e.outputs) ** B * 2 * cfg.hidden * (e.up_cols + e.ff_pad)
                    for x in (s.mixer for s in cfg.layer_specs if s.mixer.kind == "latent"):
                        weights -= 2 * x.heads * (x.width * x.qdim + x.kv_rank * x.vdim)      # of prompts only
                    # window and kept tokens of the attention layers; states are read and written
                    seen = lambda x: ctx if not x.window else ctx % x.window + 1 if x.chunked else min(ctx, x.window + x.keep_first)
                    kv = sum(x.kv_heads * (x.dim + x.vdim) * 2 * seen(x) for x in cfg.run_parts() if x.kind == "attention")
                    kv += sum(x.width * 2 * min(ctx, x.window or ctx) for x in cfg.run_mixers() if x.kind == "latent")
                    data = B * (kv + 2 * cfg.state_bytes_per_sequence())
                else:
                    data = B * ctx * cfg.kv_bytes_per_token()
                row = dict(kind="decode", size=size, model=name, batch=B, ctx=ctx, ms=t * 1e3, tokens_per_s=B / t,
                           gb_per_step=(weights + data) / 1e9, hbm_frac=(weights + data) / t / peaks()[0])
                out.append(row)
                print(json.dumps(row), flush=True)
            del eng, graph
            torch.cuda.empty_cache()


def _report(out, name, t, by=0.0, fl=0.0, **extra):
    hbm, flops, src = peaks()
    roof = max(by / hbm, fl / flops)
    row = dict(kind="kernel", name=name, us=t * 1e6, roofline_us=roof * 1e6, frac=roof / t, bound="hbm" if by / hbm > fl / flops else "tensor",
               gbs=by / t / 1e9, tflops=fl / t / 1e12, peaks=src, **extra)
    out.append(row)
    print(json.dumps(row), flush=True)


def _pages(B, ctx, page, kvh, hd):
    npg = -(-ctx // page)
    kv = torch.randn(B * npg, 2, page, kvh, hd, device="cuda", dtype=torch.bfloat16)
    idx = torch.randperm(B * npg, device="cuda").to(torch.int32)
    indptr = (torch.arange(B + 1, device="cuda") * npg).to(torch.int32)
    last = torch.full((B,), ctx - (npg - 1) * page, device="cuda", dtype=torch.int32)
    return kv, idx, indptr, last


def bench_kernels(out, size="h4096"):
    H, ff, qh, kvh, hd, gh, gd, gv, W, nb = SIZES[size]
    bf, dev = torch.bfloat16, "cuda"
    rnd = lambda *s: torch.randn(*s, device=dev, dtype=bf)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
    hk, hv, rank = gh * gd, gh * gv, 16
    sink = rnd(qh)
    window = dict(window=WINDOW, keep_first=4, softcap=50.0, sink=sink)
    # ---- attention over prompts: useful products are those of visible pairs
    for lens in ([8192], [2048] * 4):
        T, B = sum(lens), len(lens)
        kv, idx, indptr, _ = _pages(B, lens[0], 64, kvh, hd)
        q, o = rnd(T, qh * hd), torch.empty(T, qh * hd, dtype=bf, device=dev)
        work = ops.prefill_work_list(lens, lens, 64, dev)
        n = lens[0]
        for name, kw, vis in (("attn_prefill full (uniform model)", {}, n * (n + 1) // 2),
                              ("attn_prefill window, cap, sink", window, sum(min(i + 1, WINDOW + 4) for i in range(n)))):
            t = timeit(lambda i: ops.attn_prefill_paged(q, kv, idx, work, q_heads=qh, kv_heads=kvh, head_dim=hd, page_size=64, out=o, **kw))
            _report(out, name, t, fl=4.0 * B * vis * qh * hd, sequences=B, length=n)
    # ---- attention in decode
    for B, ctx in ((256, 1024), (64, 4096)):
        kv, idx, indptr, last = _pages(B, ctx, 64, kvh, hd)
        q, o = rnd(B, qh * hd), torch.empty(B, qh * hd, dtype=bf, device=dev)
        for name, kw, seen in (("attn_decode full (uniform model)", {}, ctx), ("attn_decode window, cap, sink", window, min(ctx, WINDOW + 4))):
            t = timeit(lambda i: ops.attn_decode(q, kv, idx, indptr, last, q_heads=qh, kv_heads=kvh, head_dim=hd, page_size=64, out=o, **kw))
            _report(out, name, t, by=B * seen * kvh * hd * 4.0, batch=B, ctx=ctx)
    # ---- rotation and paged write
    freqs = ops.rope_freqs(hd, 1e5, dev)
    for T in (8192, 256):
        kv = torch.zeros(T // 64 + 1, 2, 64, kvh, hd, dtype=bf, device=dev)
        pos = torch.arange(T, device=dev, dtype=torch.int32)
        nc = n_copies(T * (qh + 2 * kvh) * hd * 2)
        xs = [rnd(T, (qh + 2 * kvh) * hd) for _ in range(nc)]
        ys = [rnd(T, (qh + kvh) * hd) for _ in range(nc)]
        by = T * hd * 2.0 * (2 * qh + 2 * kvh)
        t = timeit(lambda i: ops.rope_kv_store(xs[i], pos, pos, kv, q_heads=qh, kv_heads=kvh, head_dim=hd, page_size=64, rope_theta=1e5), copies=nc)
        _report(out, "rope_kv_store (uniform model)", t, by=by + T * hd * kvh * 4.0, tokens=T)
        t = timeit(lambda i: ops.rope_store(ys[i][:, :qh * hd], ys[i][:, qh * hd:], None, pos, pos, kv, freqs, q_heads=qh, kv_heads=kvh,
                                            dim=hd, rot_dims=hd, page_size=64, interleaved=True), copies=nc)
        _report(out, "rope_store interleaved, values = keys", t, by=by + T * hd * kvh * 2.0, tokens=T)
    # ---- norms
    for T in (8192, 256):
        nc = n_copies(T * H * 4)
        w, o = rnd(H), torch.empty(T, H, dtype=bf, device=dev)
        xs = [rnd(T, H) for _ in range(nc)]
        t = timeit(lambda i: ops.rms_norm(xs[i], w, out=o), copies=nc)
        _report(out, "rms_norm (uniform model)", t, by=T * H * 4.0, tokens=T)
        xf = [x.float() for x in xs]
        t = timeit(lambda i: ops.stream_norm(xf[i], w, 1e-6, o, w_offset=1.0), copies=nc)
        _report(out, "stream_norm (fp32 stream)", t, by=T * H * 6.0, tokens=T)
    # ---- products: the uniform model's down projection (16-bit residual) against the out projection (fp32 axpy)
    for M in (8192, 256, 64, 1):
        for name, K, N, epi in (("gemm add 16-bit (uniform model)", ff, H, "add"), ("gemm fp32 axpy", ff + hv, H, "axpy"),
                                ("gemm store (uniform model, qkv)", H, (qh + 2 * kvh) * hd, "store"),
                                ("gemm store (gla projections)", H, 2 * hk + 2 * hv + rank, "store")):
            nc = n_copies(K * N * 2)
            a, bs = rnd(M, K), [rnd(K, N) * K ** -0.5 for _ in range(nc)]
            o = torch.zeros(M, N, device=dev, dtype=torch.float32 if epi == "axpy" else bf)
            kw = dict(residual=o) if epi == "add" else dict(alpha=0.5) if epi == "axpy" else {}
            t = timeit(lambda i: ops.gemm(a, bs[i], out=o, epilogue=epi, static_b=True, **kw), copies=nc)
            _report(out, name, t, by=2.0 * (M * K + K * N) + M * N * {"add": 4, "axpy": 8, "store": 2}[epi], fl=2.0 * M * N * K, M=M, N=N, K=K)
        nc = n_copies(W * 2 * (W // nb) * 2 + M * W * 10)
        us = [rnd(M, W) for _ in range(nc)]
        gw, gates = rnd(W, 2 * W // nb), torch.empty(M, 2 * W, device=dev)
        t = timeit(lambda i: ops.gemm(us[i], gw, out=gates, groups=nb, static_b=True), copies=nc)
        _report(out, "gemm block-diagonal (gates)", t, by=M * W * 10.0 + W * 4.0 * W / nb, fl=4.0 * M * W * W / nb, M=M)
    # ---- gated linear attention
    a2, a2_b, on = rnd(rank, hk) * rank ** -0.5, 2 + rnd(hk), rnd(gv)
    width = 2 * hk + 2 * hv + rank
    cut = lambda x: (x[:, :hk], x[:, hk:2 * hk], x[:, 2 * hk:2 * hk + hv], x[:, 2 * hk + hv:2 * hk + 2 * hv], x[:, 2 * hk + 2 * hv:])
    for lens in ([8192], [2048] * 4, [256] * 32):
        T, B = sum(lens), len(lens)
        x, o = rnd(T, width), torch.empty(T, hv, dtype=bf, device=dev)
        state, cum = torch.zeros(B, gh, gd, gv, device=dev), torch.empty(T * hk, device=dev)
        pos = i32([p for n in lens for p in range(n)])
        indptr, slots = i32([sum(lens[:i]) for i in range(B + 1)]), torch.arange(B, dtype=torch.int32, device=dev)
        t = timeit(lambda i: ops.gla(*cut(x), a2, a2_b, on, state, o, pos, indptr, slots, rank=rank, tau=16.0, eps=1e-6, row_lens=lens, cum=cum))
        # useful work: state term and update, causal half of a chunk's scores and of their product with v
        _report(out, "gla prompts (decay + chunks)", t, by=T * (2.0 * width + 2.0 * hv) + B * gh * gd * gv * 8.0,
                fl=T * gh * (4.0 * gd * gv + 64.0 * (gd + gv)), sequences=B, length=lens[0])
    for B in (256, 16, 1):
        x, o = rnd(B, width), torch.empty(B, hv, dtype=bf, device=dev)
        nc = 1 if B * gh * gd * gv * 4 > (300 << 20) else n_copies(B * gh * gd * gv * 4)
        states = [torch.zeros(B, gh, gd, gv, device=dev) for _ in range(min(nc, 40))]
        pos, slots = torch.full((B,), 5, dtype=torch.int32, device=dev), torch.arange(B, dtype=torch.int32, device=dev)
        t = timeit(lambda i: ops.gla(*cut(x), a2, a2_b, on, states[i], o, pos, None, slots, rank=rank, tau=16.0, eps=1e-6), copies=len(states))
        _report(out, "gla decode", t, by=B * (gh * gd * gv * 8.0 + 2.0 * width), batch=B)
    # ---- gated linear recurrence
    xb, conv, lam, gb = rnd(W), rnd(4, W), rnd(W), rnd(2 * W)
    for lens in ([8192], [2048] * 4, [1] * 256, [1]):
        T, B = sum(lens), len(lens)
        nc = min(40, n_copies(T * W * 14))
        ps = [rnd(T, 2 * W) for _ in range(nc)]
        us = [rnd(T, W) for _ in range(nc)]
        gs = [torch.randn(T, 2 * W, device=dev) for _ in range(nc)]
        o, state, hist = torch.empty(T, W, dtype=bf, device=dev), torch.zeros(B, W, device=dev), torch.zeros(B, 3, W, dtype=bf, device=dev)
        pos = i32([p for n in lens for p in range(n)]) if lens[0] > 1 else torch.full((B,), 5, dtype=torch.int32, device=dev)
        indptr = i32([sum(lens[:i]) for i in range(B + 1)]) if lens[0] > 1 else None
        slots = torch.arange(B, dtype=torch.int32, device=dev)
        t = timeit(lambda i: ops.conv_causal(ps[i][:, W:], xb, conv, xb, hist, us[i], pos, indptr, slots), copies=nc)
        _report(out, "conv_causal", t, by=T * W * 4.0, sequences=B, length=lens[0])
        t = timeit(lambda i: ops.rglru_scan(us[i], gs[i], gb, lam, ps[i][:, :W], ps[i][:, W:], xb, state, hist, o, pos, indptr, slots, block=W // nb),
                   copies=nc)
        _report(out, "rglru_scan", t, by=T * W * 14.0 + B * W * 8.0, sequences=B, length=lens[0])
    ops.check_status()


def run(part: str = "all") -> dict:
    torch.cuda.set_device(0)
    out = []
    with torch.no_grad():
        if part in ("kernels", "all"):
            bench_kernels(out)
        if part in ("models", "all"):
            bench_models(out)
    return {"metric": "hybrid_vs_uniform", "dtype": "bf16", "data": "synthetic token ids, random-init weights", "layers": LAYERS, "rows": out}
