"""The Komulorn design (attention with shared caches, mixture of experts) beside the uniform Llama-type model of equal size:
prefill and decode throughput of whole forward passes, and every kernel of the design against its roofline beside the like
kernel of the uniform model.  One GPU, bf16, random weights.

    python bench.py --komulorn [--hybrid-part models|kernels|all]

The uniform model has the same width, heads and vocabulary, and a feed-forward with as many parameters as a token of the
other one passes through.  Timing as in hybrid_bench.py."""
from __future__ import annotations

import os
import sys

import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import hybrid_bench as hb  # noqa: E402
from hybrid_bench import LAYERS, VOCAB, _pages, _report  # noqa: E402
from kernels_bench import n_copies, timeit  # noqa: E402
from blitz_scale_b200 import ops  # noqa: E402

# hidden, q heads, kv heads, key size, value size, experts, chosen, expert ff, shared ff
SIZES = {"h4096": (4096, 32, 8, 128, 128, 16, 2, 6400, 6400), "h2048": (2048, 16, 4, 128, 64, 64, 6, 1408, 2816)}


def configs(size: str):
    from blitz_scale_b200.models.config import ModelConfig
    from blitz_scale_b200.models.komulorn import shape_config
    H, qh, kvh, d, dv, E, top, ff, sff = SIZES[size]
    inter = (2 * (top * ff + sff) // 3 + 127) // 128 * 128          # two matrices per expert, three per gated feed-forward
    return {"komulorn": shape_config(f"komulorn_{size}", VOCAB, H, LAYERS, heads=qh, kv_heads=kvh, dim=d, vdim=dv, rot_dims=d // 2,
                                     experts=E, top=top, ff=ff, shared_ff=sff),
            "llama": ModelConfig(f"llama_{size}", VOCAB, H, LAYERS, qh, kvh, d, inter)}


def _values(B, ctx, page, kvh, d, dv):
    """Cache like hybrid_bench's, with values of their own size where that differs."""
    kv, idx, indptr, last = _pages(B, ctx, page, kvh, d)
    if dv != d:
        kv = ops.KVPair(kv[:, 0].contiguous(), kv[:, 1, ..., :dv].contiguous())
    return kv, idx, indptr, last


def bench_kernels(out, size):
    H, qh, kvh, d, dv, E, top, ff, sff = SIZES[size]
    bf, dev = torch.bfloat16, "cuda"
    rnd = lambda *s: torch.randn(*s, device=dev, dtype=bf)
    rep = lambda name, t, **kw: _report(out, name, t, size=size, **kw)
    gate = rnd(8192, qh)
    sizes = sorted({(d, d), (d, dv)}, reverse=True)
    # ---- attention over prompts and in decode
    for lens in ([8192], [2048] * 4):
        T, B, n = sum(lens), len(lens), lens[0]
        for kd, vd in sizes:
            kv, idx, _, _ = _values(B, n, 64, kvh, kd, vd)
            q, o = rnd(T, qh * kd), torch.empty(T, qh * vd, dtype=bf, device=dev)
            work = ops.prefill_work_list(lens, lens, 64, dev)
            for kw in ([{}] if kd == vd else []) + [dict(gate=gate[:T])]:
                name = f"attn_prefill {kd} / {vd}" + (", gate" if kw else " (uniform model)")
                t = timeit(lambda i: ops.attn_prefill_paged(q, kv, idx, work, q_heads=qh, kv_heads=kvh, head_dim=kd, page_size=64, out=o, **kw))
                rep(name, t, fl=2.0 * B * (n * (n + 1) // 2) * qh * (kd + vd), sequences=B, length=n)
    for B, ctx in ((256, 1024), (64, 4096)):
        for kd, vd in sizes:
            kv, idx, indptr, last = _values(B, ctx, 64, kvh, kd, vd)
            q, o = rnd(B, qh * kd), torch.empty(B, qh * vd, dtype=bf, device=dev)
            for kw in ([{}] if kd == vd else []) + [dict(gate=gate[:B])]:
                name = f"attn_decode {kd} / {vd}" + (", gate" if kw else " (uniform model)")
                t = timeit(lambda i: ops.attn_decode(q, kv, idx, indptr, last, q_heads=qh, kv_heads=kvh, head_dim=kd, page_size=64, out=o, **kw))
                rep(name, t, by=2.0 * B * ctx * kvh * (kd + vd), batch=B, ctx=ctx)
    # ---- rotation and paged write
    freqs = ops.rope_freqs(d // 2, 5e5, dev)
    qb, kb, vb = rnd(qh * d), rnd(kvh * d), rnd(kvh * dv)
    for T in (8192, 256):
        pos = torch.arange(T, device=dev, dtype=torch.int32)
        kv_u = torch.zeros(T // 64 + 1, 2, 64, kvh, d, dtype=bf, device=dev)
        kv, _, _, _ = _values(T // 64 + 1, 64, 64, kvh, d, dv)
        nc = n_copies(T * (qh + 2 * kvh) * d * 2)
        xs = [rnd(T, (qh + 2 * kvh) * d) for _ in range(nc)]
        ys = [rnd(T, qh * d + kvh * (d + dv) + qh) for _ in range(nc)]
        t = timeit(lambda i: ops.rope_kv_store(xs[i], pos, pos, kv_u, q_heads=qh, kv_heads=kvh, head_dim=d, page_size=64, rope_theta=1e5), copies=nc)
        rep("rope_kv_store (uniform model)", t, by=T * d * 4.0 * (qh + 2 * kvh), tokens=T)
        kw = dict(q_heads=qh, kv_heads=kvh, dim=d, rot_dims=d // 2, page_size=64, interleaved=False, gain=1.1, q_b=qb)
        a, b = qh * d, (qh + kvh) * d
        t = timeit(lambda i: ops.rope_store(ys[i][:, :a], ys[i][:, a:b], ys[i][:, b:b + kvh * dv], pos, pos, kv, freqs, k_b=kb, v_b=vb, **kw), copies=nc)
        rep("rope_store biases, half of a head", t, by=T * 4.0 * (qh * d + kvh * (d + dv)), tokens=T)
        t = timeit(lambda i: ops.rope_store(ys[i][:, :a], None, None, pos, pos, kv, freqs, **kw), copies=nc)
        rep("rope_store queries only", t, by=T * 4.0 * qh * d, tokens=T)
    # ---- norms
    for T in (8192, 256):
        nc = n_copies(T * H * 4)
        w, o = rnd(H), torch.empty(T, H, dtype=bf, device=dev)
        xs = [rnd(T, H) for _ in range(nc)]
        t = timeit(lambda i: ops.rms_norm(xs[i], w, out=o), copies=nc)
        rep("rms_norm (uniform model)", t, by=T * H * 4.0, tokens=T)
        xf = [x.float() for x in xs]
        t = timeit(lambda i: ops.stream_norm(xf[i], w, 1e-6, o), copies=nc)
        rep("stream_norm", t, by=T * H * 6.0, tokens=T)
        y = rnd(T * (top + 1), H)
        rows = torch.randperm(T * (top + 1), device=dev).to(torch.int32).view(T, top + 1)
        t = timeit(lambda i: ops.stream_norm(xf[i], w, 1e-6, o, add=y, add_rows=rows), copies=nc)
        rep("stream_norm with the experts' rows", t, by=T * H * (10.0 + 2.0 * (top + 1)), tokens=T)
    # ---- experts beside the uniform model's feed-forward products
    up, down = rnd(E, H, ff) * H ** -0.5, rnd(E, ff, H) * ff ** -0.5
    shared = [(rnd(H, sff) * H ** -0.5, rnd(sff, H) * sff ** -0.5) for _ in range(n_copies(2 * H * sff))]
    inter = configs(size)["llama"].inter
    for T in (8192, 1024, 256, 64, 16, 1):
        wg, wd = [rnd(H, 2 * inter) * H ** -0.5 for _ in range(n_copies(4 * H * inter))], [rnd(inter, H) * inter ** -0.5 for _ in range(n_copies(2 * H * inter))]
        h, g = rnd(T, H), rnd(T, inter)
        oi, res = torch.empty(T, inter, dtype=bf, device=dev), torch.zeros(T, H, dtype=bf, device=dev)
        t = timeit(lambda i: ops.gemm(h, wg[i], out=oi, epilogue="silu_mul", static_b=True), copies=len(wg))
        rep("gemm gate, up (uniform model)", t, by=2.0 * (2 * H * inter + T * (H + inter)), fl=4.0 * T * H * inter, M=T)
        t = timeit(lambda i: ops.gemm(g, wd[i], out=res, residual=res, epilogue="add", static_b=True), copies=len(wd))
        rep("gemm down (uniform model)", t, by=2.0 * (H * inter + T * (2 * H + inter)), fl=2.0 * T * H * inter, M=T)
        del wg, wd
        plans, nc = [], len(shared)            # every copy chooses other experts: weights are cold also with few tokens
        for i in range(nc):
            z = torch.randn(T, (E + 8) // 8 * 8, device=dev)
            plans.append((z, ops.moe_route(z, ops.ExpertPlan(T, E, top, True, dev))))
        rows = T * (top + 1)
        act, y = torch.empty(rows, max(ff, sff), dtype=bf, device=dev), torch.empty(rows, H, dtype=bf, device=dev)
        used = sum(int((torch.bincount(torch.topk(z[:, :E], top).indices.flatten(), minlength=E) > 0).sum()) for z, _ in plans) / nc
        w_by, fl = 2.0 * H * (used * ff + sff), 2.0 * T * H * (top * ff + sff)
        t = timeit(lambda i: ops.moe_route(plans[i][0], plans[i][1]), copies=nc)
        rep("moe_route", t, by=T * (4.0 * (E + 1) + 16.0 * top + 12.0), tokens=T)
        t = timeit(lambda i: ops.gemm_grouped(h, up, plans[i][1], act, shared=shared[i][0], gather=True, act="relu2", factors=True), copies=nc)
        rep("gemm_grouped up (gathered rows)", t, by=w_by + 2.0 * (T * H + T * (top * ff + sff)), fl=fl, M=T, experts=used)
        t = timeit(lambda i: ops.gemm_grouped(act, down, plans[i][1], y, shared=shared[i][1]), copies=nc)
        rep("gemm_grouped down", t, by=w_by + 2.0 * (rows * H + T * (top * ff + sff)), fl=fl, M=T, experts=used)
        rw = rnd(H, (E + 8) // 8 * 8)
        zs = torch.empty(T, rw.shape[1], device=dev)
        hs = [rnd(T, H) for _ in range(n_copies(T * H * 2))][:40]
        narrow = dict(bn=64, split_k=4 if T <= 2048 else 1) if T > ops.DECODE_GEMM_MAX_M else {}         # as the runner does
        t = timeit(lambda i: ops.gemm(hs[i], rw, out=zs, static_b=True, **narrow), copies=len(hs))
        rep("gemm router", t, by=2.0 * (T * H + H * rw.shape[1]) + 4.0 * T * rw.shape[1], fl=2.0 * T * H * rw.shape[1], M=T)
        # the head with capped logits beside the plain one
        if T <= 256:
            hw = [rnd(H, VOCAB) * H ** -0.5 for _ in range(n_copies(2 * H * VOCAB))]
            lo = torch.empty(T, VOCAB, device=dev)
            for name, kw in (("gemm head", {}), ("gemm head, soft cap", dict(epilogue="softcap", alpha=30.0))):
                t = timeit(lambda i: ops.gemm(h, hw[i], out=lo, static_b=True, **kw), copies=len(hw))
                rep(name, t, by=2.0 * (H * VOCAB + T * H) + 4.0 * T * VOCAB, fl=2.0 * T * H * VOCAB, M=T)
            del hw
    ops.check_status()


def run(part: str = "all") -> dict:
    torch.cuda.set_device(0)
    out = []
    with torch.no_grad():
        for size in SIZES:
            if part in ("kernels", "all"):
                bench_kernels(out, size)
                torch.cuda.empty_cache()
            if part in ("models", "all"):
                hb.bench_models(out, (size,), configs)
    return {"metric": "komulorn_vs_uniform", "dtype": "bf16", "data": "synthetic token ids, random-init weights", "layers": LAYERS, "rows": out}
