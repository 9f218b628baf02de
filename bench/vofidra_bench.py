"""The Vofidra design (several residual streams, attention with a bias by distance, latent attention, experts with identity
experts) beside the Komulorn model and the uniform Llama-type model of equal size: prefill and decode throughput of whole
forward passes, and every kernel of the design against its roofline beside the like kernel of the other two.  One GPU, bf16,
random weights.

    python bench.py --vofidra [--hybrid-part models|kernels|all]

The other models have the same width, heads and vocabulary; Komulorn as many experts of the same parameters, of which a token
chooses as many, the uniform model a feed-forward with as many parameters as a token passes through.  Timing as in
hybrid_bench.py."""
from __future__ import annotations

import os
import sys

import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import hybrid_bench as hb  # noqa: E402
from hybrid_bench import LAYERS, VOCAB, _pages, _report  # noqa: E402
from kernels_bench import n_copies, timeit  # noqa: E402
from blitz_scale_b200 import ops  # noqa: E402

# hidden, q heads, kv heads, head size, latent attention, experts, identity experts, chosen, groups, kept, expert ff, dense ff
SIZES = {"h4096": (4096, 32, 8, 128, dict(heads=32, dim=96, rot_dim=32, vdim=128, q_rank=1536, kv_rank=512), 16, 4, 3, 4, 2, 4096, 14336),
         "h2048": (2048, 16, 4, 128, dict(heads=32, dim=64, rot_dim=32, vdim=64, q_rank=768, kv_rank=256), 64, 16, 8, 8, 4, 1408, 8192)}
STREAMS, REL = 4, (32, 512)


def configs(size: str):
    from blitz_scale_b200.models import komulorn, vofidra
    from blitz_scale_b200.models.config import ModelConfig
    H, qh, kvh, d, latent, E, I, top, groups, keep, ff, dense = SIZES[size]
    chosen = max(1, round(top * E / (E + I)))                # with weights, of a token's choices
    inter = (chosen * ff + 127) // 128 * 128
    ff2 = ff * 3 // 2                                        # two matrices per expert there
    return {"vofidra": vofidra.shape_config(f"vofidra_{size}", VOCAB, H, LAYERS, heads=qh, kv_heads=kvh, dim=d, latent=latent, experts=E,
                                            identity=I, top=top, groups=groups, keep=keep, ff=ff, dense_ff=dense, streams=STREAMS, rel=REL),
            "komulorn": komulorn.shape_config(f"komulorn_{size}", VOCAB, H, LAYERS, heads=qh, kv_heads=kvh, dim=d, vdim=d, rot_dims=d // 2,
                                              experts=E, top=chosen, ff=ff2, shared_ff=0, share=1),
            "llama": ModelConfig(f"llama_{size}", VOCAB, H, LAYERS, qh, kvh, d, inter)}


def bench_kernels(out, size):
    from blitz_scale_b200.models.hybrid_config import DistanceBias
    H, qh, kvh, d, la, E, I, top, groups, keep, ff, _ = SIZES[size]
    bf, dev = torch.bfloat16, "cuda"
    rnd = lambda *s: torch.randn(*s, device=dev, dtype=bf)
    rep = lambda name, t, **kw: _report(out, name, t, size=size, **kw)
    bias = rnd(qh, len(DistanceBias(*REL).rows_by_distance()))
    # ---- attention over prompts and in decode
    for lens in ([8192], [2048] * 4, [256] * 32):
        T, B, n = sum(lens), len(lens), lens[0]
        kv, idx, _, _ = _pages(B, n, 64, kvh, d)
        q, o = rnd(T, qh * d), torch.empty(T, qh * d, dtype=bf, device=dev)
        work = ops.prefill_work_list(lens, lens, 64, dev)
        for kw in ({}, dict(bias=bias)):
            t = timeit(lambda i: ops.attn_prefill_paged(q, kv, idx, work, q_heads=qh, kv_heads=kvh, head_dim=d, page_size=64, out=o, **kw))
            rep("attn_prefill, bias by distance" if kw else "attn_prefill (uniform model)", t, fl=4.0 * B * (n * (n + 1) // 2) * qh * d,
                sequences=B, length=n)
        # latent attention: expanded keys and values of all heads (every head has its own)
        h, kd, vd, W, R = la["heads"], la["dim"] + la["rot_dim"], la["vdim"], la["kv_rank"] + la["rot_dim"], la["kv_rank"]
        pool = ops.LatentKV(rnd(T // 64, 64, 1, W), R)
        ku, vu, rows = rnd(W, h * kd) * W ** -0.5, rnd(R, h * vd) * R ** -0.5, torch.empty(T, W, dtype=bf, device=dev)
        k, v = torch.empty(T // 64, 64, h, kd, dtype=bf, device=dev), torch.empty(T // 64, 64, h, vd, dtype=bf, device=dev)
        t = timeit(lambda i: ops.latent_gather(pool, idx, rows))
        rep("latent_gather", t, by=4.0 * T * W, tokens=T)
        t = timeit(lambda i: ops.gemm(rows, ku, out=k.view(T, -1), static_b=True))
        rep("gemm keys of all heads", t, by=2.0 * (T * W + W * h * kd + T * h * kd), fl=2.0 * T * W * h * kd, M=T)
        t = timeit(lambda i: ops.gemm(rows[:, :R], vu, out=v.view(T, -1), static_b=True))
        rep("gemm values of all heads", t, by=2.0 * (T * R + R * h * vd + T * h * vd), fl=2.0 * T * R * h * vd, M=T)
        k.normal_()
        q, gate = rnd(T, h * kd), rnd(T, h)
        index, o = torch.arange(T // 64, device=dev, dtype=torch.int32), torch.empty(T, h * vd, dtype=bf, device=dev)
        t = timeit(lambda i: ops.attn_prefill_paged(q, ops.KVPair(k, v), index, work, q_heads=h, kv_heads=h, head_dim=kd, page_size=64, out=o, gate=gate))
        rep("attn_prefill, latent (expanded)", t, fl=2.0 * B * (n * (n + 1) // 2) * h * (kd + vd), sequences=B, length=n)
        del kv, k, v
    for B, ctx in ((256, 1024), (64, 4096), (16, 1024), (1, 4096)):
        kv, idx, indptr, last = _pages(B, ctx, 64, kvh, d)
        q, o = rnd(B, qh * d), torch.empty(B, qh * d, dtype=bf, device=dev)
        splits = 1
        while splits * 2 <= min((296 + B * kvh - 1) // (B * kvh), ctx // 256, 32) and B * kvh < 296:
            splits *= 2
        ws = torch.empty(max(1, ops.attn_decode_workspace_bytes(B, qh, d, splits)), dtype=torch.uint8, device=dev)
        copies = min(40, n_copies(2 * B * ctx * kvh * d * 2))
        kvs = [kv] + [kv.clone() for _ in range(copies - 1)] if B < 64 else [kv]
        for kw in ({}, dict(bias=bias)):
            t = timeit(lambda i: ops.attn_decode(q, kvs[i], idx, indptr, last, q_heads=qh, kv_heads=kvh, head_dim=d, page_size=64, out=o,
                                                 num_splits=splits, workspace=ws, **kw), copies=len(kvs))
            rep("attn_decode, bias by distance" if kw else "attn_decode (uniform model)", t, by=4.0 * B * ctx * kvh * d, batch=B, ctx=ctx)
        del kv, kvs
        h, W, R = la["heads"], la["kv_rank"] + la["rot_dim"], la["kv_rank"]
        pools = [ops.LatentKV(rnd(idx.numel(), 64, 1, W), R) for _ in range(min(40, n_copies(2 * B * ctx * W)))]
        q, o, gate, ws = rnd(B, h * W), torch.empty(B, h * R, dtype=bf, device=dev), rnd(B, h), ops.attn_latent_workspace(h, R, dev)
        t = timeit(lambda i: ops.attn_latent(q, pools[i], idx, indptr, last, heads=h, scale=W ** -0.5, workspace=ws, out=o, gate=gate, static_table=True),
                   copies=len(pools))
        rep("attn_latent", t, by=2.0 * B * ctx * W + 2.0 * B * h * (W + R), fl=2.0 * B * ctx * h * (W + R), batch=B, ctx=ctx)
        del pools
    # ---- what surrounds the latent: block-diagonal products, beside an ordinary product of the same size
    h, dm, kd, vd, W, R = la["heads"], la["dim"], la["dim"] + la["rot_dim"], la["vdim"], la["kv_rank"] + la["rot_dim"], la["kv_rank"]
    for M in (256, 64, 16, 1):
        nc = min(40, n_copies(2 * h * dm * R))
        uk, q, ql = [rnd(h * dm, R) for _ in range(nc)], rnd(M, h * kd), torch.empty(M, h * W, dtype=bf, device=dev)
        t = timeit(lambda i: ops.gemm(q, uk[i], out=ql, groups=h, a_step=kd, out_step=W, static_b=True), copies=nc)
        rep("gemm into the latent space (block-diagonal)", t, by=2.0 * (h * dm * R + M * h * (dm + R)), fl=2.0 * M * h * dm * R, M=M)
        uv, ol, o = [rnd(h * R, vd) for _ in range(nc)], rnd(M, h * R), torch.empty(M, h * vd, dtype=bf, device=dev)
        t = timeit(lambda i: ops.gemm(ol, uv[i], out=o, groups=h, a_step=R, out_step=vd, static_b=True, bn=64, split_k=1), copies=nc)
        rep("gemm out of the latent space (block-diagonal)", t, by=2.0 * (h * R * vd + M * h * (vd + R)), fl=2.0 * M * h * vd * R, M=M)
        gates = [rnd(4096, 512) for _ in range(40)]
        g_in, g_out = rnd(M, 4096), torch.empty(M, 16 * 512, device=dev)
        t = timeit(lambda i: ops.gemm(g_in, gates[i], out=g_out, groups=16, static_b=True), copies=40)
        rep("gemm block-diagonal (gates of a recurrence, Fafudra)", t, by=M * 4096 * 10.0 + 4096 * 1024.0, fl=2.0 * M * 4096 * 512, M=M)
    # ---- norms and paged writes
    freqs, lf = ops.rope_freqs(d // 2, 5e5, dev), ops.rope_freqs(la["rot_dim"], 5e5, dev)
    qb, kb, vb, qw = rnd(qh * d), rnd(kvh * d), rnd(kvh * d), rnd(d)
    for T in (8192, 256, 16):
        pos = torch.arange(T, device=dev, dtype=torch.int32)
        nc = min(40, n_copies(T * (qh + 2 * kvh) * d * 2))
        xs = [rnd(T, (qh + 2 * kvh) * d) for _ in range(nc)]
        kv = torch.zeros(T // 64 + 1, 2, 64, kvh, d, dtype=bf, device=dev)
        a, b = qh * d, (qh + kvh) * d
        cut = lambda x: (x[:, :a], x[:, a:b], x[:, b:])
        by = T * d * 4.0 * (qh + 2 * kvh)
        t = timeit(lambda i: ops.rope_kv_store(xs[i], pos, pos, kv, q_heads=qh, kv_heads=kvh, head_dim=d, page_size=64, rope_theta=1e5), copies=nc)
        rep("rope_kv_store (uniform model)", t, by=by, tokens=T)
        t = timeit(lambda i: ops.rope_store(*cut(xs[i]), pos, pos, kv, freqs, q_heads=qh, kv_heads=kvh, dim=d, rot_dims=d // 2, page_size=64,
                                            interleaved=False, gain=1.1, q_b=qb, k_b=kb, v_b=vb), copies=nc)
        rep("rope_store (Komulorn)", t, by=by, tokens=T)
        t = timeit(lambda i: ops.norm_store(*cut(xs[i]), pos, pos, kv, qw, qw, q_heads=qh, kv_heads=kvh, dim=d, page_size=64, eps=1e-6,
                                            temp_coef=0.1, temp_every=2048), copies=nc)
        rep("norm_store", t, by=by, tokens=T)
        W, R, qr, h = la["kv_rank"] + la["rot_dim"], la["kv_rank"], la["q_rank"], la["heads"]
        nc = min(40, n_copies(T * (qr + W) * 2))
        xs = [rnd(T, qr + W + (h + 7) // 8 * 8) for _ in range(nc)]
        pool = ops.LatentKV(torch.zeros(T // 64 + 1, 64, 1, W, dtype=bf, device=dev), R)
        w1, w2 = rnd(qr), rnd(R)
        t = timeit(lambda i: ops.latent_store(xs[i][:, :qr], xs[i][:, qr:qr + W], pos, pos, pool, w1, w2, lf, eps=1e-6), copies=nc)
        rep("latent_store", t, by=T * 4.0 * (qr + W), tokens=T)
        kd = la["dim"] + la["rot_dim"]
        nc = min(40, n_copies(T * h * kd * 2))
        xs = [rnd(T, h * kd) for _ in range(nc)]
        t = timeit(lambda i: ops.latent_rotate(xs[i], xs[i][:, la["dim"]:], pos, lf, heads=h, dim=la["dim"], rot=la["rot_dim"], out_step=kd), copies=nc)
        rep("latent_rotate", t, by=T * 4.0 * h * la["rot_dim"], tokens=T)
    # ---- streams beside the norm of one stream
    for T in (8192, 256, 16):
        nc = min(40, n_copies(T * H * 4 * STREAMS))
        w, o = rnd(H), torch.empty(T, H, dtype=bf, device=dev)
        xf = [torch.randn(T, STREAMS, H, device=dev) for _ in range(nc)]
        x1 = [torch.randn(T, H, device=dev) for _ in range(min(40, n_copies(T * H * 4)))]
        per = top
        y, rows, ident = rnd(T * per, H), torch.randperm(T * per, device=dev).to(torch.int32).view(T, per), torch.rand(T, device=dev)
        every = rows.clone()
        rows[torch.rand(T, per, device=dev) < I / (E + I)] = -1
        real = float((rows >= 0).sum()) / T
        mix, v = rnd(STREAMS, STREAMS), rnd(STREAMS)
        norm = (w, torch.full((1,), 0.5, dtype=bf, device=dev), w)
        t = timeit(lambda i: ops.stream_norm(x1[i], w, 1e-6, o), copies=len(x1))
        rep("stream_norm (Komulorn)", t, by=T * H * 6.0, tokens=T)
        t = timeit(lambda i: ops.stream_norm(x1[i], w, 1e-6, o, add=y, add_rows=every), copies=len(x1))
        rep("stream_norm with the experts' rows (Komulorn)", t, by=T * H * (10.0 + 2.0 * per), tokens=T)
        pd = ops.Pending(y[:T], mix, v)
        t = timeit(lambda i: ops.stream_mix(xf[i], pending=pd, read=v, norm=norm, out=o, write=True), copies=nc)
        rep("stream_mix", t, by=T * H * (8.0 * STREAMS + 4.0), tokens=T)
        pd = ops.Pending(y, mix, v, rows, ident, o)
        t = timeit(lambda i: ops.stream_mix(xf[i], pending=pd, read=v, norm=norm, out=o, write=True), copies=nc)
        rep("stream_mix with the experts' rows", t, by=T * H * (8.0 * STREAMS + 4.0 + 2.0 * real), tokens=T)
        del xf, x1
    # ---- experts
    ffp = (ff + 31) // 32 * 32
    up, down = rnd(E, H, 2 * ffp) * H ** -0.5, rnd(E, ffp, H) * ff ** -0.5
    ff2 = ff * 3 // 2
    up2, down2 = rnd(E, H, ff2) * H ** -0.5, rnd(E, ff2, H) * ff2 ** -0.5
    corr = rnd(E + I) * 0.05
    chosen = max(1, round(top * E / (E + I)))
    nc = 4                                       # every copy chooses other experts; the experts together are larger than L2
    cols = (E + I + 7) // 8 * 8
    for T in (8192, 1024, 256, 64, 16, 1):
        h = rnd(T, H)
        zs = [torch.randn(T, cols, device=dev) for _ in range(nc)]
        kw = dict(weight_on_input=False, renormalize=True, softmax=True, correction=corr, groups=groups, keep=keep)
        plans = [ops.moe_route(z, ops.ExpertPlan(T, E, top, False, dev, identity=I), **kw) for z in zs]
        plans2 = [ops.moe_route(z, ops.ExpertPlan(T, E, chosen, False, dev)) for z in zs]
        act, y = torch.empty(T * top, max(ffp, ff2), dtype=bf, device=dev), torch.empty(T * top, H, dtype=bf, device=dev)
        t = timeit(lambda i: ops.moe_route(zs[i], plans[i], **kw), copies=nc)
        rep("moe_route, groups and identity experts", t, by=T * (4.0 * (E + I) + 16.0 * top), tokens=T)
        t = timeit(lambda i: ops.moe_route(zs[i], plans2[i]), copies=nc)
        rep("moe_route (Komulorn)", t, by=T * (4.0 * E + 16.0 * chosen), tokens=T)
        for name, ps, u, dn, a, n, f in (("", plans, up, down, "silu_gate", 2 * ffp, ffp), (" (Komulorn)", plans2, up2, down2, "relu2", ff2, ff2)):
            rows = sum(int(sum(x[2] for x in p._tiles[:int(p.num_tiles)].tolist())) for p in ps) / nc
            used = sum(len({x[0] for x in p._tiles[:int(p.num_tiles)].tolist()}) for p in ps) / nc
            t = timeit(lambda i: ops.gemm_grouped(h, u, ps[i], act, gather=True, act=a, factors=True), copies=nc)
            rep("gemm_grouped up" + (", silu gate" if not name else name), t, by=2.0 * (used * H * n + T * H + rows * f), fl=2.0 * rows * H * n, M=T, experts=used)
            t = timeit(lambda i: ops.gemm_grouped(act, dn, ps[i], y), copies=nc)
            rep("gemm_grouped down" + name, t, by=2.0 * (used * H * f + rows * (H + f)), fl=2.0 * rows * H * f, M=T, experts=used)
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
    return {"metric": "vofidra_vs_komulorn_vs_uniform", "dtype": "bf16", "data": "synthetic token ids, random-init weights", "layers": LAYERS, "rows": out}
