"""The Norusun design (streams with RMS norms and convolved mixer inputs, linear attention with a token shift, latent attention in a
window, sigmoid attention in chunks beside a state space) beside the Fafudra and the uniform Llama-type model of equal size:
prefill and decode throughput of whole forward passes, and every kernel of the design against its roofline beside the like kernel
of the framework's other models.  One GPU, bf16, random weights.

    python bench.py --norusun [--hybrid-part models|kernels|all]

The models have the same width, heads, feed-forward width and vocabulary; the layers with the linear attention have no
feed-forward here (a quarter of the layers).  Timing as in hybrid_bench.py."""
from __future__ import annotations

import os
import sys

import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import hybrid_bench as hb  # noqa: E402
from hybrid_bench import LAYERS, VOCAB, WINDOW, _pages, _report  # noqa: E402
from kernels_bench import n_copies, timeit  # noqa: E402
from blitz_scale_b200 import ops  # noqa: E402

# hidden, ff, q heads, kv heads, head size, linear attention (heads, size, rank), latent attention, state space
SIZES = {"h4096": (4096, 14336, 32, 8, 128, (32, 128, 64), dict(heads=32, dim=96, rot_dim=32, vdim=128, q_rank=1024, kv_rank=512, window=WINDOW),
                   dict(heads=64, vdim=64, state=128, groups=8, taps=4, norm_groups=8)),
         "h2048": (2048, 8192, 16, 4, 128, (16, 128, 64), dict(heads=32, dim=64, rot_dim=32, vdim=64, q_rank=768, kv_rank=256, window=WINDOW),
                   dict(heads=32, vdim=64, state=128, groups=4, taps=4, norm_groups=4))}
STREAMS, TAPS = 2, 4


def configs(size: str):
    from blitz_scale_b200.models.norusun import shape_config
    H, ff, qh, kvh, d, wkv, latent, ssd = SIZES[size]
    new = shape_config(f"norusun_{size}", VOCAB, H, ("wkv", "latent_attention", "parallel", "latent_attention") * (LAYERS // 4), ff, wkv=wkv,
                       latent=latent, heads=qh, kv_heads=kvh, dim=d, chunk=WINDOW, ssd=ssd, streams=STREAMS, taps=TAPS)
    return {"norusun": new, **hb.configs(size)}


def bench_kernels(out, size):
    H, ff, qh, kvh, d, (wh, wd, rank), la, sp = SIZES[size]
    bf, dev = torch.bfloat16, "cuda"
    rnd = lambda *s: torch.randn(*s, device=dev, dtype=bf)
    rep = lambda name, t, **kw: _report(out, name, t, size=size, **kw)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
    sink, pb = rnd(max(qh, la["heads"])), rnd(qh, 1)
    chunk = dict(window=WINDOW, chunked=True, sigmoid=True, bias=pb)
    window = dict(window=WINDOW, sink=sink[:qh])
    h, kd, vd, W, R = la["heads"], la["dim"] + la["rot_dim"], la["vdim"], la["kv_rank"] + la["rot_dim"], la["kv_rank"]
    in_window = lambda n: sum(min(i + 1, WINDOW) for i in range(n))
    in_chunk = lambda n: sum(i % WINDOW + 1 for i in range(n))
    # ---- attention over prompts and in decode
    for lens in ([8192], [2048] * 4, [256] * 32):
        T, B, n = sum(lens), len(lens), lens[0]
        kv, idx, _, _ = _pages(B, n, 64, kvh, d)
        q, o = rnd(T, qh * d), torch.empty(T, qh * d, dtype=bf, device=dev)
        work = ops.prefill_work_list(lens, lens, 64, dev)
        for name, kw, vis in (("attn_prefill (uniform model)", {}, n * (n + 1) // 2), ("attn_prefill, window and sink", window, in_window(n)),
                              ("attn_prefill, sigmoid weights in chunks", chunk, in_chunk(n))):
            t = timeit(lambda i: ops.attn_prefill_paged(q, kv, idx, work, q_heads=qh, kv_heads=kvh, head_dim=d, page_size=64, out=o, **kw))
            rep(name, t, fl=4.0 * B * vis * qh * d, sequences=B, length=n)
        k, v = rnd(T // 64, 64, h, kd), rnd(T // 64, 64, h, vd)
        q, index, o = rnd(T, h * kd), torch.arange(T // 64, device=dev, dtype=torch.int32), torch.empty(T, h * vd, dtype=bf, device=dev)
        for name, kw, vis in (("attn_prefill, latent (expanded, Vofidra)", {}, n * (n + 1) // 2),
                              ("attn_prefill, latent (expanded), window and sink", dict(window=WINDOW, sink=sink[:h]), in_window(n))):
            t = timeit(lambda i: ops.attn_prefill_paged(q, ops.KVPair(k, v), index, work, q_heads=h, kv_heads=h, head_dim=kd, page_size=64, out=o, **kw))
            rep(name, t, fl=2.0 * B * vis * h * (kd + vd), sequences=B, length=n)
        del kv, k, v
    for B, ctx in ((256, 1024), (64, 4096), (16, 1024), (1, 4096)):
        kv, idx, indptr, last = _pages(B, ctx, 64, kvh, d)
        q, o = rnd(B, qh * d), torch.empty(B, qh * d, dtype=bf, device=dev)
        for name, kw, seen in (("attn_decode (uniform model)", {}, ctx), ("attn_decode, sigmoid weights in chunks", chunk, (ctx - 1) % WINDOW + 1)):
            splits = 1
            while splits * 2 <= min((296 + B * kvh - 1) // (B * kvh), seen // 256, 32) and B * kvh < 296:
                splits *= 2
            ws = torch.empty(max(1, ops.attn_decode_workspace_bytes(B, qh, d, splits)), dtype=torch.uint8, device=dev)
            kvs = [kv] + [kv.clone() for _ in range(min(40, n_copies(2 * B * seen * kvh * d * 2)) - 1)] if B < 64 else [kv]
            t = timeit(lambda i: ops.attn_decode(q, kvs[i], idx, indptr, last, q_heads=qh, kv_heads=kvh, head_dim=d, page_size=64, out=o,
                                                 num_splits=splits, workspace=ws, **kw), copies=len(kvs))
            rep(name, t, by=4.0 * B * seen * kvh * d, batch=B, ctx=ctx)
        del kv, kvs
        pools = [ops.LatentKV(rnd(idx.numel(), 64, 1, W), R) for _ in range(min(40, n_copies(2 * B * min(ctx, WINDOW) * W)))]
        q, o, ws = rnd(B, h * W), torch.empty(B, h * R, dtype=bf, device=dev), ops.attn_latent_workspace(h, R, dev)
        for name, kw, seen in (("attn_latent (Vofidra)", {}, ctx), ("attn_latent, window and sink", dict(window=WINDOW, sink=sink[:h]), min(ctx, WINDOW))):
            t = timeit(lambda i: ops.attn_latent(q, pools[i], idx, indptr, last, heads=h, scale=W ** -0.5, workspace=ws, out=o, static_table=True, **kw),
                       copies=len(pools))
            rep(name, t, by=2.0 * B * seen * W + 2.0 * B * h * (W + R), fl=2.0 * B * seen * h * (W + R), batch=B, ctx=ctx)
        del pools
    # ---- norms and paged writes
    freqs, lf = ops.rope_freqs(d, 5e5, dev), ops.rope_freqs(la["rot_dim"], 5e5, dev)
    qw, kw_ = rnd(qh * d), rnd(kvh * d)
    for T in (8192, 256, 16):
        pos = torch.arange(T, device=dev, dtype=torch.int32)
        xs = [rnd(T, (qh + 2 * kvh) * d) for _ in range(min(40, n_copies(T * (qh + 2 * kvh) * d * 2)))]
        kv = torch.zeros(T // 64 + 1, 2, 64, kvh, d, dtype=bf, device=dev)
        a, b = qh * d, (qh + kvh) * d
        cut = lambda x: (x[:, :a], x[:, a:b], x[:, b:])
        by = T * d * 4.0 * (qh + 2 * kvh)
        t = timeit(lambda i: ops.rope_kv_store(xs[i], pos, pos, kv, q_heads=qh, kv_heads=kvh, head_dim=d, page_size=64, rope_theta=1e5), copies=len(xs))
        rep("rope_kv_store (uniform model)", t, by=by, tokens=T)
        t = timeit(lambda i: ops.rope_store(*cut(xs[i]), pos, pos, kv, freqs, q_heads=qh, kv_heads=kvh, dim=d, rot_dims=d, page_size=64,
                                            interleaved=False, q_w=qw, k_w=kw_, eps=1e-5), copies=len(xs))
        rep("rope_store with a norm over all heads", t, by=by, tokens=T)
        qr = la["q_rank"]
        xs = [rnd(T, qr + W) for _ in range(min(40, n_copies(T * (qr + W) * 2)))]
        pool = ops.LatentKV(torch.zeros(T // 64 + 1, 64, 1, W, dtype=bf, device=dev), R)
        w1, w2 = rnd(qr), rnd(R)
        ys = [rnd(T, h * kd) for _ in range(min(40, n_copies(T * h * kd * 2)))]
        for name, inter in ((" (Vofidra)", False), (", neighbouring pairs", True)):
            t = timeit(lambda i: ops.latent_store(xs[i][:, :qr], xs[i][:, qr:], pos, pos, pool, w1, w2, lf, eps=1e-6, interleaved=inter), copies=len(xs))
            rep("latent_store" + name, t, by=T * 4.0 * (qr + W), tokens=T)
            t = timeit(lambda i: ops.latent_rotate(ys[i], ys[i][:, la["dim"]:], pos, lf, heads=h, dim=la["dim"], rot=la["rot_dim"], out_step=kd,
                                                   interleaved=inter), copies=len(ys))
            rep("latent_rotate" + name, t, by=T * 4.0 * h * la["rot_dim"], tokens=T)
    # ---- streams, convolved inputs
    conv, mu, one = rnd(TAPS, H), torch.rand(5, H, device=dev).to(bf), torch.ones(1, dtype=bf, device=dev)
    mix, v, w = rnd(STREAMS, STREAMS), rnd(STREAMS), rnd(H)
    for T in (8192, 256, 16, 1):
        xf = [torch.randn(T, STREAMS, H, device=dev) for _ in range(min(40, n_copies(T * H * 4 * STREAMS)))]
        o, y, o5 = torch.empty(T, H, dtype=bf, device=dev), rnd(T, 2 * H), torch.empty(T, 5 * H, dtype=bf, device=dev)
        norm = (w, torch.full((1,), 0.5, dtype=bf, device=dev), w)
        pd = ops.Pending(y[:, :H].clone(memory_format=torch.contiguous_format), mix, v)
        by = T * H * (8.0 * STREAMS + 4.0)
        x1 = [torch.randn(T, H, device=dev) for _ in range(min(40, n_copies(T * H * 4)))]
        t = timeit(lambda i: ops.stream_norm(x1[i], w, 1e-6, o), copies=len(x1))
        rep("stream_norm (Fafudra)", t, by=T * H * 6.0, tokens=T)
        del x1
        t = timeit(lambda i: ops.stream_mix(xf[i], pending=pd, read=v, norm=norm, out=o, write=True), copies=len(xf))
        rep("stream_mix (Vofidra)", t, by=by, tokens=T)
        args = dict(eps=1e-5, read=v, w=one, write=True)
        t = timeit(lambda i: ops.stream_rms(xf[i], pending=pd._replace(bias=w), out=o, **args), copies=len(xf))
        rep("stream_rms", t, by=by, tokens=T)
        two = ops.Pending(y, mix, v, norms=(w, w))
        t = timeit(lambda i: ops.stream_rms(xf[i], pending=two, out=o, **args), copies=len(xf))
        o32 = torch.empty(T, H, device=dev)
        t2 = timeit(lambda i: ops.stream_rms(xf[i], pending=pd, out=o32, **args), copies=len(xf))
        rep("stream_rms, fp32 output", t2, by=by + 2.0 * T * H, tokens=T)
        rep("stream_rms, two normed outputs", t, by=by + 2.0 * T * H, tokens=T)
        pos, slots = torch.full((T,), 9, dtype=torch.int32, device=dev), torch.arange(T, dtype=torch.int32, device=dev)
        hist, shift = torch.zeros(T, TAPS - 1, H, device=dev), torch.zeros(T, H, device=dev)
        if T <= 256:
            st = ops.TokenState(conv, hist)
            t = timeit(lambda i: ops.stream_rms(xf[i], pending=pd, out=o, tokens=st, pos=pos, seq_slot=slots, **args), copies=len(xf))
            rep("stream_rms with the convolution (decode)", t, by=by + 8.0 * T * H * (TAPS - 1), tokens=T)
            st = ops.TokenState(conv, hist, mu, shift)
            t = timeit(lambda i: ops.stream_rms(xf[i], pending=pd, out=o5, tokens=st, pos=pos, seq_slot=slots, **args), copies=len(xf))
            rep("stream_rms with convolution and mixes (decode)", t, by=by + 8.0 * T * H * (TAPS - 1) + 16.0 * T * H, tokens=T)
        del xf
    C = sp["heads"] * sp["vdim"] + 2 * sp["groups"] * sp["state"]
    cb, zero, sc = rnd(C), torch.zeros(max(C, H), dtype=bf, device=dev), rnd(TAPS, C)
    for lens in ([8192], [2048] * 4, [256] * 32, [1] * 256):
        T, B = sum(lens), len(lens)
        pos = i32([p for n in lens for p in range(n)]) if lens[0] > 1 else torch.full((B,), 9, dtype=torch.int32, device=dev)
        indptr, slots = i32([sum(lens[:i]) for i in range(B + 1)]) if lens[0] > 1 else None, torch.arange(B, dtype=torch.int32, device=dev)
        nc = min(40, n_copies(T * max(C, H) * 4))
        xs, us = [rnd(T, max(C, H)) for _ in range(nc)], [torch.empty(T, max(C, H), dtype=bf, device=dev) for _ in range(nc)]
        hist = torch.zeros(B, TAPS - 1, max(C, H), dtype=bf, device=dev)
        cut = lambda x, n: x.view(-1)[:T * n].view(T, n)
        hc, hh = (hist.view(-1)[:B * (TAPS - 1) * C].view(B, TAPS - 1, C), hist.view(-1)[:B * (TAPS - 1) * H].view(B, TAPS - 1, H))
        t = timeit(lambda i: ops.conv_causal(cut(xs[i], H), zero[:H], conv, zero[:H], hh, cut(us[i], H), pos, indptr, slots), copies=nc)
        rep("conv_causal (Fafudra)", t, by=T * H * 4.0, sequences=B, length=lens[0])
        t = timeit(lambda i: ops.token_conv(cut(xs[i], C), sc, hc, cut(us[i], C), pos, indptr, slots, bias=cb, silu=True), copies=nc)
        rep("token_conv, silu", t, by=T * C * 4.0, sequences=B, length=lens[0])
        if lens[0] == 1:
            continue
        x32, h32 = [torch.randn(T, H, device=dev) for _ in range(2)], torch.zeros(B, TAPS - 1, H, device=dev)
        t = timeit(lambda i: ops.token_conv(x32[i], conv, h32, cut(us[i], H), pos, indptr, slots, residual=True), copies=2)
        rep("token_conv, fp32 input and its convolution", t, by=T * H * 6.0, sequences=B, length=lens[0])
        o5, shift, lasth = [torch.empty(T, 5 * H, dtype=bf, device=dev) for _ in range(2)], torch.zeros(B, H, device=dev), torch.empty(B, H, device=dev)
        t = timeit(lambda i: ops.token_conv(x32[i % 2], conv, h32, o5[i % 2], pos, indptr, slots, residual=True, mu=mu, shift=shift, last=lasth), copies=2)
        rep("token_conv with mixes", t, by=T * H * 14.0, sequences=B, length=lens[0])
    # ---- products
    n = wh * wd
    for M in (8192, 256, 64, 1):
        nc = min(40, n_copies(H * 2 * ff * 2))
        a, bs, gb = rnd(M, H), [rnd(H, 2 * ff) * H ** -0.5 for _ in range(nc)], rnd(2 * ff)
        o = torch.empty(M, ff, dtype=bf, device=dev)
        for name, kw in (("gemm silu(gate) * up (uniform model)", dict(epilogue="silu_mul")),
                         ("gemm clamped unit with biases", dict(epilogue="clamp_glu", alpha=7.0, beta=1.702, bias=gb))):
            t = timeit(lambda i: ops.gemm(a, bs[i], out=o, static_b=True, **kw), copies=nc)
            rep(name, t, by=2.0 * (M * H + 2 * H * ff + M * ff), fl=4.0 * M * H * ff, M=M)
        del bs
        nc = min(40, n_copies(4 * H * n * 2))
        ws, a5, o4 = [rnd(4 * H, n) * H ** -0.5 for _ in range(nc)], rnd(M, 5 * H), torch.empty(M, 4 * n, dtype=bf, device=dev)
        by, fl = 2.0 * (4 * M * H + 4 * H * n + 4 * M * n), 8.0 * M * H * n
        t = timeit(lambda i: ops.gemm(a5[:, :4 * H], ws[i], out=o4, groups=4, static_b=True), copies=nc)
        rep("gemm of four mixes (block-diagonal)", t, by=by, fl=fl, M=M)
        wide = [w_.view(H, 4 * n) for w_ in ws]
        t = timeit(lambda i: ops.gemm(a, wide[i], out=o4, static_b=True), copies=nc)
        rep("gemm store, as many columns (uniform model)", t, by=2.0 * (M * H + 4 * H * n + 4 * M * n), fl=fl, M=M)
        del ws, wide
        w1, low = rnd(H, rank), torch.empty(M, rank, device=dev)
        narrow = dict(bn=64, split_k=4 if M <= 2048 else 1) if M > ops.DECODE_GEMM_MAX_M else {}
        t = timeit(lambda i: ops.gemm(a5[:, 4 * H:], w1, out=low, static_b=True, **narrow))
        rep("gemm decay, narrow", t, by=2.0 * (M * H + H * rank) + 4.0 * M * rank, fl=2.0 * M * H * rank, M=M)
    # ---- linear attention
    gh, gd, gv, gr = hb.SIZES[size][5], hb.SIZES[size][6], hb.SIZES[size][7], 16
    a2, a2b, gn = rnd(gr, gh * gd) * gr ** -0.5, 2 + rnd(gh * gd), rnd(gv)
    gw = 2 * gh * gd + 2 * gh * gv + gr
    gcut = lambda x: x.split([gh * gd, gh * gd, gh * gv, gh * gv, gr], 1)
    w2, w0, bonus, on = rnd(rank, n) * rank ** -0.5, -2.5 + 0.5 * rnd(n), rnd(n), rnd(n)
    w3 = w0 + 3
    for lens in ([8192], [2048] * 4, [256] * 32):
        T, B = sum(lens), len(lens)
        pos, indptr, slots = i32([p for k in lens for p in range(k)]), i32([sum(lens[:i]) for i in range(B + 1)]), torch.arange(B, dtype=torch.int32, device=dev)
        x, o = rnd(T, gw), torch.empty(T, gh * gv, dtype=bf, device=dev)
        st, cum = torch.zeros(B, gh, gd, gv, device=dev), torch.empty(T * max(gh * gd, n), device=dev)
        t = timeit(lambda i: ops.gla(*gcut(x), a2, a2b, gn, st, o, pos, indptr, slots, rank=gr, tau=16.0, eps=1e-6, row_lens=lens, cum=cum))
        rep("gla prompts (Fafudra)", t, by=T * 2.0 * (gw + gh * gv) + B * gh * gd * gv * 8.0, fl=T * gh * (4.0 * gd * gv + 64.0 * (gd + gv)), sequences=B, length=lens[0])
        x, low, o, st = rnd(T, 4 * n), torch.randn(T, rank, device=dev), torch.empty(T, n, dtype=bf, device=dev), torch.zeros(B, wh, wd, wd, device=dev)
        t = timeit(lambda i: ops.wkv(*x.split(n, 1), low, w2, w0, bonus, on, st, o, pos, indptr, slots, rank=rank, eps=1e-5, row_lens=lens, cum=cum))
        t2 = timeit(lambda i: ops.wkv(*x.split(n, 1), low, w2, w3, bonus, on, st, o, pos, indptr, slots, rank=rank, eps=1e-5, row_lens=lens, cum=cum))
        rep("wkv prompts, very fast decays", t2, by=T * (10.0 * n + 4.0 * rank) + B * wh * wd * wd * 8.0, fl=T * wh * (4.0 * wd * wd + 128.0 * wd), sequences=B, length=lens[0])
        rep("wkv prompts", t, by=T * (10.0 * n + 4.0 * rank) + B * wh * wd * wd * 8.0, fl=T * wh * (4.0 * wd * wd + 128.0 * wd), sequences=B, length=lens[0])
        S, P, N, G = sp["heads"], sp["vdim"], sp["state"], sp["groups"]
        u, z, o, st = rnd(T, C), rnd(T, S * P + S), torch.empty(T, S * P, dtype=bf, device=dev), torch.zeros(B, S, N, P, device=dev)
        db = -2 + rnd(S)
        t = timeit(lambda i: ops.ssd(*u.split([S * P, G * N, G * N], 1), z[:, :S * P], z[:, S * P:], db, db, db, st, o, pos, indptr, slots, groups=G, row_lens=lens))
        rep("ssd prompts", t, by=T * 2.0 * (C + 2 * S * P + S) + B * S * N * P * 8.0, fl=T * S * (4.0 * N * P + 64.0 * P) + T * G * 64.0 * N, sequences=B, length=lens[0])
    for B in (256, 16, 1):
        slots, pos = torch.arange(B, dtype=torch.int32, device=dev), torch.full((B,), 5, dtype=torch.int32, device=dev)
        states = lambda *s: [torch.zeros(B, *s, device=dev) for _ in range(min(40, n_copies(4 * B * s[0] * s[1] * s[2])))]
        x, o, sts = rnd(B, gw), torch.empty(B, gh * gv, dtype=bf, device=dev), states(gh, gd, gv)
        t = timeit(lambda i: ops.gla(*gcut(x), a2, a2b, gn, sts[i], o, pos, None, slots, rank=gr, tau=16.0, eps=1e-6), copies=len(sts))
        rep("gla decode (Fafudra)", t, by=B * (gh * gd * gv * 8.0 + 2.0 * gw), batch=B)
        x, low, o, sts = rnd(B, 4 * n), torch.randn(B, rank, device=dev), torch.empty(B, n, dtype=bf, device=dev), states(wh, wd, wd)
        t = timeit(lambda i: ops.wkv(*x.split(n, 1), low, w2, w0, bonus, on, sts[i], o, pos, None, slots, rank=rank, eps=1e-5), copies=len(sts))
        rep("wkv decode", t, by=B * (wh * wd * wd * 8.0 + 10.0 * n), batch=B)
        u, z, o, sts = rnd(B, C), rnd(B, S * P + S), torch.empty(B, S * P, dtype=bf, device=dev), states(S, N, P)
        t = timeit(lambda i: ops.ssd(*u.split([S * P, G * N, G * N], 1), z[:, :S * P], z[:, S * P:], db, db, db, sts[i], o, pos, None, slots, groups=G), copies=len(sts))
        rep("ssd decode", t, by=B * (S * N * P * 8.0 + 2.0 * (C + 2 * S * P)), batch=B)
    for T in (8192, 256, 16):
        width = S * P
        xs, w = [rnd(T, width) for _ in range(min(40, n_copies(T * width * 2)))], rnd(width)
        o = torch.empty(T, width, dtype=bf, device=dev)
        t = timeit(lambda i: ops.rms_norm(xs[i], w, out=o), copies=len(xs))
        rep("rms_norm (uniform model)", t, by=T * width * 4.0, tokens=T)
        t = timeit(lambda i: ops.part_norm(xs[i], w, sp["norm_groups"], 1e-5), copies=len(xs))
        rep("part_norm", t, by=T * width * 4.0, tokens=T)
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
    return {"metric": "norusun_vs_fafudra_vs_uniform", "dtype": "bf16", "data": "synthetic token ids, random-init weights", "layers": LAYERS, "rows": out}
