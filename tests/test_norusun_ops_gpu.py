"""Mechanisms of the Norusun design in the kernels, each against a plain fp64 computation, on inputs that make a mistake visible: keys
that stand out just inside and outside windows and chunks, histories and states left behind by other sequences, fast and slow
decays, sizes of every kind."""
import math

import pytest
import torch
import torch.nn.functional as F

import norusun_plain as plain

pytestmark = pytest.mark.gpu

DEV = "cuda"
BF, F32, HF = torch.bfloat16, torch.float32, torch.float16


@pytest.fixture(scope="module")
def ops():
    torch.cuda.set_device(0)
    from blitz_scale_b200 import ops as o
    return o


def _rel(a, b):
    return float((a.double().cpu() - b.double().cpu()).norm() / b.double().cpu().norm())


def _worst(got, want):
    """Largest relative error of a row."""
    got, want = got.double().cpu().flatten(1), want.double().flatten(1)
    return float(((got - want).norm(dim=1) / want.norm(dim=1).clamp_min(1e-2 * want.norm(dim=1).max())).max())


def _i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


pad = lambda n: (n + 7) // 8 * 8
d = lambda t: t.double()
dev = lambda t: t.to(DEV)


# ------------------------------------------------------------------------------------------------ streams
@pytest.mark.parametrize("S", [1, 2, 3, 5, 8])
@pytest.mark.parametrize("H", [7, 64, 1100, 4096, 9000])
@pytest.mark.parametrize("dt", [BF, F32])
def test_streams(ops, S, H, dt):
    g = torch.Generator().manual_seed(S * H)
    r = lambda *s: torch.randn(*s, generator=g)
    T, V, eps = 9, 30, 0.05
    x, embed, y = r(T, S, H), r(V, H).to(dt), r(T, 2 * H).to(dt)
    mix, out_w, in_w = r(S, S).to(dt), r(S).to(dt), r(S).to(dt)
    bias, w0, w1, w = (r(H).to(dt) for _ in range(4))
    ids = torch.randint(0, V, (T,), generator=g)
    tol = 3e-6 if dt == F32 else 4e-3
    half = lambda a, wt: plain.rms(d(a), eps) * d(wt)
    co = (dev(mix), dev(out_w))
    sources = {"none": (None, None), "dense": (ops.Pending(dev(y[:, :H].contiguous()), *co), d(y[:, :H])),
               "bias": (ops.Pending(dev(y[:, :H].contiguous()), *co, bias=dev(bias)), d(y[:, :H]) + d(bias)),
               "two": (ops.Pending(dev(y), *co, norms=(dev(w0), dev(w1))), 0.5 * (half(y[:, :H], w0) + half(y[:, H:], w1)))}
    for fresh in (False, True):
        start = d(embed)[ids][:, None].expand(T, S, H) if fresh else d(x)
        kw = dict(eps=eps, **(dict(ids=_i32(ids.tolist()), embed=dev(embed)) if fresh else {}))
        for name, (pending, want_y) in sources.items():
            for weight, off in ((w[:1], 0.0), (w, 0.5)):
                xs = start.transpose(0, 1)
                if pending is not None:
                    xs = plain.streams_out(xs, d(mix), d(out_w), want_y)
                norm = lambda u: plain.rms(u, eps) * (off + d(weight))
                xd, h = x.to(DEV), torch.full((T, H), 9.0, dtype=dt, device=DEV)
                ops.stream_rms(xd, **kw, pending=pending, read=dev(in_w), w=dev(weight), w_offset=off, out=h, write=pending is not None)
                assert _rel(h, norm(plain.streams_in(xs, d(in_w)))) < tol, (name, fresh)
                assert _rel(xd.transpose(0, 1), xs if pending is not None else d(x).transpose(0, 1)) < 1e-6
                h32 = torch.empty(T, H, device=DEV)
                ops.stream_rms(x.to(DEV), **kw, pending=pending, read=dev(in_w), w=dev(weight), w_offset=off, out=h32)
                assert _rel(h32, norm(plain.streams_in(xs, d(in_w)))) < 3e-6
                # some rows only, nothing kept, the plain sum
                at = torch.tensor([5, 2, 9, 2])
                xd, h, tot = x.to(DEV), torch.empty(4, H, dtype=dt, device=DEV), torch.empty(4, H, device=DEV)
                ops.stream_rms(xd, **kw, pending=pending, w=dev(weight), w_offset=off, out=h, total=tot, rows=_i32(at.tolist()), row_offset=-1)
                assert _rel(tot, xs.sum(0)[at - 1]) < 2e-6 and _rel(h, norm(xs.sum(0))[at - 1]) < tol
                assert torch.equal(xd.cpu(), x)
    ops.check_status()
    ops.stream_rms(x.to(DEV), eps=eps, ids=_i32([0, V] + [1] * (T - 2)), embed=dev(embed), w=dev(w), out=torch.empty(T, H, dtype=dt, device=DEV))
    with pytest.raises(RuntimeError):          # a token id outside the vocabulary is reported, not read
        ops.check_status()


def _mixes(h, mu):
    """[T, mixes * width]"""
    prev = plain.shifted(h)
    return torch.cat([h + (prev - h) * m for m in mu], 1)


@pytest.mark.parametrize("taps,mixes", [(1, 0), (2, 0), (4, 0), (4, 5), (7, 3), (1, 5), (16, 1)])
@pytest.mark.parametrize("H", [7, 64, 1100])
@pytest.mark.parametrize("dt", [BF, F32])
def test_convolved_input_of_decoded_tokens(ops, taps, mixes, H, dt):
    """Sequences that decode side by side on slots with other sequences' remains, one of them idle at times, beside padding rows."""
    g = torch.Generator().manual_seed(taps * H)
    r = lambda *s: torch.randn(*s, generator=g)
    n, slots, lens = 3, 5, (20, 9, 14)
    conv, mu, w = (0.6 * r(taps, H)).to(dt), (0.5 + 0.4 * r(mixes, H)).to(dt) if mixes else None, r(1).to(dt)
    one = torch.ones(1, dtype=dt, device=DEV)
    state = ops.TokenState(dev(conv), torch.full((slots, taps - 1, H), 50.0, device=DEV), dev(mu) if mixes else None,
                           torch.full((slots, H), 50.0, device=DEV) if mixes else None)
    x = [r(k, 1, H) for k in lens]
    want = []
    for s in x:
        h = plain.rms(d(s[:, 0]), 0.01) * d(w)
        c = h + plain.causal_conv(h, d(conv).T)
        want.append(_mixes(c, d(mu)) if mixes else c)
    slot_of, at, got = (3, 0, 4), [0] * n, [[] for _ in lens]
    k = 0
    while any(a < m for a, m in zip(at, lens)):
        live = [i for i in range(n) if at[i] < lens[i] and not (i == 1 and k % 3 == 1)]
        rows = torch.cat([x[i][at[i]:at[i] + 1] for i in live] + [r(1, 1, H)])
        out = torch.empty(len(live) + 1, max(1, mixes) * H, dtype=dt, device=DEV)
        ops.stream_rms(rows.to(DEV), eps=0.01, read=one, w=dev(w), out=out, tokens=state, pos=_i32([at[i] for i in live] + [0]),
                       seq_slot=_i32([slot_of[i] for i in live] + [-1]))
        for j, i in enumerate(live):
            got[i].append(out[j].cpu())
            at[i] += 1
        k += 1
    ops.check_status()
    for a, b in zip(got, want):
        assert _worst(torch.stack(a), b) < (3e-6 if dt == F32 else 5e-3)
    if taps > 1:
        assert bool((state.hist[[1, 2]] == 50.0).all())


# ------------------------------------------------------------------------------------------------ short convolutions
@pytest.mark.parametrize("W", [5, 64, 1036, 8200])
@pytest.mark.parametrize("taps,mixes", [(1, 0), (3, 0), (4, 0), (4, 5), (6, 2), (1, 5), (2, 1)])
@pytest.mark.parametrize("dt,xt", [(BF, BF), (BF, F32), (F32, F32)])
def test_token_convolution(ops, W, taps, mixes, dt, xt):
    """Portions of many sizes of several sequences side by side, on slots that hold other sequences' remains."""
    g = torch.Generator().manual_seed(W + taps)
    r = lambda *s: torch.randn(*s, generator=g)
    conv, bias = (r(taps, W) * taps ** -0.5).to(dt), (0.3 * r(W)).to(dt)
    mu = (0.5 + 0.4 * r(mixes, W)).to(dt) if mixes else None
    cuts = {0: [1, 2, 40, 1, 3, 53], 1: [2, 2, 1, 1, 2, 1], 2: [70, 1, 0, 1, 1, 30]}
    x = {i: r(sum(c), W).to(xt) for i, c in cuts.items()}
    kind = dict(residual=True) if mixes else dict(bias=dev(bias), silu=True) if taps % 2 == 0 else dict(bias=dev(bias))

    def expect(s):
        c = plain.causal_conv(d(s), d(conv).T)
        if mixes:
            return _mixes(d(s) + c, d(mu))
        c = c + d(bias)
        return F.silu(c) if taps % 2 == 0 else c
    hist = torch.full((5, taps - 1, W), 30.0, dtype=xt, device=DEV)
    shift = torch.full((5, W), 30.0, dtype=xt, device=DEV) if mixes else None
    got, at, slot = {i: [] for i in cuts}, {i: 0 for i in cuts}, {0: 4, 1: 2, 2: 0}
    for k in range(6):
        live = [i for i in cuts if cuts[i][k]]
        n = [cuts[i][k] for i in live]
        buf = torch.zeros(sum(n), W + 8, dtype=xt, device=DEV)       # a column range of a wider buffer
        rows = buf[:, :W]
        rows.copy_(torch.cat([x[i][at[i]:at[i] + c] for i, c in zip(live, n)]))
        out = torch.full((sum(n), max(1, mixes) * W), 9.0, dtype=dt, device=DEV)
        more = dict(mu=dev(mu), shift=shift, last=torch.empty(len(n), W, dtype=xt, device=DEV)) if mixes else {}
        pos = _i32([at[i] + t for i, c in zip(live, n) for t in range(c)])
        single = not mixes and all(c == 1 for c in n)
        ops.token_conv(rows, dev(conv), hist, out, pos, None if single else _i32([sum(n[:j]) for j in range(len(n) + 1)]),
                       _i32([slot[i] for i in live]), **kind, **more)
        first = 0
        for i, c in zip(live, n):
            got[i].append(out[first:first + c].cpu())
            first += c
            at[i] += c
    ops.check_status()
    for i in cuts:
        assert _worst(torch.cat(got[i]), expect(x[i])) < (4e-6 if dt == F32 else 8e-3), i
        keep = min(taps - 1, len(x[i]))
        assert keep == 0 or torch.equal(hist[slot[i], taps - 1 - keep:].cpu(), x[i][len(x[i]) - keep:])
    assert taps == 1 or bool((hist[[1, 3]] == 30.0).all())


def test_convolution_of_a_long_prompt(ops):
    g = torch.Generator().manual_seed(0)
    T, W = 5000, 512
    x, conv = torch.randn(T, W, generator=g).to(BF), torch.randn(4, W, generator=g).to(BF)
    out, hist = torch.empty(T, W, dtype=BF, device=DEV), torch.zeros(1, 3, W, dtype=BF, device=DEV)
    ops.token_conv(dev(x), dev(conv), hist, out, _i32(list(range(T))), _i32([0, T]), _i32([0]), silu=True)
    ops.check_status()
    assert _worst(out, F.silu(plain.causal_conv(d(x), d(conv).T))) < 8e-3 and torch.equal(hist[0].cpu(), x[-3:])


# ------------------------------------------------------------------------------------------------ clamped unit
@pytest.mark.parametrize("M", [1, 5, 64, 130, 256, 300, 1000])
@pytest.mark.parametrize("N,K", [(136, 200), (512, 256), (1408, 96), (51, 121), (72, 64)])
@pytest.mark.parametrize("dt", [BF, HF, F32])
def test_clamped_unit(ops, M, N, K, dt):
    g = torch.Generator().manual_seed(M + N)
    pn = pad(N) if N % 8 and dt != F32 else N
    a, b, c = torch.randn(M, K, generator=g).to(dt), torch.zeros(K, 2 * pn), torch.zeros(2 * pn)
    for at in (0, pn):
        b[:, at:at + N] = 1.5 * torch.randn(K, N, generator=g) * K ** -0.5
        c[at:at + N] = 0.7 * torch.randn(N, generator=g)
    b, c = b.to(dt), c.to(dt)
    for limit, beta in ((1.1, 1.702), (0.25, 0.5), (1e30, 3.0)):
        z = d(a) @ d(b) + d(c)
        gate, up = z[:, :pn].clamp(max=limit), z[:, pn:].clamp(-limit, limit)
        want = gate * torch.sigmoid(beta * gate) * (up + 1)
        for path in ({}, dict(decode_path=False, pair_path=False), dict(pair_path=True), dict(bn=128, split_k=3)):
            if path and (dt == F32 or pn % 8 or K % 8 or K < 192 and "split_k" in path or ("pair_path" in path and pn < 64)):
                continue
            out = torch.full((M, pn), 7.0, dtype=dt, device=DEV)
            ops.gemm(dev(a), dev(b), out=out, epilogue="clamp_glu", alpha=limit, beta=beta, bias=dev(c), static_b=True, **path)
            ops.check_status()
            assert _rel(out, want) < {F32: 3e-6, BF: 4e-3, HF: 1e-3}[dt], (limit, path)


# ------------------------------------------------------------------------------------------------ norm over whole rows, rotation
@pytest.mark.parametrize("dim,vdim,rot,qh,kvh", [(64, 64, 24, 6, 3), (128, 96, 128, 12, 1), (40, 24, 8, 4, 2), (22, 13, 10, 9, 3), (64, 64, 64, 1, 1), (16, 8, 0, 2, 2)])
@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("pairs", [False, True])
def test_norm_of_whole_rows_before_the_rotation(ops, dim, vdim, rot, qh, kvh, dt, pairs):
    g = torch.Generator().manual_seed(dim)
    page, eps, base, slot = 16, 0.02, 500.0, [3, 17, 40, 111, 64, -1, 0]
    T = len(slot)
    at = [0, pad(qh * dim), pad(qh * dim) + pad(kvh * dim)]
    x = torch.randn(T, at[2] + pad(kvh * vdim) + 16, generator=g).to(dt)
    cut = lambda t: (t[:, :qh * dim], t[:, at[1]:at[1] + kvh * dim], t[:, at[2]:at[2] + kvh * vdim])
    qw, kw = (1 + 0.5 * torch.randn(qh * dim, generator=g)).to(dt), (1 + 0.5 * torch.randn(kvh * dim, generator=g)).to(dt)
    q, k, v = map(d, cut(x))
    want_q = plain.rotate((plain.rms(q, eps) * d(qw)).view(T, qh, dim), rot, base, pairs)
    want_k = plain.rotate((plain.rms(k, eps) * d(kw)).view(T, kvh, dim), rot, base, pairs)
    kv = torch.zeros(7, 2, page, kvh, dim, dtype=dt, device=DEV) if dim == vdim else ops.KVPair(
        torch.zeros(7, page, kvh, dim, dtype=dt, device=DEV), torch.zeros(7, page, kvh, vdim, dtype=dt, device=DEV))
    xd = x.to(DEV)
    ops.rope_store(*cut(xd), _i32(list(range(T))), _i32(slot), kv, ops.rope_freqs(rot, base, DEV), q_heads=qh, kv_heads=kvh, dim=dim, rot_dims=rot,
                   page_size=page, interleaved=pairs, q_w=dev(qw), k_w=dev(kw), eps=eps)
    ops.check_status()
    tol = 2e-6 if dt == F32 else 5e-3
    assert _rel(cut(xd)[0].reshape(T, qh, dim), want_q) < tol
    assert torch.equal(xd[:, qh * dim:].cpu(), x[:, qh * dim:])
    K, V = (t.reshape(7 * page, kvh, -1).cpu() for t in ((kv[0], kv[1]) if isinstance(kv, tuple) else (kv[:, 0], kv[:, 1])))
    for t, s in enumerate(slot):
        if s >= 0:
            assert _rel(K[s], want_k[t]) < tol and torch.equal(V[s], v[t].view(kvh, vdim).to(dt))
    assert sum(bool(r.any()) for r in K) == len(slot) - 1


# ------------------------------------------------------------------------------------------------ sigmoid weights in chunks
# (heads, kv heads, dim, vdim, page, chunk)
CHUNKS = [(6, 3, 64, 64, 16, 50), (12, 1, 128, 96, 64, 130), (4, 4, 40, 24, 16, 128), (9, 3, 22, 13, 16, 7), (16, 2, 128, 128, 64, 64), (1, 1, 8, 128, 128, 1),
          (4, 2, 64, 64, 32, 1000), (10, 2, 72, 40, 8, 257), (2, 2, 64, 64, 64, 0)]


@pytest.mark.parametrize("softmax", [False, True])
@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("case", CHUNKS)
def test_attention_in_chunks(ops, case, dt, softmax):
    """Prompts, portions behind any prefix, and single tokens with and without key splits.  One key in twelve, and those on both
    sides of every chunk's edge and around pages, take most of the weight; the values of keys outside are large."""
    H, G, dim, dv, page, chunk = case
    if softmax and not chunk:
        return
    lens, q_lens = [700, 65, 1, 300, 389], [700, 65, 1, 2, 260]
    g = torch.Generator().manual_seed(H * dim + dv)
    scale = 0.8 * dim ** -0.5
    bias = (torch.randn(H, 1, generator=g) - 2.0).to(dt)
    npages = [-(-n // page) for n in lens]
    perm = torch.randperm(sum(npages), generator=g).tolist()
    shape = (sum(npages), page, G)
    kv = torch.zeros(shape[0], 2, *shape[1:], dim, dtype=dt, device=DEV) if dim == dv else ops.KVPair(
        torch.zeros(*shape, dim, dtype=dt, device=DEV), torch.zeros(*shape, dv, dtype=dt, device=DEV))
    K, V = (kv[0], kv[1]) if isinstance(kv, tuple) else (kv[:, 0], kv[:, 1])
    u = torch.randn(dim, generator=g)
    u = u / u.norm() * dim ** 0.5
    want, qs, at = [], [], 0
    for n, ql, np_ in zip(lens, q_lens, npages):
        k, v = torch.randn(n, G, dim, generator=g), torch.randn(n, G, dv, generator=g).to(dt)
        size = chunk or 10 ** 6
        loud = sorted({p for e in range(0, n + 1, size) for p in (e - 1, e)} | {p for e in range(0, n, page) for p in (e, e + page - 1)} | set(range(0, n, 12)))
        loud = [p for p in loud if 0 <= p < n]
        k[loud] = 0.3 * k[loud] + 0.8 * u
        k, q = k.to(dt), (0.5 * torch.randn(n, H, dim, generator=g) + u).to(dt)
        for i in range(np_):
            part = slice(i * page, min(n, (i + 1) * page))
            K[perm[at + i], :part.stop - part.start] = k[part].to(DEV)
            V[perm[at + i], :part.stop - part.start] = v[part].to(DEV)
        at += np_
        flaws = ("softmax", "no_weight_bias") if softmax else ()
        o = torch.stack([plain.sigmoid_attention(d(q[:, h]), d(k[:, h // (H // G)]), d(v[:, h // (H // G)]), scale, size, d(bias[h]), flaws) for h in range(H)], 1)
        want.append(o[n - ql:])
        qs.append(q[n - ql:])
    T = sum(q_lens)
    proj = torch.zeros(T, pad(H * dim) + 8, dtype=dt, device=DEV)
    q = proj[:, :H * dim]
    q.copy_(torch.cat(qs).reshape(T, -1))
    pos = _i32([p for n, ql in zip(lens, q_lens) for p in range(n - ql, n)])
    tokp, indptr = (_i32([sum(x[:i]) for i in range(len(lens) + 1)]) for x in (q_lens, npages))
    indices, last = _i32(perm), _i32([n - (c - 1) * page for n, c in zip(lens, npages)])
    tol = 8e-6 if dt == F32 else 2.4e-2

    def check(out, rows, what):
        ops.check_status()
        for i, (w, r) in enumerate(zip(want, rows)):
            assert _worst(out[r].reshape(-1, H, dv), w[-len(r):]) < tol, (what, i)
    all_rows = [list(range(int(tokp[i]), int(tokp[i + 1]))) for i in range(len(lens))]
    extra = dict(window=chunk, chunked=chunk > 0, **(dict() if softmax else dict(sigmoid=True, bias=dev(bias))))
    buf = torch.full((T, pad(H * dv) + 8), 7.0, dtype=dt, device=DEV)
    ops.attn_ragged(q, kv, pos, tokp, indptr, indices, buf, q_heads=H, kv_heads=G, dim=dim, page_size=page, scale=scale, **extra)
    check(buf[:, :H * dv], all_rows, "general")
    if not ops.attn_tensor_core(q, H, G, dim, page, dv):
        assert dt == F32 or dim % 8 or dv % 8
        return
    buf.fill_(7.0)
    kw = dict(q_heads=H, kv_heads=G, head_dim=dim, page_size=page, sm_scale=scale, **extra)
    ops.attn_prefill_paged(q, kv, indices, ops.prefill_work_list(q_lens, lens, page, DEV), out=buf, **kw)
    check(buf[:, :H * dv], all_rows, "prefill")
    assert bool((buf[:, H * dv:] == 7.0).all())
    last_rows = [r[-1] for r in all_rows]
    for splits in (1, 2, 8):
        o = torch.full((len(lens), pad(H * dv) + 8), 7.0, dtype=dt, device=DEV)
        ops.attn_decode(q[last_rows], kv, indices, indptr, last, num_splits=splits, out=o, **kw)
        check(o[:, :H * dv], [[i] for i in range(len(lens))], ("decode", splits))
        assert bool((o[:, H * dv:] == 7.0).all())


# ------------------------------------------------------------------------------------------------ latent attention
@pytest.mark.parametrize("heads,dim,rot", [(5, 48, 16), (32, 64, 32), (3, 13, 6), (1, 8, 2), (40, 128, 64), (4, 24, 8)])
@pytest.mark.parametrize("dt", [BF, F32])
def test_latent_rotation_of_neighbours(ops, heads, dim, rot, dt):
    g = torch.Generator().manual_seed(dim)
    T, base, rank, page = 40, 300.0, 24, 8
    q = torch.randn(T, heads * (dim + rot), generator=g).to(dt)
    want = plain.rotate(d(q).view(T, heads, dim + rot)[..., dim:], rot, base, True)
    fr, pos = ops.rope_freqs(rot, base, DEV), _i32(list(range(T)))
    tol = 2e-6 if dt == F32 else 4e-3
    args = dict(heads=heads, dim=dim, rot=rot, interleaved=True)
    inplace = q.to(DEV)
    ops.latent_rotate(inplace, inplace[:, dim:], pos, fr, out_step=dim + rot, **args)
    got = inplace.view(T, heads, dim + rot)
    assert _rel(got[..., dim:], want) < tol and torch.equal(got[..., :dim].cpu(), q.view(T, heads, -1)[..., :dim])
    out = torch.full((T, heads * (rank + rot)), 7.0, dtype=dt, device=DEV)
    ops.latent_rotate(q.to(DEV), out[:, rank:], pos, fr, out_step=rank + rot, **args)
    got = out.view(T, heads, rank + rot)
    assert _rel(got[..., rank:], want) < tol and bool((got[..., :rank] == 7.0).all())
    # the keys' shared part, with the write
    x, w = torch.randn(T, rank + rot, generator=g).to(dt), (1 + 0.3 * torch.randn(rank, generator=g)).to(dt)
    kv = ops.LatentKV(torch.zeros(6, page, 1, rank + rot, dtype=dt, device=DEV), rank)
    ops.latent_store(None, dev(x), pos, _i32(list(range(4, T + 4))), kv, None, dev(w), fr, eps=0.02, interleaved=True)
    ops.check_status()
    rows = kv.pool.view(-1, rank + rot)[4:T + 4]
    assert _rel(rows[:, :rank], plain.rms(d(x[:, :rank]), 0.02) * d(w)) < tol and _rel(rows[:, rank:], plain.rotate(d(x[:, rank:]), rot, base, True)) < tol


LATENT = [(1, 80, 64, 64, 1), (5, 136, 104, 16, 37), (32, 288, 256, 64, 64), (40, 96, 80, 8, 129), (64, 576, 512, 64, 500), (128, 320, 320, 128, 63), (33, 16, 8, 32, 0),
          (20, 360, 320, 16, 200)]


@pytest.mark.parametrize("lens", [[1], [130, 0, 700, 64, 65, 37, 38], [(i * 37) % 300 for i in range(170)], [3000]])
@pytest.mark.parametrize("case", LATENT)
def test_latent_decode_attention_in_a_window(ops, case, lens):
    """A sink that takes about half of the weight; the keys just inside and just outside the window stand out, those outside most."""
    H, W, R, page, window = case
    B = len(lens)
    for dt in (BF, HF, F32):
        if dt != BF and B > 7:
            continue
        g = torch.Generator().manual_seed(H + B)
        npages = [-(-n // page) for n in lens]
        perm = torch.randperm(sum(npages) + 2, generator=g)[:max(1, sum(npages))].tolist()
        kv = ops.LatentKV(torch.zeros(sum(npages) + 2, page, 1, W, dtype=dt, device=DEV), R)
        q, scale = torch.randn(B, H, W, generator=g), 0.8 * W ** -0.5
        sink = (0.8 * W ** 0.5 * 0.9 + torch.randn(H, generator=g)).to(dt)
        want, at = torch.zeros(B, H, R, dtype=torch.float64), 0
        u = torch.randn(W, generator=g)
        u = u / u.norm() * W ** 0.5
        q = (0.5 * q + u).to(dt)
        for b, n in enumerate(lens):
            k = torch.randn(n, W, generator=g)
            edge = n - window if window else 0
            loud = sorted({p for p in (edge, edge + 1, page - 1, page, 63, 64, 127, 128, n // 2, n - 1) if 0 <= p < n})
            k[loud] = k[loud] * 0.3 + 0.9 * u
            if window and 0 < edge <= n:
                k[max(0, edge - 2):edge] += 1.2 * u
            k = k.to(dt)
            for i in range(npages[b]):
                part = k[i * page:(i + 1) * page]
                kv.pool[perm[at + i], :len(part), 0] = part.to(DEV)
            at += npages[b]
            lo = max(0, edge)
            if n:
                s = torch.cat([d(q[b]) @ d(k[lo:]).T * scale, d(sink)[:, None]], 1)
                want[b] = torch.softmax(s, -1)[:, :-1] @ d(k[lo:, :R])
        indptr = _i32([sum(npages[:i]) for i in range(B + 1)])
        last = _i32([n - (p - 1) * page if p else 0 for n, p in zip(lens, npages)])
        qd, out = q.reshape(B, -1).to(DEV), torch.full((B, H * R), 7.0, dtype=dt, device=DEV)
        live = [b for b, n in enumerate(lens) if n]
        extra = dict(window=window, sink=dev(sink))

        def check(what):
            ops.check_status()
            if live:
                assert _worst(out.view(B, H, R)[live], want[live]) < (8e-6 if dt == F32 else 2e-2), (what, dt)
            assert all(not out[b].any() for b, n in enumerate(lens) if n == 0)
        ops.attn_ragged(qd, kv, _i32([max(0, n - 1) for n in lens]), None, indptr, _i32(perm), out, q_heads=H, kv_heads=1, dim=W, page_size=page,
                        scale=scale, **extra)
        check("general")
        if dt != F32:
            for keys in (0, 64):
                out.fill_(7.0)
                ops.attn_latent(qd, kv, _i32(perm), indptr, last, heads=H, scale=scale, workspace=ops.attn_latent_workspace(H, R, DEV), out=out, keys=keys, **extra)
                check("tensor cores")


@pytest.mark.parametrize("H,W,R,page,window", [(5, 136, 104, 16, 37), (32, 544, 512, 64, 129), (72, 80, 64, 32, 1)])
def test_latent_attention_of_prompt_tokens_in_a_window(ops, H, W, R, page, window):
    """Tokens of a ragged step as rows of their own, behind any prefix, in several launches: against the general kernel."""
    lens, q_lens = [900, 1, 65, 300, 1100], [900, 1, 2, 260, 130]
    g = torch.Generator().manual_seed(H)
    npages = [-(-n // page) for n in lens]
    perm = torch.randperm(sum(npages), generator=g).tolist()
    kv = ops.LatentKV(torch.randn(sum(npages), page, 1, W, generator=g).to(DEV, BF), R)
    T = sum(q_lens)
    q, sink = torch.randn(T, H * W, generator=g).to(DEV, BF), (2 + torch.randn(H, generator=g)).to(DEV, BF)
    pos = _i32([p for n, ql in zip(lens, q_lens) for p in range(n - ql, n)])
    tokp, indptr = (_i32([sum(x[:i]) for i in range(len(lens) + 1)]) for x in (q_lens, npages))
    want, got = torch.empty(T, H * R, dtype=BF, device=DEV), torch.full((T, H * R), math.nan, dtype=BF, device=DEV)
    scale, extra = 1.2 * W ** -0.5, dict(window=window, sink=sink)
    ops.attn_ragged(q, kv, pos, tokp, indptr, _i32(perm), want, q_heads=H, kv_heads=1, dim=W, page_size=page, scale=scale, **extra)
    ops.attn_latent(q, kv, _i32(perm), indptr, indptr, heads=H, scale=scale, workspace=ops.attn_latent_workspace(H, R, DEV), out=got,
                    pos=pos, tok_indptr=tokp, **extra)
    ops.check_status()
    err = (got.float() - want.float()).norm(dim=1) / want.float().norm(dim=1)
    assert float(err.max()) < 2e-2, int(err.argmax())


# ------------------------------------------------------------------------------------------------ recurrences
def _portions(ops, cuts, slots, run, whole, tol, keep=None):
    """Sequences in portions side by side on used slots: run(live, starts, counts, pos, tok_indptr, seq_slot, lens) gives the rows."""
    got, at = {i: [] for i in cuts}, {i: 0 for i in cuts}
    for k in range(max(map(len, cuts.values()))):
        live = [i for i in cuts if k < len(cuts[i]) and cuts[i][k]]
        n = [cuts[i][k] for i in live]
        pos = _i32([at[i] + t for i, c in zip(live, n) for t in range(c)])
        single = all(c == 1 for c in n)
        out = run([(i, at[i], c) for i, c in zip(live, n)], pos, None if single else _i32([sum(n[:j]) for j in range(len(n) + 1)]),
                  _i32([slots[i] for i in live]), n)
        ops.check_status()
        first = 0
        for i, c in zip(live, n):
            got[i].append(out[first:first + c].cpu())
            first += c
            at[i] += c
    for i in cuts:
        assert _worst(torch.cat(got[i]), whole[i]) < tol, i


@pytest.mark.parametrize("heads,dim,rank", [(5, 40, 12), (2, 64, 24), (1, 128, 64), (3, 13, 5), (7, 32, 8), (1, 8, 1), (2, 200, 7), (24, 96, 16)])
@pytest.mark.parametrize("decay", ["slow", "mixed", "fast"])
@pytest.mark.parametrize("dt", [BF, F32])
def test_wkv(ops, heads, dim, rank, decay, dt):
    """Portions of every size against the recurrence token by token; decays from almost none to more than e^-80 per token."""
    g = torch.Generator().manual_seed(heads * dim)
    r = lambda *s: torch.randn(*s, generator=g)
    n, eps = heads * dim, 1e-4
    cuts = {0: [1, 2, 64, 1, 15, 33, 130], 1: [200, 1, 1, 2, 40], 2: [3, 1, 1, 17, 0, 1, 64], 3: [64, 63, 1, 128]}
    tok = {i: sum(c) for i, c in cuts.items()}
    x = {i: (r(t, 4 * n)).to(dt) for i, t in tok.items()}
    low = {i: 2.0 * r(t, rank) for i, t in tok.items()}
    w2, bonus, norm = (1.5 * r(rank, n) * rank ** -0.5).to(dt), (0.5 + 1.5 * r(n)).to(dt), (1 + 0.3 * r(n)).to(dt)
    w0 = ({"slow": -6.0, "mixed": -1.5, "fast": 1.5}[decay] + {"slow": 0.5, "mixed": 2.5, "fast": 2.0}[decay] * r(n)).to(dt)
    whole = {}
    for i, t in tok.items():
        q, k, v, gate = (d(a) for a in x[i].split(n, 1))
        w = torch.exp(-torch.exp(torch.tanh(d(low[i])) @ d(w2) + d(w0)))
        heads_of = lambda a: a.view(t, heads, dim)
        o = plain.wkv_recurrence(heads_of(q), heads_of(k), heads_of(v), heads_of(w), d(bonus).view(heads, dim))
        whole[i] = (plain.rms(o, eps).reshape(t, n) * d(norm)) * F.silu(gate)
    state = torch.full((6, heads, dim, dim), 40.0, device=DEV)
    weights = [dev(a) for a in (w2, w0, bonus, norm)]

    def run(parts, pos, tokp, slot, lens):
        rows = torch.cat([x[i][a:a + c] for i, a, c in parts]).to(DEV)
        lw = torch.zeros(len(rows), pad(rank), device=DEV)
        lw[:, :rank] = torch.cat([low[i][a:a + c] for i, a, c in parts])
        out = torch.full((len(rows), pad(n)), 7.0, dtype=dt, device=DEV)
        ops.wkv(*rows.split(n, 1), lw, *weights, state, out, pos, tokp, slot, rank=rank, eps=eps, row_lens=lens)
        assert bool((out[:, n:] == 7.0).all())
        return out[:, :n]
    _portions(ops, cuts, {0: 4, 1: 1, 2: 0, 3: 5}, run, whole, 2e-5 if dt == F32 else 1.5e-2)
    assert bool((state[[2, 3]] == 40.0).all())


@pytest.mark.parametrize("heads,vdim,state,groups", [(6, 40, 56, 3), (4, 64, 128, 4), (2, 128, 64, 2), (5, 7, 9, 5), (1, 8, 8, 1), (80, 64, 128, 8), (3, 72, 16, 1), (2, 16, 200, 1)])
@pytest.mark.parametrize("decay", ["slow", "fast"])
@pytest.mark.parametrize("dt", [BF, F32])
def test_state_space(ops, heads, vdim, state, groups, decay, dt):
    g = torch.Generator().manual_seed(heads * vdim)
    r = lambda *s: torch.randn(*s, generator=g)
    inner, bc = heads * vdim, groups * state
    cuts = {0: [1, 2, 64, 1, 15, 33, 130], 1: [200, 1, 1, 2, 40], 2: [3, 1, 1, 17, 0, 1, 64], 3: [64, 63, 1, 128]}
    tok = {i: sum(c) for i, c in cuts.items()}
    x = {i: r(t, inner + 2 * bc).to(dt) for i, t in tok.items()}
    z = {i: r(t, pad(inner) + heads).to(dt) for i, t in tok.items()}
    bias, skip = (r(heads) - 1).to(dt), (1 + 0.5 * r(heads)).to(dt)
    a_log = ({"slow": -4.0, "fast": 3.0}[decay] + r(heads)).to(dt)
    whole = {}
    for i, t in tok.items():
        u, B, C = (d(a) for a in x[i].split([inner, bc, bc], 1))
        step = F.softplus(d(z[i][:, pad(inner):]) + d(bias), threshold=1e9)
        y = plain.ssd_recurrence(u.reshape(t, heads, vdim), B.reshape(t, groups, state), C.reshape(t, groups, state), step, torch.exp(d(a_log)), d(skip))
        whole[i] = y.reshape(t, inner) * F.silu(d(z[i][:, :inner]))
    st = torch.full((6, heads, state, vdim), 40.0, device=DEV)

    def run(parts, pos, tokp, slot, lens):
        rows, zz = (torch.cat([s[i][a:a + c] for i, a, c in parts]).to(DEV) for s in (x, z))
        out = torch.full((len(rows), pad(inner)), 7.0, dtype=dt, device=DEV)
        ops.ssd(*rows.split([inner, bc, bc], 1), zz[:, :inner], zz[:, pad(inner):], dev(bias), dev(a_log), dev(skip), st, out, pos, tokp, slot,
                groups=groups, row_lens=lens)
        assert bool((out[:, inner:] == 7.0).all())
        return out[:, :inner]
    _portions(ops, cuts, {0: 4, 1: 1, 2: 0, 3: 5}, run, whole, 2e-5 if dt == F32 else 1.5e-2)
    assert bool((st[[2, 3]] == 40.0).all())


@pytest.mark.parametrize("width,parts", [(240, 4), (8192, 8), (8192, 1), (35, 5), (64, 64), (9000, 3)])
@pytest.mark.parametrize("dt", [BF, F32])
def test_norm_in_parts(ops, width, parts, dt):
    g = torch.Generator().manual_seed(width)
    x, w = torch.randn(5, pad(width) + 8, generator=g).to(dt), torch.randn(width, generator=g).to(dt)
    x[:, :width] *= torch.rand(width, generator=g).to(dt) + 0.1
    want = plain.rms(d(x[:, :width]).view(5, parts, -1), 0.01).reshape(5, -1) * d(w)
    xd = x.to(DEV)
    ops.part_norm(xd[:, :width], dev(w), parts, 0.01)
    assert _rel(xd[:, :width], want) < (2e-6 if dt == F32 else 4e-3) and torch.equal(xd[:, width:].cpu(), x[:, width:])
