"""Mechanisms of the Komulorn design in the kernels, each against a plain fp32 / fp64 computation, on inputs that make a
mistake visible: keys that stand out at page borders and far away, routers with clear and with skewed choices, sizes of
every kind."""
import math

import pytest
import torch

import komulorn_plain as plain

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


def _i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


# ------------------------------------------------------------------------------------------------ soft-capped logits
@pytest.mark.parametrize("M", [1, 5, 64, 130, 256, 300])
@pytest.mark.parametrize("N,K", [(320, 256), (2048, 96), (101, 77)])
@pytest.mark.parametrize("dt", [BF, F32, HF])
def test_softcap_epilogue(ops, M, N, K, dt):
    g = torch.Generator().manual_seed(M + N)
    a, b = torch.randn(M, K, generator=g).to(dt), (torch.randn(K, N, generator=g) * 9 * K ** -0.5).to(dt)
    want = 7.5 * torch.tanh(a.double() @ b.double() / 7.5)
    out = torch.empty(M, N, device=DEV)
    ops.gemm(a.to(DEV), b.to(DEV), out=out, epilogue="softcap", alpha=7.5, static_b=True)
    ops.check_status()
    assert _rel(out, want) < 2e-6 and float(want.abs().max()) > 7.4


# ------------------------------------------------------------------------------------------------ rotation, biases, paged write
def _pools(ops, pages, page, kvh, dim, vdim, dt, pair):
    if pair:
        return ops.KVPair(torch.zeros(pages, page, kvh, dim, dtype=dt, device=DEV), torch.zeros(pages, page, kvh, vdim, dtype=dt, device=DEV))
    assert dim == vdim
    return torch.zeros(pages, 2, page, kvh, dim, dtype=dt, device=DEV)


def _planes(kv):
    return (kv[0], kv[1]) if isinstance(kv, tuple) else (kv[:, 0], kv[:, 1])


@pytest.mark.parametrize("dim,vdim,rot", [(64, 32, 32), (128, 128, 64), (40, 96, 12), (22, 13, 10), (16, 8, 2), (64, 64, 64), (48, 24, 0)])
@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("biased", [True, False])
@pytest.mark.parametrize("interleaved", [False, True])
def test_rotation_with_biases(ops, dim, vdim, rot, dt, biased, interleaved):
    from blitz_scale_b200.models.hybrid_config import YarnScaling
    qh, kvh, page, base = 4, 2, 16, 700.0
    y = YarnScaling(3.0, 50.0, 6.0, 1.0)
    g = torch.Generator().manual_seed(dim + vdim)
    pos = torch.tensor([0, 1, 15, 16, 31, 5, 90000])
    T = len(pos)
    pad = lambda n: (n + 7) // 8 * 8
    at = [0, pad(qh * dim), pad(qh * dim) + pad(kvh * dim)]
    x = torch.randn(T, at[2] + pad(kvh * vdim) + 16, generator=g).to(dt)
    cut = lambda t: (t[:, :qh * dim], t[:, at[1]:at[1] + kvh * dim], t[:, at[2]:at[2] + kvh * vdim])
    bias = [torch.randn(n, generator=g).to(dt) for n in (qh * dim, kvh * dim, kvh * vdim)] if biased else [None] * 3
    full = [(v.double() + (b.double() if biased else 0)).reshape(T, -1, d) for v, b, d in zip(cut(x), bias, (dim, dim, vdim))]

    def rotate(t):
        if not rot:
            return t
        freq, gain = plain.yarn_frequencies(rot, base, dict(factor=3.0, original=50.0, fast=6.0, slow=1.0))
        out = t.clone()
        for i, f in enumerate(freq):
            iu, iv = (2 * i, 2 * i + 1) if interleaved else (i, i + rot // 2)
            c, s = (torch.cos(pos.double() * f) * gain)[:, None], (torch.sin(pos.double() * f) * gain)[:, None]
            out[..., iu], out[..., iv] = t[..., iu] * c - t[..., iv] * s, t[..., iv] * c + t[..., iu] * s
        return out
    fr = ops.rope_freqs(rot, base, DEV, y.stretch(rot, base) if rot else None)
    slot = [3, 17, 40, 111, 64, -1, 0]
    dev = lambda t: None if t is None else t.to(DEV)
    kw = dict(q_heads=qh, kv_heads=kvh, dim=dim, rot_dims=rot, page_size=page, interleaved=interleaved, gain=y.gain)
    tol = 3e-6 if dt == F32 else 4e-3
    for pair in ((True, False) if dim == vdim else (True,)):
        kv = _pools(ops, 7, page, kvh, dim, vdim, dt, pair)
        xd = x.clone().to(DEV)
        q, k, v = cut(xd)
        ops.rope_store(q, k, v, pos.to(DEV, torch.int32), _i32(slot), kv, fr, **kw, q_b=dev(bias[0]), k_b=dev(bias[1]), v_b=dev(bias[2]))
        ops.check_status()
        assert _rel(q.reshape(T, qh, dim), rotate(full[0])) < tol
        K, V = (t.reshape(7 * page, kvh, -1).cpu() for t in _planes(kv))
        kr = rotate(full[1])
        for t, s in enumerate(slot):
            if s >= 0:
                assert _rel(K[s], kr[t]) < tol and _rel(V[s], full[2][t]) < tol
        assert sum(bool(r.any()) for r in K) == sum(bool(r.any()) for r in V) == len(slot) - 1
        # queries alone: the cache stays as it is
        before, xd = [t.clone() for t in _planes(kv)], x.clone().to(DEV)
        ops.rope_store(cut(xd)[0], None, None, pos.to(DEV, torch.int32), _i32(slot), kv, fr, **kw, q_b=dev(bias[0]))
        assert _rel(cut(xd)[0].reshape(T, qh, dim), rotate(full[0])) < tol
        assert all(torch.equal(a, b) for a, b in zip(before, _planes(kv)))
        assert torch.equal(xd[:, qh * dim:].cpu(), x[:, qh * dim:])


# ------------------------------------------------------------------------------------------------ attention
# (heads, kv heads, dim, vdim, page, gate)
ATT = [(4, 2, 64, 32, 16, True), (12, 1, 128, 128, 64, True), (5, 5, 40, 96, 16, True), (10, 5, 128, 48, 64, False), (9, 3, 22, 13, 16, True),
       (22, 2, 64, 64, 32, True), (6, 1, 96, 8, 8, True), (1, 1, 8, 128, 128, True), (16, 1, 72, 120, 64, True), (3, 1, 200, 300, 16, True)]


@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("case", ATT)
def test_attention_of_unequal_sizes(ops, case, dt):
    """Prompts, portions behind any prefix, and single tokens with and without key splits.  A few keys stand out (the first
    ones, those at page and block borders, the last): one that is missed or seen too early decides the output."""
    H, G, d, dv, page, gated = case
    lens, q_lens = [700, 65, 1, 300, 389], [700, 65, 1, 2, 260]
    g = torch.Generator().manual_seed(H * d + dv)
    scale = 0.8 * d ** -0.5
    npages = [-(-n // page) for n in lens]
    perm = torch.randperm(sum(npages), generator=g).tolist()
    kv = _pools(ops, sum(npages), page, G, d, dv, dt, d != dv)
    K, V = _planes(kv)
    want, qs, gates, at = [], [], [], 0
    for n, ql, np_ in zip(lens, q_lens, npages):
        k, v = torch.randn(n, G, d, generator=g), torch.randn(n, G, dv, generator=g).to(dt)
        u = torch.randn(d, generator=g)
        u = u / u.norm() * d ** 0.5
        loud = sorted({p for p in (0, 1, page - 1, page, 63, 64, 127, 128, 129, 255, 256, n // 2, n - 2, n - 1) if 0 <= p < n})
        k[loud] = k[loud] * 0.3 + 0.9 * u
        k = k.to(dt)
        q = (0.5 * torch.randn(n, H, d, generator=g) + u).to(dt)[n - ql:]
        z = (2 * torch.randn(ql, H, generator=g)).to(dt)
        for i in range(np_):
            part = slice(i * page, min(n, (i + 1) * page))
            K[perm[at + i], :part.stop - part.start] = k[part].to(DEV)
            V[perm[at + i], :part.stop - part.start] = v[part].to(DEV)
        at += np_
        o = torch.zeros(ql, H, dv, dtype=torch.float64)
        see = torch.arange(n)[None] <= torch.arange(n - ql, n)[:, None]
        for h in range(H):
            s = (q[:, h].double() @ k[:, h // (H // G)].double().T * scale).masked_fill(~see, -math.inf)
            o[:, h] = torch.softmax(s, -1) @ v[:, h // (H // G)].double()
        want.append(o * torch.sigmoid(z.double())[..., None] if gated else o)
        qs.append(q)
        gates.append(z)
    T = sum(q_lens)
    pad = lambda n: (n + 7) // 8 * 8
    proj = torch.zeros(T, pad(H * d) + pad(H) + 8, dtype=dt, device=DEV)       # queries and gates as columns of one projection
    q, gate = proj[:, :H * d], proj[:, pad(H * d):pad(H * d) + H]
    q.copy_(torch.cat(qs).reshape(T, -1))
    gate.copy_(torch.cat(gates))
    if not gated:
        gate = None
    pos = _i32([p for n, ql in zip(lens, q_lens) for p in range(n - ql, n)])
    tokp, indptr = (_i32([sum(x[:i]) for i in range(len(lens) + 1)]) for x in (q_lens, npages))
    indices, last = _i32(perm), _i32([n - (u - 1) * page for n, u in zip(lens, npages)])
    tol = 8e-6 if dt == F32 else 2.4e-2

    def check(out, rows, what):
        ops.check_status()
        for i, (w, r) in enumerate(zip(want, rows)):
            got, w = out[r].reshape(-1, H, dv).double().cpu(), w[-len(r):]
            err = (got - w).flatten(1).norm(dim=1) / w.flatten(1).norm(dim=1).clamp_min(1e-3)
            assert float(err.max()) < tol, (what, i, int(err.argmax()), float(err.max()))
    all_rows = [list(range(int(tokp[i]), int(tokp[i + 1]))) for i in range(len(lens))]
    buf = torch.full((T, pad(H * dv) + 8), 7.0, dtype=dt, device=DEV)
    ops.attn_ragged(q, kv, pos, tokp, indptr, indices, buf, q_heads=H, kv_heads=G, dim=d, page_size=page, scale=scale, gate=gate)
    check(buf[:, :H * dv], all_rows, "general")
    assert bool((buf[:, H * dv:] == 7.0).all())
    if not ops.attn_tensor_core(q, H, G, d, page, dv):
        assert dt == F32 or d % 8 or dv % 8 or max(d, dv) > 128
        return
    buf.fill_(7.0)
    work = ops.prefill_work_list(q_lens, lens, page, DEV)
    kw = dict(q_heads=H, kv_heads=G, head_dim=d, page_size=page, sm_scale=scale)
    ops.attn_prefill_paged(q, kv, indices, work, out=buf, gate=gate, **kw)
    check(buf[:, :H * dv], all_rows, "prefill")
    assert bool((buf[:, H * dv:] == 7.0).all())
    rows = [r[-1] for r in all_rows]
    for splits in (1, 2, 8):
        o = torch.full((len(lens), pad(H * dv) + 8), 7.0, dtype=dt, device=DEV)
        ops.attn_decode(q[rows], kv, indices, indptr, last, num_splits=splits, gate=gate[rows] if gated else None, out=o, **kw)
        check(o[:, :H * dv], [[i] for i in range(len(lens))], ("decode", splits))
        assert bool((o[:, H * dv:] == 7.0).all())


# ------------------------------------------------------------------------------------------------ experts
def _experts(T, E, top, H, ff, sff, dt, seed, skew=0.0):
    g = torch.Generator().manual_seed(seed)
    r = lambda *s: torch.randn(*s, generator=g)
    h = r(T, H).to(dt)
    w = {f"e{e}.{n}": (r(*s) * s[1] ** -0.5).to(dt) for e in range(E) for n, s in (("up", (ff, H)), ("down", (H, ff)))}
    if sff:
        w.update({"shared.up": (r(sff, H) * H ** -0.5).to(dt), "shared.down": (r(H, sff) * sff ** -0.5).to(dt)})
    z = 1.5 * r(T, E + bool(sff)) + skew * torch.linspace(2, -2, E + bool(sff))
    return h, w, z


def _run_experts(ops, h, w, z, E, top, sff, plan, bn=0, tile_rows=128, fetch=0, **how):
    dev = lambda n: torch.stack([w[f"e{e}.{n}"].T.contiguous() for e in range(E)]).to(DEV)
    up, down = dev("up"), dev("down")
    s_up, s_down = (w[f"shared.{n}"].T.contiguous().to(DEV) if sff else None for n in ("up", "down"))
    T, H = h.shape
    ops.moe_route(z.to(DEV), plan, tile_rows=tile_rows, **how)
    act = torch.full((plan.rows, max(up.shape[2], sff)), math.nan, dtype=h.dtype, device=DEV)      # nothing unwritten may be read
    y = torch.full((plan.rows, H), math.nan, dtype=h.dtype, device=DEV)
    ops.gemm_grouped(h.to(DEV), up, plan, act, shared=s_up, gather=True, act="relu2", factors=True, bn=bn, fetch=fetch)
    ops.gemm_grouped(act, down, plan, y, shared=s_down, bn=bn)
    x = torch.ones(T, H, device=DEV)
    out = torch.empty(T, H, dtype=h.dtype, device=DEV)
    gain = torch.full((H,), 0.5, dtype=h.dtype, device=DEV)
    ops.stream_norm(x, gain, 1e-5, out, add=y, add_rows=plan.place)
    ops.check_status()
    assert _rel(out, 0.5 * x.cpu().double() / (x.cpu().double().square().mean(-1, keepdim=True) + 1e-5).sqrt()) < (1e-6 if h.dtype == F32 else 4e-3)
    return x.cpu() - 1


def _want_experts(h, w, z, E, top, sff):
    """The oracle's experts with a router that reads the logits themselves."""
    hd = torch.cat([h.double(), z.double()], 1)
    H = h.shape[1]
    wide = lambda t: torch.cat([t.double(), torch.zeros(t.shape[0], z.shape[1], dtype=torch.float64)], 1)
    ws = {n: wide(t) if n.endswith("up") else torch.cat([t.double(), torch.zeros(z.shape[1], t.shape[1], dtype=torch.float64)], 0) for n, t in w.items()}
    pick = lambda a, b: torch.cat([torch.zeros(b - a, H + a, dtype=torch.float64), torch.eye(b - a, dtype=torch.float64),
                                   torch.zeros(b - a, z.shape[1] - b, dtype=torch.float64)], 1)
    ws["router"] = pick(0, E)
    if sff:
        ws["shared.sg"] = pick(E, E + 1)
    out = plain.experts(hd, ws.__getitem__, {"router": {"experts": E, "top": top}, "shared": {"ff": sff} if sff else None})
    return out[:, :H]


@pytest.mark.parametrize("T", [1, 7, 64, 300])
@pytest.mark.parametrize("E,top,H,ff,sff,skew", [(6, 2, 128, 64, 136, 0.0), (20, 1, 200, 104, 64, 3.0), (3, 3, 64, 8, 0, 0.0), (130, 5, 72, 40, 48, 1.0),
                                                 (1, 1, 328, 264, 8, 0.0)])
@pytest.mark.parametrize("dt", [BF, HF])
def test_experts_on_the_tensor_cores(ops, T, E, top, H, ff, sff, skew, dt):
    h, w, z = _experts(T, E, top, H, ff, sff, dt, T + E, skew)
    want = _want_experts(h, w, z, E, top, sff)
    plan = ops.ExpertPlan(300, E, top, bool(sff), DEV)
    for bn, fetch in ((0, 0), (64, 1), (128, 1), (256, 1), (64, 2), (128, 2), (256, 2)):
        got = _run_experts(ops, h, w, z, E, top, sff, plan, bn, fetch=fetch)
        assert _rel(got, want) < (8e-3 if dt == BF else 1e-3), (bn, fetch)


@pytest.mark.parametrize("T,E,top,H,ff,sff", [(1, 5, 2, 33, 21, 7), (130, 5, 3, 121, 51, 30), (90, 9, 1, 64, 72, 136), (200, 2, 2, 40, 10, 0)])
@pytest.mark.parametrize("dt", [F32, BF])
def test_experts_of_any_size(ops, T, E, top, H, ff, sff, dt):
    h, w, z = _experts(T, E, top, H, ff, sff, dt, T + E)
    plan = ops.ExpertPlan(T, E, top, bool(sff), DEV)
    got = _run_experts(ops, h, w, z, E, top, sff, plan, tile_rows=64)
    assert _rel(got, _want_experts(h, w, z, E, top, sff)) < (2e-6 if dt == F32 else 8e-3)


@pytest.mark.parametrize("T,E,top,shared", [(1, 1, 1, 1), (5, 7, 7, 1), (3000, 3, 1, 0), (2000, 1000, 8, 1), (257, 64, 6, 1), (33, 40, 32, 0)])
def test_router(ops, T, E, top, shared):
    """Choices, weights, sorted rows and work list; twice on the same buffers (the counters are cleared by the kernel)."""
    g = torch.Generator().manual_seed(T)
    plan = ops.ExpertPlan(T + 3, E, top, bool(shared), DEV)
    for rnd, (renorm, on_input) in enumerate(((False, True), (True, False))):
        z = 4 * torch.randn(T, E + shared + 5, generator=g)
        if rnd:
            z[:, 1:] -= 30.0                       # everyone's first choice is expert 0; scores near 0 and near 1
        ops.moe_route(z.to(DEV), plan, renormalize=renorm, weight_on_input=on_input, tile_rows=128)
        ops.check_status()
        s = torch.sigmoid(z[:, :E].double())
        val, idx = torch.topk(z[:, :E], top)       # by the logits: scores of 1 - 1e-9 tie in fp32
        wt = s.gather(1, idx)
        if renorm:
            wt = wt / wt.sum(1, keepdim=True)
        place, src = plan.place.cpu().long(), plan.src.cpu().long()
        fac, tiles = plan.factors.cpu().double(), plan._tiles.cpu()[:int(plan.num_tiles)].tolist()
        per = top + shared
        assert sorted(place.flatten().tolist()) == list(range(T * per)) and torch.equal(src[place], torch.arange(T)[:, None].expand(T, per))
        counts = torch.bincount(idx.flatten(), minlength=E)
        begin = torch.cumsum(counts, 0) - counts
        owner = torch.searchsorted(torch.cumsum(counts, 0), place[:, :top].contiguous(), right=True)
        assert torch.equal(owner.sort(1).values, idx.sort(1).values)
        got = torch.zeros(T, E, dtype=torch.float64).scatter_(1, owner, fac[place[:, :top], 0 if on_input else 1])
        assert torch.allclose(got, torch.zeros(T, E, dtype=torch.float64).scatter_(1, idx, wt), rtol=1e-5, atol=1e-30)
        assert bool((fac[place[:, :top], 1 if on_input else 0] == 1).all())
        if shared:
            assert torch.equal(place[:, top], T * top + torch.arange(T))
            assert torch.allclose(fac[T * top:T * per, 1], torch.sigmoid(z[:, E].double()), rtol=1e-6) and bool((fac[T * top:T * per, 0] == 1).all())
        want = [[e, int(begin[e]) + 128 * i, min(128, int(counts[e]) - 128 * i), 0] for e in range(E) for i in range(-(-int(counts[e]) // 128))]
        assert tiles == want
        assert not plan.counters[:E + 1].any()


@pytest.mark.parametrize("H", [7, 64, 250, 4096, 9000])
@pytest.mark.parametrize("dt", [BF, F32])
def test_stream_norm_adds_rows(ops, H, dt):
    g = torch.Generator().manual_seed(H)
    T, n = 5, 3
    x, y, w = torch.randn(T, H, generator=g), torch.randn(20, H, generator=g).to(dt), torch.randn(H, generator=g).to(dt)
    rows = torch.randint(0, 20, (T, n), generator=g)
    want = x.double() + y.double()[rows].sum(1)
    xd, out = x.to(DEV), torch.empty(T, H, dtype=dt, device=DEV)
    ops.stream_norm(xd, w.to(DEV), 1e-3, out, add=y.to(DEV), add_rows=rows.to(DEV, torch.int32))
    assert _rel(xd, want) < 1e-6 and _rel(out, plain.rms_norm(want, w.double(), 1e-3)) < (1e-6 if dt == F32 else 4e-3)
    xd = x.to(DEV)
    ops.stream_norm(xd, None, 0.0, None, add=y.to(DEV), add_rows=rows.to(DEV, torch.int32))
    assert _rel(xd, want) < 1e-6
    ops.check_status()
