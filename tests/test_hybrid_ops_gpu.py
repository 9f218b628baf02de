"""Kernels of the hybrid models, each against a plain fp32 / fp64 computation of the same mechanism, on inputs that make a
mistake visible: single keys that stand out placed at and around every edge, sizes of every kind."""
import math

import pytest
import torch

import fafudra_plain as plain

pytestmark = pytest.mark.gpu

DEV = "cuda"
BF, F32, HF = torch.bfloat16, torch.float32, torch.float16


@pytest.fixture(scope="module")
def ops():
    torch.cuda.set_device(0)
    from blitz_scale_b200 import ops as o
    return o


def _rel(a, b):
    return float((a.float().cpu() - b.float().cpu()).norm() / b.float().cpu().norm())


def _i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


# ------------------------------------------------------------------------------------------------ matrix products
@pytest.mark.parametrize("M", [1, 5, 64, 130, 256, 300, 1000])
@pytest.mark.parametrize("N,K", [(320, 256), (64, 2048), (1024, 96), (2048, 512)])
@pytest.mark.parametrize("dt", [BF, HF])
def test_fp32_outputs_of_the_tensor_core_products(ops, M, N, K, dt):
    g = torch.Generator().manual_seed(M + N)
    a, b = torch.randn(M, K, generator=g).to(dt), (torch.randn(K, N, generator=g) * K ** -0.5).to(dt)
    x = torch.randn(M, N, generator=g)
    want = a.double() @ b.double()
    ad, bd = a.to(DEV), b.to(DEV)
    out = torch.empty(M, N, device=DEV)
    ops.gemm(ad, bd, out=out, static_b=True)
    assert _rel(out, want) < 2e-6
    acc = x.to(DEV)
    ops.gemm(ad, bd, out=acc, epilogue="axpy", alpha=0.7)
    assert _rel(acc, x.double() + 0.7 * want) < 2e-6
    ops.check_status()


@pytest.mark.parametrize("M,N,K", [(1, 7, 5), (33, 100, 121), (70, 64, 64), (129, 203, 90)])
@pytest.mark.parametrize("dt", [F32, BF])
def test_products_of_any_size(ops, M, N, K, dt):
    g = torch.Generator().manual_seed(K)
    a, b = torch.randn(M, K, generator=g).to(dt), (torch.randn(K, 2 * N, generator=g) * K ** -0.5).to(dt)
    tol = 2e-6 if dt == F32 else 4e-3
    gate, up = a.double() @ b[:, :N].double(), a.double() @ b[:, N:].double()
    assert _rel(ops.gemm(a.to(DEV), b[:, :N].contiguous().to(DEV)), gate) < tol
    assert _rel(ops.gemm(a.to(DEV), b.to(DEV), epilogue="silu_mul"), plain.silu(gate) * up) < tol
    acc = torch.ones(M, N, device=DEV)
    ops.gemm(a.to(DEV), b[:, :N].contiguous().to(DEV), out=acc, epilogue="axpy", alpha=-2.0)
    assert _rel(acc, 1 - 2 * gate) < 2e-6


@pytest.mark.parametrize("M", [1, 40, 300])
@pytest.mark.parametrize("groups,n", [(3, 64), (2, 128), (5, 18), (1, 64), (4, 80)])
@pytest.mark.parametrize("dt", [BF, F32])
def test_block_diagonal_products(ops, M, groups, n, dt):
    g = torch.Generator().manual_seed(n)
    a = torch.randn(M, groups * n, generator=g).to(dt)
    b = (torch.randn(groups * n, 2 * n, generator=g) * n ** -0.5).to(dt)
    want = torch.cat([a[:, i * n:(i + 1) * n].double() @ b[i * n:(i + 1) * n].double() for i in range(groups)], 1)
    out = torch.empty(M, groups * 2 * n, device=DEV)
    ops.gemm(a.to(DEV), b.to(DEV), out=out, groups=groups)
    ops.check_status()
    assert _rel(out, want) < 2e-6


# ------------------------------------------------------------------------------------------------ stream and norm
@pytest.mark.parametrize("H", [7, 64, 250, 4096, 9000])
@pytest.mark.parametrize("dt", [BF, F32])
def test_stream_norm(ops, H, dt):
    g = torch.Generator().manual_seed(H)
    T, V = 5, 11
    emb, step, w = (torch.randn(*s, generator=g).to(dt) for s in ((V, H), (H,), (H,)))
    ids = torch.tensor([0, 10, 3, 3, 7])
    x = torch.randn(T, H, generator=g)
    norm = lambda s: plain.rms_norm(s.double(), 1e-3) * (1 + w.double())
    tol = 1e-6 if dt == F32 else 4e-3
    for init, add, with_step in ((True, False, False), (True, False, True), (False, True, True), (False, False, True), (False, False, False)):
        want = emb[ids].float() if init else x + (emb[ids].float() if add else 0)
        if with_step:
            want = want + step.float()
        xd, out = x.to(DEV), torch.empty(T, H, dtype=dt, device=DEV)
        ops.stream_norm(xd, w.to(DEV), 1e-3, out, w_offset=1.0, ids=ids.to(DEV, torch.int32), embed=emb.to(DEV), init=init,
                        add_embed=add, step=step.to(DEV) if with_step else None)
        assert torch.allclose(xd.cpu(), want, rtol=1e-6, atol=1e-6) and _rel(out, norm(want)) < tol
    out = torch.empty(2, H, dtype=dt, device=DEV)
    ops.stream_norm(x.to(DEV), w.to(DEV), 1e-3, out, w_offset=1.0, rows=_i32([5, 2]), row_offset=-1)
    assert _rel(out, norm(x[[4, 1]])) < tol
    ops.check_status()
    # a token id outside the vocabulary is reported, not read
    ops.stream_norm(x.to(DEV), w.to(DEV), 1e-3, torch.empty(T, H, dtype=dt, device=DEV), ids=_i32([0, V, 1, 2, 3]), embed=emb.to(DEV), init=True)
    with pytest.raises(RuntimeError):
        ops.check_status()


# ------------------------------------------------------------------------------------------------ attention
class Pages:
    """Sequences on shuffled pages of one layer's pool."""

    def __init__(self, lens, page, kvh, dim, dt):
        self.page, self.npages = page, [(n + page - 1) // page for n in lens]
        total = sum(self.npages)
        perm = torch.randperm(total, generator=torch.Generator().manual_seed(total)).tolist()
        self.kv = torch.zeros(total, 2, page, kvh, dim, dtype=dt, device=DEV)
        self.table, at = [], 0
        for n in self.npages:
            self.table.append(perm[at:at + n])
            at += n
        self.indptr = _i32([sum(self.npages[:i]) for i in range(len(lens) + 1)])
        self.indices = _i32([p for t in self.table for p in t])
        self.last = _i32([n - (u - 1) * page for n, u in zip(lens, self.npages)])

    def slot(self, s, pos):
        return self.table[s][pos // self.page] * self.page + pos % self.page

    def put(self, s, k, v):
        for i in range(k.shape[0]):
            self.kv[self.table[s][i // self.page], 0, i % self.page] = k[i]
            self.kv[self.table[s][i // self.page], 1, i % self.page] = v[i]


@pytest.mark.parametrize("interleaved", [True, False])
@pytest.mark.parametrize("dim,rot", [(64, 64), (64, 20), (20, 12), (9, 0), (9, 4)])
@pytest.mark.parametrize("dt", [BF, F32])
def test_rotation_and_paged_write(ops, dim, rot, interleaved, dt):
    qh, kvh, page = 4, 2, 16
    g = torch.Generator().manual_seed(dim + rot)
    pos = torch.tensor([0, 1, 15, 16, 31, 5, 100000])
    T = len(pos)
    row = (qh + 2 * kvh) * dim + 3 * (dim % 2 == 0) * 2       # a pitch of its own
    x = torch.randn(T, row, generator=g).to(dt)
    pages = Pages([112], page, kvh, dim, dt)
    slot = [pages.slot(0, p % 112) for p in pos.tolist()]
    slot[5] = -1
    fr = ops.rope_freqs(rot, 500.0, DEV)
    rotate = lambda t: plain.rotate_pairs(t.double(), pos, rot, 500.0, not interleaved)
    q, k, v = x[:, :qh * dim], x[:, qh * dim:(qh + kvh) * dim], x[:, (qh + kvh) * dim:(qh + 2 * kvh) * dim]
    for own_v in (True, False):
        xd = x.clone().to(DEV)
        pages.kv.zero_()
        cut = lambda a, b: xd[:, a * dim:b * dim]
        ops.rope_store(cut(0, qh), cut(qh, qh + kvh), cut(qh + kvh, qh + 2 * kvh) if own_v else None, pos.to(DEV, torch.int32),
                       _i32(slot), pages.kv, fr, q_heads=qh, kv_heads=kvh, dim=dim, rot_dims=rot, page_size=page, interleaved=interleaved)
        ops.check_status()
        tol = 2e-6 if dt == F32 else 4e-3
        assert _rel(cut(0, qh), rotate(q.reshape(T, qh, dim)).reshape(T, -1)) < tol
        kr = rotate(k.reshape(T, kvh, dim))
        flat = pages.kv.cpu()
        for t in range(T):
            if slot[t] >= 0:
                at = flat[slot[t] // page, :, slot[t] % page]
                assert _rel(at[0], kr[t]) < tol
                assert torch.equal(at[1], (v if own_v else k).reshape(T, kvh, dim)[t])
        written = {s for s in slot if s >= 0}
        assert sum(bool(flat[s // page, :, s % page].any()) for s in range(112)) == len(written)


def _dense(q, k, v, pos, window, first, cap, sink, scale):
    """q [T, H, d] at positions pos; k, v [n, G, d]; fp64."""
    T, H, d = q.shape
    out = torch.zeros(T, H, d, dtype=torch.float64)
    g = H // k.shape[1]
    j = torch.arange(k.shape[0])
    for h in range(H):
        s = q[:, h].double() @ k[:, h // g].double().T * scale
        if cap:
            s = cap * torch.tanh(s / cap)
        i = pos[:, None]
        see = (j[None] <= i) & ((i - j[None] < window) | (j[None] < first) if window else torch.ones_like(s, dtype=torch.bool))
        s = s.masked_fill(~see, -math.inf)
        m = s.max(-1).values
        if sink is not None:
            m = torch.maximum(m, sink[h].double())
        e = torch.exp(s - m[:, None])
        den = e.sum(-1) + (torch.exp(sink[h].double() - m) if sink is not None else 0)
        out[:, h] = (e / den[:, None]) @ v[:, h // g].double()
    return out


# (heads, kv heads, dim, page, window, kept, cap, sink)
ATT = [(8, 1, 64, 64, 90, 7, 25.0, True), (8, 2, 128, 16, 100, 3, 0.0, True), (4, 4, 64, 16, 1, 1, 10.0, False),
       (4, 2, 128, 64, 130, 0, 5.0, True), (8, 4, 64, 32, 500, 200, 40.0, True), (4, 1, 128, 16, 0, 0, 20.0, True),
       (6, 2, 20, 16, 33, 5, 8.0, True), (4, 2, 64, 16, 70, 130, 25.0, True)]


@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("case", ATT)
def test_windowed_attention(ops, case, dt):
    """Prompts and portions (any prefix) and single tokens.  Keys that stand out sit just inside and just outside the
    window, at page borders and among the first tokens: one that is missed or seen too long decides the output."""
    H, G, d, page, window, first, cap, with_sink = case
    lens, q_lens = [700, 65, 1, 300, 389], [700, 65, 1, 2, 260]
    g = torch.Generator().manual_seed(H * d + window)
    scale = d ** -0.5
    pages = Pages(lens, page, G, d, dt)
    sink = (1.0 + torch.randn(H, generator=g)).to(dt) if with_sink else None
    ks, vs, qs = [], [], []
    for n in lens:
        k, v = torch.randn(n, G, d, generator=g), torch.randn(n, G, d, generator=g)
        u = torch.randn(d, generator=g)
        u = u / u.norm() * d ** 0.5
        loud = sorted({p for p in (0, 1, first - 1, first, first + 1, page - 1, page, n - window - 1, n - window, n - window + 1, n - 2,
                                   63, 64, 127, 128, 129, n // 2) if 0 <= p < n})
        k[loud] = k[loud] * 0.3 + 0.8 * u            # about 0.8 sqrt(d) in score against a query along u
        ks.append(k.to(dt))
        vs.append(v.to(dt))
        q = 0.5 * torch.randn(n, H, d, generator=g) + u
        qs.append(q.to(dt))
        pages.put(len(ks) - 1, ks[-1].to(DEV), vs[-1].to(DEV))
    want = [_dense(qs[s][n - ql:], ks[s], vs[s], torch.arange(n - ql, n), window, first, cap, sink, scale)
            for s, (n, ql) in enumerate(zip(lens, q_lens))]
    T = sum(q_lens)
    pos = _i32([p for n, ql in zip(lens, q_lens) for p in range(n - ql, n)])
    tokp = _i32([sum(q_lens[:i]) for i in range(len(lens) + 1)])
    q = torch.cat([qs[s][n - ql:] for s, (n, ql) in enumerate(zip(lens, q_lens))]).reshape(T, H * d).to(DEV)
    wide = torch.zeros(T, H * d + 24, dtype=dt, device=DEV)      # query columns of a wider projection
    wide[:, :H * d] = q
    q = wide[:, :H * d]
    kw = dict(window=window, keep_first=first, softcap=cap, sink=sink.to(DEV) if with_sink else None)
    tol = 3e-6 if dt == F32 else 8e-3

    def check(out, what):
        ops.check_status()
        at = 0
        for w, ql in zip(want, q_lens):
            got = out[at:at + ql].reshape(ql, H, d).double().cpu()
            err = (got - w).flatten(1).norm(dim=1) / w.flatten(1).norm(dim=1).clamp_min(1e-3)
            assert float(err.max()) < (tol if dt == F32 else 3 * tol), (what, ql, int(err.argmax()), float(err.max()))
            at += ql
    out = torch.full((T, H * d), 7.0, dtype=dt, device=DEV)
    ops.attn_ragged(q, pages.kv, pos, tokp, pages.indptr, pages.indices, out, q_heads=H, kv_heads=G, dim=d, page_size=page, scale=scale, **kw)
    check(out, "general")
    if not ops.attn_tensor_core(q, H, G, d, page):
        assert dt == F32 or d not in (64, 128)
        return
    out = torch.full((T, H * d), 7.0, dtype=dt, device=DEV)
    work = ops.prefill_work_list(q_lens, lens, page, DEV)
    ops.attn_prefill_paged(q, pages.kv, pages.indices, work, q_heads=H, kv_heads=G, head_dim=d, page_size=page, out=out, sm_scale=scale, **kw)
    check(out, "prefill")
    rows = torch.stack([q[int(tokp[i + 1]) - 1] for i in range(len(lens))])
    last = [w[-1:] for w in want]
    for splits in (1, 2, 8):
        o = ops.attn_decode(rows, pages.kv, pages.indices, pages.indptr, pages.last, q_heads=H, kv_heads=G, head_dim=d,
                            page_size=page, num_splits=splits, sm_scale=scale, **kw)
        ops.check_status()
        for i, w in enumerate(last):
            err = _rel(o[i].view(1, H, d), w)
            assert err < tol, ("decode", splits, lens[i], err)


# ------------------------------------------------------------------------------------------------ recurrences
def _cut(n, sizes):
    out, at, i = [], 0, 0
    while at < n:
        s = min(sizes[i % len(sizes)], n - at)
        out.append((at, at + s))
        at += s
        i += 1
    return out


@pytest.mark.parametrize("sizes", [[1000], [1], [2, 5, 64, 63, 1, 17], [128, 1, 30]])
@pytest.mark.parametrize("heads,dim,vdim,rank,tau", [(2, 64, 64, 16, 16.0), (3, 32, 128, 4, 1.0), (2, 12, 22, 5, 2.0), (1, 128, 256, 16, 8.0),
                                                      (16, 48, 200, 8, 1.0), (13, 128, 256, 16, 16.0)])
@pytest.mark.parametrize("dt", [BF, F32])
def test_gated_linear_attention(ops, heads, dim, vdim, rank, tau, sizes, dt):
    """Three sequences cut alike, on scattered state slots that hold garbage before; decays from nearly none to nearly
    total, with channels of both kinds in one head."""
    lens = [150, 33, 1] if sizes != [1] else [70, 33, 1]
    g = torch.Generator().manual_seed(dim + vdim)
    hk, hv, eps = heads * dim, heads * vdim, 1e-5
    r = lambda *s: torch.randn(*s, generator=g)
    w = {"a2": (3.0 * r(rank, hk) * rank ** -0.5).to(dt), "a2_b": (4.0 * r(hk)).to(dt), "norm": (1 + 0.3 * r(vdim)).to(dt)}
    seqs = [{"q": r(n, hk), "k": r(n, hk) * dim ** -0.25, "v": r(n, hv), "g": r(n, hv), "low": r(n, rank)} for n in lens]
    seqs = [{n: t.to(dt) for n, t in s.items()} for s in seqs]
    ident = lambda n: torch.eye(n, dtype=torch.float64)
    want = []
    for s in seqs:           # the oracle's mixer with identity projections on stacked inputs
        d = {n: t.double() for n, t in s.items()}
        h = torch.cat([d[n] for n in ("q", "k", "v", "g", "low")], 1)
        sel, at = {}, 0
        for n, wd in (("q", hk), ("k", hk), ("v", hv), ("g", hv), ("a1", rank)):
            sel[n] = torch.zeros(wd, h.shape[1], dtype=torch.float64)
            sel[n][:, at:at + wd] = ident(wd)
            at += wd
        sel.update({"a2": w["a2"].double().T, "a2.b": w["a2_b"].double(), "norm": w["norm"].double(), "o": ident(hv)})
        want.append(plain.gla(h, sel.__getitem__, dict(heads=heads, dim=dim, vdim=vdim, tau=tau), eps))
    slots = [4, 0, 2]
    state = torch.full((5, heads, dim, vdim), 1e3, device=DEV)
    pad = lambda n: (n + 7) // 8 * 8
    widths = [("q", hk), ("k", hk), ("v", hv), ("g", hv), ("low", rank)]
    got = [[] for _ in lens]
    for lo, hi in _cut(max(lens), sizes):
        rows = [i for i, n in enumerate(lens) if n > lo]
        cnt = [min(hi, lens[i]) - lo for i in rows]
        T = sum(cnt)
        x = torch.zeros(T, sum(pad(n) for _, n in widths), dtype=dt, device=DEV)
        parts, at = {}, 0
        for n, wd in widths:
            parts[n] = x[:, at:at + wd]
            parts[n].copy_(torch.cat([seqs[i][n][lo:lo + c] for i, c in zip(rows, cnt)]))
            at += pad(wd)
        out = torch.zeros(T, pad(hv), dtype=dt, device=DEV)
        pos = _i32([p for c in cnt for p in range(lo, lo + c)])
        indptr = None if all(c == 1 for c in cnt) else _i32([sum(cnt[:i]) for i in range(len(cnt) + 1)])
        ops.gla(parts["q"], parts["k"], parts["v"], parts["g"], parts["low"], w["a2"].to(DEV), w["a2_b"].to(DEV), w["norm"].to(DEV),
                state, out, pos, indptr, _i32([slots[i] for i in rows]), rank=rank, tau=tau, eps=eps, row_lens=cnt)
        ops.check_status()
        at = 0
        for i, c in zip(rows, cnt):
            got[i].append(out[at:at + c, :hv].float().cpu())
            at += c
    for i, wnt in enumerate(want):
        o = torch.cat(got[i])
        err = (o - wnt.float()).norm(dim=1) / wnt.float().norm(dim=1)
        tol = 3e-5 if dt == F32 else 1.2e-2
        # an output that all but cancels before its norm is ill-conditioned
        assert float(err.median()) < tol / 2 and int((err > tol).sum()) <= len(err) // 25, (i, int(err.argmax()), float(err.max()), float(err.median()))
    assert float(state[1].min()) == 1e3 == float(state[3].max())          # other slots untouched


@pytest.mark.parametrize("sizes", [[1000], [1], [2, 5, 64, 63, 1, 17], [128, 1, 30]])
@pytest.mark.parametrize("width,blocks,taps", [(128, 2, 4), (90, 5, 3), (64, 1, 1), (200, 2, 7)])
@pytest.mark.parametrize("dt", [BF, F32])
def test_gated_linear_recurrence(ops, width, blocks, taps, sizes, dt):
    lens = [150, 33, 1] if sizes != [1] else [70, 33, 1]
    g = torch.Generator().manual_seed(width)
    r = lambda *s: torch.randn(*s, generator=g)
    b = width // blocks
    w = {"y.b": 0.3 * r(width), "x.b": 0.3 * r(width), "conv": 0.6 * r(width, taps), "conv.b": 0.3 * r(width),
         "ra": r(blocks, b, b) * b ** -0.5, "ri": r(blocks, b, b) * b ** -0.5, "ra.b": r(blocks, b), "ri.b": r(blocks, b), "lam": -4 + 3 * r(width)}
    w = {n: t.to(dt) for n, t in w.items()}
    xs = [(r(n, width).to(dt), r(n, width).to(dt)) for n in lens]       # y, x projections
    want = []
    for y, x in xs:
        e = torch.eye(width, dtype=torch.float64)
        z = torch.zeros(width, width, dtype=torch.float64)
        d = {n: t.double() for n, t in w.items()}
        d.update(y=torch.cat([e, z], 1), x=torch.cat([z, e], 1), o=e)
        want.append(plain.rglru(torch.cat([y, x], 1).double(), d.__getitem__, dict(width=width, blocks=blocks, conv=taps)))
    dev = {n: t.to(DEV) for n, t in w.items()}
    gates_w = torch.cat([torch.cat([w["ra"][i].T, w["ri"][i].T], 1) for i in range(blocks)]).contiguous().to(DEV)
    gate_b = torch.stack([w["ra.b"], w["ri.b"]], 1).reshape(-1).contiguous().to(DEV)
    conv = w["conv"].T.contiguous().to(DEV)
    slots = [4, 0, 2]
    state = torch.full((5, width), 1e3, device=DEV)
    hist = torch.full((5, taps - 1, width), 1e3, device=DEV).to(dt)
    got = [[] for _ in lens]
    for lo, hi in _cut(max(lens), sizes):
        rows = [i for i, n in enumerate(lens) if n > lo]
        cnt = [min(hi, lens[i]) - lo for i in rows]
        T = sum(cnt)
        proj = torch.cat([torch.cat([xs[i][0][lo:lo + c], xs[i][1][lo:lo + c]], 1) for i, c in zip(rows, cnt)]).to(DEV)
        y, x = proj[:, :width], proj[:, width:]
        u, gates, out = torch.empty(T, width, dtype=dt, device=DEV), torch.empty(T, 2 * width, device=DEV), torch.empty(T, width, dtype=dt, device=DEV)
        pos = _i32([p for c in cnt for p in range(lo, lo + c)])
        indptr = None if all(c == 1 for c in cnt) else _i32([sum(cnt[:i]) for i in range(len(cnt) + 1)])
        sl = _i32([slots[i] for i in rows])
        ops.conv_causal(x, dev["x.b"], conv, dev["conv.b"], hist, u, pos, indptr, sl)
        ops.gemm(u, gates_w, out=gates, groups=blocks)
        ops.rglru_scan(u, gates, gate_b, dev["lam"], y, x, dev["y.b"], state, hist, out, pos, indptr, sl, block=b)
        ops.check_status()
        at = 0
        for i, c in zip(rows, cnt):
            got[i].append(out[at:at + c].float().cpu())
            at += c
    for i, wnt in enumerate(want):
        err = _rel(torch.cat(got[i]), wnt)
        assert err < (2e-6 if dt == F32 else 8e-3), (i, err)
    assert float(state[1].min()) == 1e3 == float(state[3].max())
