"""Mechanisms of the Vofidra design in the kernels, each against a plain fp32 / fp64 computation, on inputs that make a
mistake visible: keys that stand out at page borders, at the edges of the bias table and far away, routers with close groups,
sizes of every kind."""
import math

import pytest
import torch

import vofidra_plain as plain

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


pad = lambda n: (n + 7) // 8 * 8


# ------------------------------------------------------------------------------------------------ several residual streams
@pytest.mark.parametrize("S", [1, 2, 3, 4, 8])
@pytest.mark.parametrize("H", [7, 64, 1100, 4096])
@pytest.mark.parametrize("dt", [BF, F32])
def test_streams(ops, S, H, dt):
    g = torch.Generator().manual_seed(S * H)
    r = lambda *s: torch.randn(*s, generator=g)
    T, V, n = 9, 30, 5
    x, embed, y = r(T, S, H), r(V, H).to(dt), r(T, H).to(dt)
    mix, out_w, in_w = r(S, S).to(dt), r(S).to(dt), r(S).to(dt)
    w, b, alpha = r(H).to(dt), r(H).to(dt), torch.tensor([0.7]).to(dt)
    rows_of = torch.randint(-1, 20, (T, n), generator=g)
    many, ident, prev = r(20, H).to(dt), r(T).abs(), r(T, H).to(dt)
    ident[3] = 0.0
    ids = torch.randint(0, V, (T,), generator=g)
    d, dev = (lambda t: t.double()), (lambda t: t.to(DEV))
    norm = tuple(map(dev, (w, alpha, b)))
    tol = 2e-6 if dt == F32 else 4e-3
    y_rows = torch.stack([sum((d(many[k]) for k in row.tolist() if k >= 0), torch.zeros(H, dtype=torch.float64)) for row in rows_of])
    sources = {"none": (None, None), "dense": (ops.Pending(dev(y), dev(mix), dev(out_w)), d(y)),
               "rows": (ops.Pending(dev(many), dev(mix), dev(out_w), _i32(rows_of.tolist())), y_rows),
               "identity": (ops.Pending(dev(many), dev(mix), dev(out_w), _i32(rows_of.tolist()), dev(ident), dev(prev)),
                            y_rows + d(ident)[:, None] * d(prev))}
    for fresh in (False, True):
        start = d(embed)[ids][:, None].expand(T, S, H) if fresh else d(x)
        kw = dict(ids=_i32(ids.tolist()), embed=dev(embed)) if fresh else {}
        for name, (pending, want_y) in sources.items():
            xs = start.transpose(0, 1)
            if pending is not None:
                xs = plain.streams_out(xs, d(mix), d(out_w), want_y)
            u = plain.streams_in(xs, d(in_w))
            want = plain.dyt(u, d(w), d(b), d(alpha))
            xd, h = x.to(DEV), torch.full((T, H), 9.0, dtype=dt, device=DEV)
            if name == "identity":              # what the sublayer read is replaced by what the next one reads
                h = pending.prev.clone()
                pending = pending._replace(prev=h)
            ops.stream_mix(xd, **kw, pending=pending, read=dev(in_w), norm=norm, out=h, write=pending is not None)
            assert _rel(h, want) < tol, (name, fresh)
            assert _rel(xd.transpose(0, 1), xs if pending is not None else d(x).transpose(0, 1)) < 1e-6
            # some rows only, nothing kept, the plain sum
            at = torch.tensor([5, 2, 9, 2])
            xd, h, tot = x.to(DEV), torch.empty(4, H, dtype=dt, device=DEV), torch.empty(4, H, device=DEV)
            pending = sources[name][0]
            ops.stream_mix(xd, **kw, pending=pending, norm=norm, out=h, total=tot, rows=_i32(at.tolist()), row_offset=-1)
            assert _rel(tot, xs.sum(0)[at - 1]) < 1e-6 and _rel(h, plain.dyt(xs.sum(0), d(w), d(b), d(alpha))[at - 1]) < tol
            assert torch.equal(xd.cpu(), x)
    ops.check_status()


# ------------------------------------------------------------------------------------------------ normed heads and the paged write
@pytest.mark.parametrize("dim,vdim,qh,kvh", [(64, 64, 6, 3), (128, 96, 12, 1), (40, 24, 4, 4), (22, 13, 9, 3), (256, 8, 2, 2), (264, 16, 2, 1), (8, 8, 1, 1)])
@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("temp", [None, {"coef": 0.4, "every": 16}, {"coef": 1.5, "every": 1}])
def test_norm_store(ops, dim, vdim, qh, kvh, dt, temp):
    g = torch.Generator().manual_seed(dim)
    page, eps, slot = 16, 1e-3, [3, 17, 40, 111, 64, -1, 0]
    pos = [0, 14, 15, 16, 31, 5, 90000]
    T = len(pos)
    at = [0, pad(qh * dim), pad(qh * dim) + pad(kvh * dim)]
    x = torch.randn(T, at[2] + pad(kvh * vdim) + 16, generator=g).to(dt)
    cut = lambda t: (t[:, :qh * dim], t[:, at[1]:at[1] + kvh * dim], t[:, at[2]:at[2] + kvh * vdim])
    qw, kw = (1 + 0.5 * torch.randn(dim, generator=g)).to(dt), (1 + 0.5 * torch.randn(dim, generator=g)).to(dt)
    q, k, v = (t.double().reshape(T, -1, n) for t, n in zip(cut(x), (dim, dim, vdim)))
    scale = plain.temperature(max(pos) + 1, temp, torch.float64)[pos] if temp else torch.ones(T, dtype=torch.float64)
    want_q, want_k = plain.rms_norm(q, qw.double(), eps) * scale[:, None, None], plain.rms_norm(k, kw.double(), eps)
    kv = torch.zeros(7, 2, page, kvh, dim, dtype=dt, device=DEV) if dim == vdim else ops.KVPair(
        torch.zeros(7, page, kvh, dim, dtype=dt, device=DEV), torch.zeros(7, page, kvh, vdim, dtype=dt, device=DEV))
    xd = x.to(DEV)
    ops.norm_store(*cut(xd), _i32(pos), _i32(slot), kv, qw.to(DEV), kw.to(DEV), q_heads=qh, kv_heads=kvh, dim=dim, page_size=page, eps=eps,
                   **(dict(temp_coef=temp["coef"], temp_every=temp["every"]) if temp else {}))
    ops.check_status()
    tol = 2e-6 if dt == F32 else 4e-3
    assert _rel(cut(xd)[0].reshape(T, qh, dim), want_q) < tol
    assert torch.equal(xd[:, qh * dim:].cpu(), x[:, qh * dim:])
    K, V = (t.reshape(7 * page, kvh, -1).cpu() for t in ((kv[0], kv[1]) if isinstance(kv, tuple) else (kv[:, 0], kv[:, 1])))
    for t, s in enumerate(slot):
        if s >= 0:
            assert _rel(K[s], want_k[t]) < tol and torch.equal(V[s], v[t].to(dt))
    assert sum(bool(r.any()) for r in K) == len(slot) - 1


# ------------------------------------------------------------------------------------------------ a bias by distance
# (heads, kv heads, dim, vdim, page, rows, far)
BIAS = [(6, 3, 64, 64, 16, 20, 100), (12, 1, 128, 96, 64, 32, 200), (4, 4, 40, 24, 16, 9, 600), (9, 3, 22, 13, 16, 7, 12), (16, 2, 128, 128, 64, 64, 128),
        (1, 1, 8, 128, 128, 2, 2), (10, 2, 72, 40, 32, 33, 1000)]


@pytest.mark.parametrize("dt", [BF, F32])
@pytest.mark.parametrize("case", BIAS)
def test_attention_with_a_distance_bias(ops, case, dt):
    """Prompts, portions behind any prefix, and single tokens with and without key splits.  Neighbouring rows of the table
    differ by several units, so that a key on the wrong side of an edge takes or loses most of the weight."""
    from blitz_scale_b200.models.hybrid_config import DistanceBias
    H, G, d, dv, page, rows, far = case
    lens, q_lens = [700, 65, 1, 300, 389], [700, 65, 1, 2, 260]
    g = torch.Generator().manual_seed(H * d + dv)
    scale = 0.6 * d ** -0.5
    spread = DistanceBias(rows, far).rows_by_distance()
    table = (3 * torch.randn(rows, H, generator=g)).to(dt)
    bias = table[torch.tensor(spread)].t().contiguous()
    npages = [-(-n // page) for n in lens]
    perm = torch.randperm(sum(npages), generator=g).tolist()
    shape = (sum(npages), page, G)
    kv = torch.zeros(shape[0], 2, *shape[1:], d, dtype=dt, device=DEV) if d == dv else ops.KVPair(
        torch.zeros(*shape, d, dtype=dt, device=DEV), torch.zeros(*shape, dv, dtype=dt, device=DEV))
    K, V = (kv[0], kv[1]) if isinstance(kv, tuple) else (kv[:, 0], kv[:, 1])
    want, qs, at = [], [], 0
    for n, ql, np_ in zip(lens, q_lens, npages):
        k, v = torch.randn(n, G, d, generator=g).to(dt), torch.randn(n, G, dv, generator=g).to(dt)
        q = torch.randn(n, H, d, generator=g).to(dt)
        for i in range(np_):
            part = slice(i * page, min(n, (i + 1) * page))
            K[perm[at + i], :part.stop - part.start] = k[part].to(DEV)
            V[perm[at + i], :part.stop - part.start] = v[part].to(DEV)
        at += np_
        of = torch.tensor([plain.bucket(x, rows, far) for x in range(n)])
        dist = (torch.arange(n)[:, None] - torch.arange(n)[None]).clamp(min=0)
        o = torch.stack([plain.softmax_values(q[:, h].double(), k[:, h // (H // G)].double(), v[:, h // (H // G)].double(), scale,
                                              table[of, h].double()[dist]) for h in range(H)], 1)
        want.append(o[n - ql:])
        qs.append(q[n - ql:])
    T = sum(q_lens)
    proj = torch.zeros(T, pad(H * d) + 8, dtype=dt, device=DEV)
    q = proj[:, :H * d]
    q.copy_(torch.cat(qs).reshape(T, -1))
    pos = _i32([p for n, ql in zip(lens, q_lens) for p in range(n - ql, n)])
    tokp, indptr = (_i32([sum(x[:i]) for i in range(len(lens) + 1)]) for x in (q_lens, npages))
    indices, last = _i32(perm), _i32([n - (u - 1) * page for n, u in zip(lens, npages)])
    bias = bias.to(DEV)
    tol = 8e-6 if dt == F32 else 2.4e-2

    def check(out, at, what):
        ops.check_status()
        for i, (w, r) in enumerate(zip(want, at)):
            got, w = out[r].reshape(-1, H, dv).double().cpu(), w[-len(r):]
            err = (got - w).flatten(1).norm(dim=1) / w.flatten(1).norm(dim=1).clamp_min(1e-3)
            assert float(err.max()) < tol, (what, i, int(err.argmax()), float(err.max()))
    all_rows = [list(range(int(tokp[i]), int(tokp[i + 1]))) for i in range(len(lens))]
    buf = torch.full((T, pad(H * dv) + 8), 7.0, dtype=dt, device=DEV)
    ops.attn_ragged(q, kv, pos, tokp, indptr, indices, buf, q_heads=H, kv_heads=G, dim=d, page_size=page, scale=scale, bias=bias)
    check(buf[:, :H * dv], all_rows, "general")
    if not ops.attn_tensor_core(q, H, G, d, page, dv):
        assert dt == F32 or d % 8 or dv % 8
        return
    buf.fill_(7.0)
    kw = dict(q_heads=H, kv_heads=G, head_dim=d, page_size=page, sm_scale=scale, bias=bias)
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
@pytest.mark.parametrize("q_rank,rank,rot", [(88, 104, 32), (768, 256, 32), (1536, 512, 64), (35, 21, 6), (8, 8, 2), (64, 40, 0), (16, 2000, 16)])
@pytest.mark.parametrize("dt", [BF, F32])
def test_latent_store_and_gather(ops, q_rank, rank, rot, dt):
    g = torch.Generator().manual_seed(rank)
    page, eps, base = 8, 1e-3, 700.0
    pos, slot = [0, 1, 7, 8, 5, 90000], [3, 17, 40, 55, -1, 0]
    T, at, W = len(pos), pad(q_rank), rank + rot
    x = torch.randn(T, at + pad(W) + 8, generator=g).to(dt)
    qw, kw = (1 + 0.5 * torch.randn(q_rank, generator=g)).to(dt), (1 + 0.5 * torch.randn(rank, generator=g)).to(dt)
    kv = ops.LatentKV(torch.zeros(7, page, 1, W, dtype=dt, device=DEV), rank)
    xd = x.to(DEV)
    ops.latent_store(xd[:, :q_rank], xd[:, at:at + W], _i32(pos), _i32(slot), kv, qw.to(DEV), kw.to(DEV), ops.rope_freqs(rot, base, DEV), eps=eps)
    ops.check_status()
    tol = 2e-6 if dt == F32 else 4e-3
    assert _rel(xd[:, :q_rank], plain.rms_norm(x[:, :q_rank].double(), qw.double(), eps)) < tol and torch.equal(xd[:, q_rank:].cpu(), x[:, q_rank:])
    full = x[:, at:at + W].double()
    at_pos = lambda t: plain.rotate_half(full[t, rank:].expand(pos[t] + 1, rot), rot, base)[-1] if pos[t] < 100 else None
    rows = kv.pool.view(-1, W).cpu()
    for t, s in enumerate(slot):
        if s < 0:
            continue
        assert _rel(rows[s, :rank], plain.rms_norm(full[t, :rank], kw.double(), eps)) < tol
        if rot and pos[t] < 100:
            assert _rel(rows[s, rank:], at_pos(t)) < tol
        elif rot:
            a = pos[t] * torch.tensor([base ** (-2.0 * i / rot) for i in range(rot // 2)], dtype=torch.float64)
            u, v = full[t, rank:rank + rot // 2], full[t, rank + rot // 2:]
            assert _rel(rows[s, rank:], torch.cat([u * a.cos() - v * a.sin(), v * a.cos() + u * a.sin()])) < tol
    assert sum(bool(r.any()) for r in rows) == len(slot) - 1
    pages = [5, 0, 6, 0]
    out = torch.full((len(pages) * page, W), 7.0, dtype=dt, device=DEV)
    if page * W * out.element_size() % 16 == 0:
        ops.latent_gather(kv, _i32(pages), out)
        assert torch.equal(out.view(len(pages), page, W), kv.pool[pages, :, 0])


@pytest.mark.parametrize("heads,dim,rot", [(5, 48, 32), (32, 64, 32), (3, 13, 6), (1, 8, 2), (40, 128, 64), (4, 24, 16)])
@pytest.mark.parametrize("dt", [BF, F32])
def test_latent_rotate(ops, heads, dim, rot, dt):
    g = torch.Generator().manual_seed(dim)
    T, base, rank = 40, 300.0, 24
    q = torch.randn(T, heads * (dim + rot), generator=g).to(dt)
    want = plain.rotate_half(q.double().view(T, heads, dim + rot)[..., dim:], rot, base)
    fr, pos = ops.rope_freqs(rot, base, DEV), _i32(list(range(T)))
    tol = 2e-6 if dt == F32 else 4e-3
    inplace = q.to(DEV)
    ops.latent_rotate(inplace, inplace[:, dim:], pos, fr, heads=heads, dim=dim, rot=rot, out_step=dim + rot)
    got = inplace.view(T, heads, dim + rot)
    assert _rel(got[..., dim:], want) < tol and torch.equal(got[..., :dim].cpu(), q.view(T, heads, -1)[..., :dim])
    out = torch.full((T, heads * (rank + rot)), 7.0, dtype=dt, device=DEV)
    ops.latent_rotate(q.to(DEV), out[:, rank:], pos, fr, heads=heads, dim=dim, rot=rot, out_step=rank + rot)
    got = out.view(T, heads, rank + rot)
    assert _rel(got[..., rank:], want) < tol and bool((got[..., :rank] == 7.0).all())


LATENT = [(1, 80, 64, 64), (5, 136, 104, 16), (32, 288, 256, 64), (40, 96, 80, 8), (64, 576, 512, 64), (128, 320, 320, 128), (33, 16, 8, 32), (256, 288, 256, 64)]


@pytest.mark.parametrize("lens", [[1], [130, 0, 700, 64, 65], [(i * 37) % 300 for i in range(170)], [3000]])
@pytest.mark.parametrize("case", LATENT)
def test_latent_decode_attention(ops, case, lens):
    """One key row for all heads; a few rows stand out (the first ones, those at page and block borders, the last)."""
    H, W, R, page = case
    B = len(lens)
    for dt in (BF, HF, F32):
        if dt != BF and B > 5:
            continue
        g = torch.Generator().manual_seed(H + B)
        npages = [-(-n // page) for n in lens]
        perm = torch.randperm(sum(npages) + 2, generator=g)[:max(1, sum(npages))].tolist()
        kv = ops.LatentKV(torch.zeros(sum(npages) + 2, page, 1, W, dtype=dt, device=DEV), R)
        q, z, scale = torch.randn(B, H, W, generator=g), (2 * torch.randn(B, H, generator=g)).to(dt), 0.8 * W ** -0.5
        want, at = torch.zeros(B, H, R, dtype=torch.float64), 0
        u = torch.randn(W, generator=g)
        u = u / u.norm() * W ** 0.5
        q = (0.5 * q + u).to(dt)
        for b, n in enumerate(lens):
            k = torch.randn(n, W, generator=g)
            loud = sorted({p for p in (0, 1, page - 1, page, 63, 64, 127, 128, 129, 255, 256, n // 2, n - 2, n - 1) if 0 <= p < n})
            k[loud] = k[loud] * 0.3 + 0.9 * u
            k = k.to(dt)
            for i in range(npages[b]):
                part = k[i * page:(i + 1) * page]
                kv.pool[perm[at + i], :len(part), 0] = part.to(DEV)
            at += npages[b]
            if n:
                want[b] = torch.softmax(q[b].double() @ k.double().T * scale, -1) @ k[:, :R].double() * torch.sigmoid(z[b].double())[:, None]
        indptr = _i32([sum(npages[:i]) for i in range(B + 1)])
        last = _i32([n - (p - 1) * page if p else 0 for n, p in zip(lens, npages)])
        qd, zd, out = q.reshape(B, -1).to(DEV), z.to(DEV), torch.full((B, H * R), 7.0, dtype=dt, device=DEV)
        live = [b for b, n in enumerate(lens) if n]
        tol = 8e-6 if dt == F32 else 2e-2

        def check(what):
            ops.check_status()
            got = out.view(B, H, R).double().cpu()
            err = ((got - want).flatten(1).norm(dim=1) / want.flatten(1).norm(dim=1).clamp_min(1e-3))[live]
            assert float(err.max()) < tol, (what, dt, int(err.argmax()), float(err.max()))
            assert all(not got[b].any() for b, n in enumerate(lens) if n == 0)
        ops.attn_ragged(qd, kv, _i32([max(0, n - 1) for n in lens]), None, indptr, _i32(perm), out, q_heads=H, kv_heads=1, dim=W, page_size=page,
                        scale=scale, gate=zd)
        check("general")
        assert ops.attn_latent_supported(qd, B, H, kv) == (dt != F32)
        if dt != F32:
            out.fill_(7.0)
            ops.attn_latent(qd, kv, _i32(perm), indptr, last, heads=H, scale=scale, workspace=ops.attn_latent_workspace(H, R, DEV), out=out, gate=zd)
            check("tensor cores")


@pytest.mark.parametrize("H,W,R,page", [(5, 136, 104, 16), (32, 544, 512, 64), (72, 80, 64, 32)])
def test_latent_attention_of_prompt_tokens(ops, H, W, R, page):
    """Tokens of a ragged step as rows of their own, behind any prefix, in several launches: against the general kernel."""
    lens, q_lens = [900, 1, 65, 300, 1100], [900, 1, 2, 260, 130]
    g = torch.Generator().manual_seed(H)
    npages = [-(-n // page) for n in lens]
    perm = torch.randperm(sum(npages), generator=g).tolist()
    kv = ops.LatentKV(torch.randn(sum(npages), page, 1, W, generator=g).to(DEV, BF), R)
    T = sum(q_lens)
    q, gate = torch.randn(T, H * W, generator=g).to(DEV, BF), torch.randn(T, H, generator=g).to(DEV, BF)
    pos = _i32([p for n, ql in zip(lens, q_lens) for p in range(n - ql, n)])
    tokp, indptr = (_i32([sum(x[:i]) for i in range(len(lens) + 1)]) for x in (q_lens, npages))
    want, got = torch.empty(T, H * R, dtype=BF, device=DEV), torch.full((T, H * R), math.nan, dtype=BF, device=DEV)
    scale = 1.2 * W ** -0.5
    ops.attn_ragged(q, kv, pos, tokp, indptr, _i32(perm), want, q_heads=H, kv_heads=1, dim=W, page_size=page, scale=scale, gate=gate)
    ops.attn_latent(q, kv, _i32(perm), indptr, indptr, heads=H, scale=scale, workspace=ops.attn_latent_workspace(H, R, DEV), out=got, gate=gate,
                    pos=pos, tok_indptr=tokp)
    ops.check_status()
    err = (got.float() - want.float()).norm(dim=1) / want.float().norm(dim=1)
    assert float(err.max()) < 2e-2, int(err.argmax())


@pytest.mark.parametrize("M", [1, 5, 130, 300])
@pytest.mark.parametrize("G,K,N,a_step,out_step", [(5, 48, 104, 80, 136), (32, 64, 256, 96, 288), (3, 13, 21, 19, 27), (4, 256, 64, 256, 64), (2, 72, 40, 72, 40),
                                                   (1, 24, 16, 40, 24), (8, 200, 8, 208, 16)])
@pytest.mark.parametrize("dt", [BF, F32])
def test_block_diagonal_product_over_parts_of_wider_blocks(ops, M, G, K, N, a_step, out_step, dt):
    g = torch.Generator().manual_seed(M + K)
    a, b = torch.randn(M, pad(G * a_step), generator=g).to(dt), (torch.randn(G * K, N, generator=g) * K ** -0.5).to(dt)
    out = torch.full((M, pad(G * out_step)), 7.0, dtype=dt, device=DEV)
    ops.gemm(a.to(DEV), b.to(DEV), out=out, groups=G, a_step=a_step, out_step=out_step, static_b=True)
    ops.check_status()
    for i in range(G):
        want = a[:, i * a_step:i * a_step + K].double() @ b[i * K:(i + 1) * K].double()
        assert _rel(out[:, i * out_step:i * out_step + N], want) < (2e-6 if dt == F32 else 4e-3)
        assert bool((out[:, i * out_step + N:(i + 1) * out_step] == 7.0).all())


# ------------------------------------------------------------------------------------------------ experts
@pytest.mark.parametrize("T", [1, 7, 64, 300])
@pytest.mark.parametrize("E,I,top,H,ff,groups", [(7, 3, 3, 200, 72, (5, 3)), (20, 12, 6, 96, 32, (8, 3)), (5, 0, 2, 136, 104, None), (1, 1, 2, 64, 8, None),
                                                 (130, 30, 5, 72, 40, (16, 4)), (4, 1, 2, 121, 33, None), (2, 6, 4, 88, 24, (2, 1))])
@pytest.mark.parametrize("dt", [BF, F32])
def test_gated_experts(ops, T, E, I, top, H, ff, groups, dt):
    """Router, both grouped products and the streams' sum of the rows against the oracle's experts."""
    g = torch.Generator().manual_seed(T + E)
    r = lambda *s: torch.randn(*s, generator=g)
    h, z = r(T, H).to(dt), 2.0 * r(T, E + I)
    w = {f"e{e}.{n}": (r(*s) * s[1] ** -0.5).to(dt) for e in range(E) for n, s in (("gate", (ff, H)), ("up", (ff, H)), ("down", (H, ff)))}
    corr = (0.2 * r(E + I)).to(dt)
    router = {"experts": E, "identity": I, "top": top, "groups": {"count": groups[0], "keep": groups[1]} if groups else None}
    want = torch.zeros(T, H, dtype=torch.float64)
    for t in range(T):
        for e, wt in plain.route(z[t].double(), corr.double(), router)[0]:
            y = h[t].double() if e >= E else plain.gated_ff(h[t:t + 1].double(), *(w[f"e{e}.{n}"].double() for n in ("gate", "up", "down")))[0]
            want[t] += wt * y
    ffp = (ff + 31) // 32 * 32
    wide = lambda m: torch.cat([m.T, torch.zeros(H, ffp - ff, dtype=dt)], 1)
    up = torch.stack([ops.interleave_gate(wide(w[f"e{e}.gate"]), wide(w[f"e{e}.up"])) for e in range(E)]).to(DEV)
    down = torch.stack([torch.cat([w[f"e{e}.down"].T, torch.zeros(ffp - ff, H, dtype=dt)], 0) for e in range(E)]).to(DEV)
    hd = h.to(DEV)
    tc = ops.grouped_tensor_core(hd, up, down)
    assert tc == (dt == BF and H % 8 == 0)
    plan = ops.ExpertPlan(300, E, top, False, DEV, identity=I)
    for bn, fetch in ((0, 0), (64, 1), (128, 1), (256, 1), (64, 2), (256, 2)) if tc else ((0, 0),):
        ops.moe_route(z.to(DEV), plan, weight_on_input=False, renormalize=True, softmax=True, correction=corr.to(DEV),
                      groups=groups[0] if groups else 0, keep=groups[1] if groups else 0, tile_rows=128 if tc else 64)
        act = torch.full((plan.rows, ffp), math.nan, dtype=dt, device=DEV)      # nothing unwritten may be read
        y = torch.full((plan.rows, H), math.nan, dtype=dt, device=DEV)
        ops.gemm_grouped(hd, up, plan, act, gather=True, act="silu_gate", factors=True, bn=bn, fetch=fetch)
        ops.gemm_grouped(act, down, plan, y, bn=bn)
        x, one = torch.zeros(T, 1, H, device=DEV), torch.ones(1, 1, dtype=dt, device=DEV)
        tot = torch.empty(T, H, device=DEV)
        ops.stream_mix(x, pending=ops.Pending(y, one, one[0], plan.place, plan.ident, hd if I else None), total=tot)
        ops.check_status()
        assert _rel(tot, want) < (3e-6 if dt == F32 else 8e-3), (bn, fetch)


@pytest.mark.parametrize("T,E,I,top,groups,keep", [(1, 1, 1, 1, 1, 1), (5, 7, 0, 7, 0, 0), (3000, 3, 3, 2, 3, 2), (2000, 900, 100, 8, 100, 7), (257, 48, 16, 6, 8, 4),
                                                   (33, 40, 32, 32, 2, 1), (40, 500, 12, 3, 256, 2)])
@pytest.mark.parametrize("softmax,corrected", [(True, True), (True, False), (False, True)])
def test_router_with_groups_and_identity_experts(ops, T, E, I, top, groups, keep, softmax, corrected):
    """Choices, weights, sorted rows and work list; twice on the same buffers."""
    g = torch.Generator().manual_seed(T)
    O = E + I
    plan = ops.ExpertPlan(T + 3, E, top, False, DEV, identity=I)
    for renorm in (True, False):
        z = 3 * torch.randn(T, O + 5, generator=g)
        corr = 0.3 * torch.randn(O, generator=g) if corrected else torch.zeros(O)
        ops.moe_route(z.to(DEV), plan, weight_on_input=False, renormalize=renorm, softmax=softmax, correction=corr.to(DEV) if corrected else None,
                      groups=groups, keep=keep, tile_rows=128)
        ops.check_status()
        zz = z[:, :O].double()
        s = torch.softmax(zz, -1) if softmax else torch.sigmoid(zz)
        choice = s + corr.double()
        if groups:
            best = choice.view(T, groups, -1).max(-1).values.sort(-1, descending=True).indices[:, :keep]
            kept = torch.zeros(T, groups, dtype=torch.bool).scatter_(1, best, True)
            choice = choice.masked_fill(~kept.repeat_interleave(O // groups, 1), -math.inf)
        val, idx = choice.sort(-1, descending=True)
        tight = lambda v: 1e-5 * v.abs() + (1e-6 if corrected else 0.0)
        clear = torch.ones(T, dtype=torch.bool) if top == O or top == O // max(1, groups) * keep else val[:, top - 1] - val[:, top] > tight(val[:, top])
        if groups and keep < groups:
            gs = (s + corr.double()).view(T, groups, -1).max(-1).values.sort(-1, descending=True).values
            clear &= gs[:, keep - 1] - gs[:, keep] > tight(gs[:, keep])
        assert int(clear.sum()) > 0.9 * T                       # fp32 scores may order closer ones either way
        idx = idx[:, :top]
        wt = s.gather(1, idx)
        if renorm:
            wt = wt / wt.sum(1, keepdim=True)
        want = torch.zeros(T, O, dtype=torch.float64).scatter_(1, idx, wt)
        place, src = plan.place.cpu().long(), plan.src.cpu().long()
        fac, tiles = plan.factors.cpu().double(), plan._tiles.cpu()[:int(plan.num_tiles)].tolist()
        real = place >= 0
        n = int(real.sum())
        assert sorted(place[real].tolist()) == list(range(n)) and torch.equal(src[place[real]], real.nonzero()[:, 0])
        assert bool((fac[:n, 0] == 1).all()) and sum(t[2] for t in tiles) == n
        owner = torch.zeros(n, dtype=torch.long)
        for e, r0, rows, _ in tiles:
            owner[r0:r0 + rows] = e
        assert torch.equal(owner, owner.sort().values)
        got = torch.zeros(T, E, dtype=torch.float64)
        got[src[:n], owner] = fac[:n, 1]
        assert torch.allclose(got[clear], want[clear, :E], rtol=2e-5, atol=1e-12)
        if I:
            assert torch.allclose(plan.ident.cpu().double()[clear], want[clear, E:].sum(1), rtol=2e-5, atol=1e-12)
            assert bool(((~real).sum(1)[clear] == (want[clear, E:] > 0).sum(1)).all())
        assert not plan.counters[:E + 1].any()
