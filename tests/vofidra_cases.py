"""Small Vofidra configurations and random weights for the tests: sizes, head counts, layer orders and constants of their own,
some of them on purpose odd (nothing a multiple of 8) or equal to 1."""
from __future__ import annotations

import json
from typing import Dict, Optional

import torch

from komulorn_cases import write  # noqa: F401  (a checkpoint folder)


def attention(heads=6, kv_heads=3, dim=64, vdim=64, bias_max=100, rows=20, temp=(0.4, 16), scale=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "bias_max": bias_max, "scale": 0.9 * dim ** -0.5 if scale is None else scale}
    if temp:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return "attention", m, rows


def latent(heads=5, dim=48, rot_dim=32, vdim=72, q_rank=88, kv_rank=104, base=3000.0, scale=None):
    return "latent_attention", {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
                                "rot": {"base": base, "dims": rot_dim}, "scale": 1.1 * (dim + rot_dim) ** -0.5 if scale is None else scale}, 0


def dense(ff=136):
    return {"kind": "dense", "ff": ff}


def moe(experts=7, identity=3, top=3, ff=72, groups=(5, 3)):
    r = {"experts": experts, "identity": identity, "top": top}
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "router": r, "expert": {"ff": ff}}


def config(mixers, mlps, width=200, vocab=211, eps=1e-5, cap: Optional[float] = 12.0, streams=3) -> dict:
    out = {"architecture": "Vofidra", "norm": {"eps": eps}, "vocab": vocab, "width": width, "logit_softcap": cap, "streams": streams,
           "layers": [{"type": kind, "mixer": m, "mlp": f} for (kind, m, _), f in zip(mixers, mlps)]}
    out = json.loads(json.dumps(out))
    ROWS[json.dumps(out)] = [rows for _, _, rows in mixers]
    return out


ROWS: Dict[str, list] = {}     # rows of the distance biases, which a configuration does not say


def weights(c: dict, seed: int = 0, dtype=torch.bfloat16) -> Dict[str, torch.Tensor]:
    """Checkpoint tensors; activations of order one, coefficients, biases and gates large enough to matter, logits that reach
    the cap."""
    g = torch.Generator().manual_seed(seed)
    r = lambda *s: torch.randn(*s, generator=g)
    lin = lambda o, i: r(o, i) * i ** -0.5
    H, S, w = c["width"], c["streams"], {}

    def norm(name):
        w[name], w[name + ".b"], w[name + ".alpha"] = 1.2 + 0.3 * r(H), 0.4 * r(H), torch.tensor(0.6) + 0.1 * r(())
    w["embed"] = r(c["vocab"], H)
    norm("final.norm")
    w["head"] = 10.0 * lin(c["vocab"], H)
    for i, (L, rows) in enumerate(zip(c["layers"], ROWS[json.dumps(c)])):
        p, m, f, q = f"l{i}.mix.", L["mixer"], L["mlp"], f"l{i}.mlp."
        for k in (1, 2) if f else (1,):
            norm(f"l{i}.norm{k}")
            w[f"l{i}.hc{k}.in"] = 1.0 / S + 0.4 * r(S)
            w[f"l{i}.hc{k}.out"] = 0.8 + 0.5 * r(S)
            w[f"l{i}.hc{k}.mix"] = 0.7 * torch.eye(S) + 0.35 * r(S, S)
        h = m["heads"]
        if L["type"] == "attention":
            for n, o in (("q", h * m["dim"]), ("k", m["kv_heads"] * m["dim"]), ("v", m["kv_heads"] * m["vdim"])):
                w[p + n] = lin(o, H)
            w[p + "q.norm"], w[p + "k.norm"] = 1.6 + 0.4 * r(m["dim"]), 1.3 + 0.4 * r(m["dim"])
            w[p + "rel"] = 1.5 * r(rows, h)
        else:
            d, rd = m["dim"], m["rot_dim"]
            w[p + "dq"], w[p + "dkv"] = lin(m["q_rank"], H), 2.0 * lin(m["kv_rank"] + rd, H)
            w[p + "dq.norm"], w[p + "dkv.norm"] = 1.0 + 0.3 * r(m["q_rank"]), 1.0 + 0.3 * r(m["kv_rank"])
            w[p + "uq"], w[p + "uk"] = 1.6 * lin(h * (d + rd), m["q_rank"]), 1.3 * lin(h * d, m["kv_rank"])
            w[p + "uv"], w[p + "g"] = lin(h * m["vdim"], m["kv_rank"]), 2.0 * lin(h, H)
        w[p + "o"] = 1.5 * lin(H, h * m["vdim"])
        if f and f["kind"] == "dense":
            w[q + "gate"], w[q + "up"], w[q + "down"] = 1.5 * lin(f["ff"], H), lin(f["ff"], H), 1.5 * lin(H, f["ff"])
        elif f:
            n, ff = f["router"]["experts"], f["expert"]["ff"]
            o = n + f["router"]["identity"]
            # near-equal scores whose order the correction decides often; identity experts among the likely ones
            w[q + "router"], w[q + "correction"] = 2.0 * lin(o, H), 0.15 * r(o)
            for e in range(n):
                w[f"{q}e{e}.gate"], w[f"{q}e{e}.up"], w[f"{q}e{e}.down"] = 1.5 * lin(ff, H), lin(ff, H), 2.0 * lin(H, ff)
    return {n: t.to(dtype).contiguous() for n, t in w.items()}


def clear_tokens(c: dict, w: Dict[str, torch.Tensor], n: int, seed: int, margin: float = 0.006):
    """Random tokens whose router decisions are all clear ones (choice scores at least `margin` from another choice), so that
    rounded activations take the same experts; and the oracle's logits."""
    from vofidra_plain import Plain
    g = torch.Generator().manual_seed(seed)
    new = lambda k: torch.randint(0, c["vocab"], (k,), generator=g)
    toks = new(n)
    p = Plain(c, w, torch.float32)
    for _ in range(400):
        logits = p.run(toks.tolist())
        close = (p.margin < margin).nonzero()[:, 0]
        if len(close) == 0:
            return toks.tolist(), logits
        early = close[:(len(close) + 1) // 2]       # a position's choices depend on it and the ones before it
        toks[early] = new(len(early))
    raise AssertionError("no clear tokens found")


CASES = {
    # sizes the tensor-core kernels take; both mixers, both feed-forwards, a layer without one
    "regular": config([attention(), latent(), attention(rows=9, bias_max=33, temp=None), latent(heads=8, dim=64, vdim=64, kv_rank=64, rot_dim=16)],
                      [dense(), moe(), None, moe(experts=14, identity=2, top=5, ff=40, groups=(4, 2))]),
    # values of another size than keys, twelve query heads on a key head, one stream, no groups, no identity experts
    "values": config([attention(heads=12, kv_heads=1, dim=128, vdim=96, rows=32, bias_max=64, temp=(0.2, 7)), latent(heads=2, dim=96, rot_dim=32, vdim=128, q_rank=64, kv_rank=256)],
                     [moe(experts=5, identity=0, top=2, groups=None), dense(ff=64)], width=136, vocab=152, cap=5.0, streams=1),
    # a latent of several chunks of value columns, many streams
    "wide": config([latent(heads=32, dim=16, rot_dim=64, vdim=16, q_rank=40, kv_rank=320, scale=0.05), attention(heads=4, kv_heads=4, dim=40, vdim=24, rows=11, bias_max=50)],
                   [moe(experts=20, identity=12, top=6, ff=32, groups=(8, 3)), moe(experts=2, identity=6, top=4, ff=24, groups=(2, 1))], width=96, vocab=128, streams=5),
    # expanded heads larger than the prompt kernel takes: prompts stay in the latent space; more than 64 heads
    "deep": config([latent(heads=3, dim=120, rot_dim=40, vdim=136, q_rank=72, kv_rank=72), latent(heads=72, dim=8, rot_dim=16, vdim=8, q_rank=64, kv_rank=136, scale=0.1)],
                   [None, moe()], width=104, vocab=144, streams=4),
    # nothing a multiple of 8
    "odd": config([latent(heads=3, dim=13, rot_dim=6, vdim=11, q_rank=35, kv_rank=21), attention(heads=9, kv_heads=3, dim=22, vdim=13, rows=7, bias_max=12, temp=(1.5, 3))],
                  [dense(ff=51), moe(experts=4, identity=1, top=2, ff=33, groups=None)], width=121, vocab=157, streams=2),
    # values equal to 1: one head, one expert, one chosen, one group, one pair of rotated dimensions, temperature at every token
    "ones": config([attention(heads=1, kv_heads=1, dim=16, vdim=8, rows=2, bias_max=2, temp=(0.5, 1), scale=0.2), latent(heads=1, dim=8, rot_dim=2, vdim=8, q_rank=8, kv_rank=8)],
                   [moe(experts=1, identity=1, top=1, ff=8, groups=(1, 1)), moe(experts=1, identity=0, top=1, ff=8, groups=None)], width=64, vocab=96, cap=None),
}
