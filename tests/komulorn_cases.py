"""Small Komulorn configurations and random weights for the tests: sizes, head counts, layer orders and constants of their
own, some of them on purpose odd (nothing a multiple of 8) or equal to 1."""
from __future__ import annotations

import json
from pathlib import Path
from typing import Dict, Optional

import torch


def attention(heads=4, kv_heads=2, dim=64, vdim=32, rot_dims=32, base=5000.0, scaling=(3.0, 96, 16.0, 1.0), scale=None,
              kv_from: Optional[int] = None):
    rot = {"base": base, "dims": rot_dims}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": rot, "scale": 0.9 * dim ** -0.5 if scale is None else scale}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def moe(experts=6, top=2, ff=72, shared=104):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}, "shared": {"ff": shared} if shared else None}


def config(mixers, mlps, width=200, vocab=211, eps=1e-5, cap: Optional[float] = 12.0) -> dict:
    out = {"architecture": "Komulorn", "norm": {"eps": eps}, "vocab": vocab, "width": width, "logit_softcap": cap,
           "layers": [{"type": "attention", "mixer": json.loads(json.dumps(m)), "mlp": json.loads(json.dumps(f))}
                      for m, f in zip(mixers, mlps)]}
    return out


def weights(c: dict, seed: int = 0, dtype=torch.bfloat16) -> Dict[str, torch.Tensor]:
    """Checkpoint tensors; activations of order one, biases and gates large enough to matter, logits that reach the cap."""
    g = torch.Generator().manual_seed(seed)
    r = lambda *s: torch.randn(*s, generator=g)
    lin = lambda o, i: r(o, i) * i ** -0.5
    H, w = c["width"], {}
    w["embed"] = r(c["vocab"], H)
    w["final.norm"] = 1.0 + 0.3 * r(H)
    w["head"] = 10.0 * lin(c["vocab"], H)
    for i, L in enumerate(c["layers"]):
        p, m = f"l{i}.mix.", L["mixer"]
        w[f"l{i}.norm1"] = 1.0 + 0.2 * r(H)
        for n, o in (("q", m["heads"] * m["dim"]), ("k", m["kv_heads"] * m["dim"]), ("v", m["kv_heads"] * m["vdim"])):
            if n == "q" or "kv_from" not in m:
                # scores of a few units: rotation, scale and biases are all visible in the output
                w[p + n], w[p + n + ".b"] = (1.5 if n != "v" else 1.0) * lin(o, H), 0.7 * r(o)
        w[p + "g"] = 2.0 * lin(m["heads"], H)
        w[p + "o"] = 1.5 * lin(H, m["heads"] * m["vdim"])
        if L["mlp"]:
            f, q = L["mlp"], f"l{i}.mlp."
            w[f"l{i}.norm2"] = 1.0 + 0.2 * r(H)
            w[q + "router"] = 3.0 * lin(f["router"]["experts"], H)
            for e in range(f["router"]["experts"]):
                w[f"{q}e{e}.up"], w[f"{q}e{e}.down"] = 1.3 * lin(f["expert"]["ff"], H), lin(H, f["expert"]["ff"])
            if f["shared"]:
                n = f["shared"]["ff"]
                w[q + "shared.up"], w[q + "shared.down"], w[q + "shared.sg"] = lin(n, H), lin(H, n), 2.0 * lin(1, H)
    return {n: t.to(dtype).contiguous() for n, t in w.items()}


def write(directory, c: dict, w: Dict[str, torch.Tensor]) -> str:
    """A checkpoint folder."""
    from blitz_scale_b200.models.convert import write_safetensors
    d = Path(directory)
    d.mkdir(parents=True, exist_ok=True)
    (d / "config.json").write_text(json.dumps(c))
    write_safetensors(d / "model.safetensors", w)
    return str(d)


def clear_tokens(c: dict, w: Dict[str, torch.Tensor], n: int, seed: int, margin: float = 0.15):
    """Random tokens whose router decisions are all clear ones (logits at least `margin` from another choice), so that rounded
    activations take the same experts; and the oracle's logits."""
    from komulorn_plain import Plain
    g = torch.Generator().manual_seed(seed)
    new = lambda k: torch.randint(0, c["vocab"], (k,), generator=g)
    toks = new(n)
    p = Plain(c, w, torch.float32)
    for _ in range(200):
        logits = p.run(toks.tolist())
        close = (p.margin < margin).nonzero()[:, 0]
        if len(close) == 0:
            return toks.tolist(), logits
        early = close[:(len(close) + 1) // 2]       # a position's choices depend on it and the ones before it
        toks[early] = new(len(early))
    raise AssertionError("no clear tokens found")


CASES = {
    # sizes the tensor-core kernels take; two layers read the cache of one that is not their neighbour; a layer of attention alone
    "regular": config([attention(), attention(), attention(kv_from=0), attention(kv_from=0, scale=0.2), attention(kv_from=1)],
                      [moe(), moe(experts=9, top=3, ff=40, shared=64), None, moe(), moe(ff=136)]),
    # keys and values of one size (one cache tensor), twelve query heads on a key head
    "head128": config([attention(heads=12, kv_heads=1, dim=128, vdim=128, rot_dims=64), attention(heads=6, kv_heads=2, dim=128, vdim=128, rot_dims=128)],
                      [moe(experts=4, top=4), moe(experts=20, top=1, ff=64, shared=0)], width=192, vocab=264),
    # values wider than keys, sizes between the kernels' tiles, a rotation whose pairs are no multiple of 8
    "values": config([attention(heads=5, kv_heads=5, dim=40, vdim=96, rot_dims=12, base=300.0), attention(heads=10, kv_heads=5, dim=40, vdim=96, rot_dims=40, kv_from=0)],
                     [moe(experts=7, top=1, ff=96, shared=48)] * 2, width=136, vocab=152, cap=5.0),
    # nothing a multiple of 8
    "odd": config([attention(heads=9, kv_heads=3, dim=22, vdim=13, rot_dims=10, scaling=(2.0, 40, 8.0, 2.0)),
                   attention(heads=3, kv_heads=3, dim=22, vdim=13, rot_dims=10, scaling=(2.0, 40, 8.0, 2.0), kv_from=0), attention(heads=2, kv_heads=1, dim=9, vdim=21, rot_dims=2)],
                  [moe(experts=5, top=3, ff=51, shared=30), moe(experts=3, top=1, ff=7, shared=9), None], width=121, vocab=157),
    # values equal to 1: one head, one expert, one pair of rotated dimensions
    "ones": config([attention(heads=1, kv_heads=1, dim=16, vdim=8, rot_dims=2, scaling=(1.0, 64, 32.0, 1.0), scale=0.2)], [moe(experts=1, top=1, ff=8, shared=8)],
                   width=64, vocab=96, cap=1.0),
    # no scaled rotation, no cap, no shared expert, another layer's cache right away
    "plain": config([attention(heads=2, kv_heads=2, dim=64, vdim=64, rot_dims=64, scaling=None), attention(heads=8, kv_heads=2, dim=64, vdim=64, rot_dims=64, scaling=None, kv_from=0)],
                    [None, moe(experts=8, top=2, ff=64, shared=0)], width=160, vocab=128, cap=None),
}
