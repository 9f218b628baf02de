"""Small Fafudra configurations and random weights for the tests: sizes, head counts, layer orders, windows and constants
of their own, some of them on purpose odd (nothing a multiple of 8) or equal to 1."""
from __future__ import annotations

import json
from pathlib import Path
from typing import Dict, Optional

import torch


def attention(heads=4, kv_heads=2, dim=64, size=40, keep_first=3, rot_dims=None, base=5000.0, scale=None, softcap=20.0):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim,
                                           "mask": {"size": size, "keep_first": keep_first},
                                           "rot": {"base": base, "dims": dim if rot_dims is None else rot_dims},
                                           "scale": dim ** -0.5 if scale is None else scale, "softcap": softcap}}


def gla(heads=3, dim=32, vdim=64, tau=8.0, rank=8):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau, "rank": rank}}


def rglru(width=192, blocks=3, conv=4):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv}}


def config(layers, width=136, vocab=211, ff: Optional[list] = None, loop=None, eps=1e-5, residual_mult=0.6) -> dict:
    ff = ff if ff is not None else [112] * len(layers)
    out = {"architecture": "Fafudra", "layers": [], "norm": {"eps": eps}, "residual_mult": residual_mult, "vocab": vocab,
           "width": width}
    for L, f in zip(layers, ff):
        out["layers"].append({**json.loads(json.dumps(L)), "mlp": {"ff": f, "kind": "dense"} if f else None})
    if loop:
        out["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return out


def weights(c: dict, seed: int = 0, dtype=torch.bfloat16) -> Dict[str, torch.Tensor]:
    """Checkpoint tensors; activations of order one, every bias and sink large enough to matter."""
    g = torch.Generator().manual_seed(seed)
    r = lambda *s: torch.randn(*s, generator=g)
    lin = lambda o, i: r(o, i) * i ** -0.5
    H, w = c["width"], {}
    w["embed"] = 0.5 * r(c["vocab"], H)
    # gains of either sign: with tied embeddings the greedy token would otherwise be the input token again
    w["final.norm"] = -1.0 + r(H)
    if "loop" in c:
        w["loop.step"] = 0.5 * r(c["loop"]["times"], H)
    for i, L in enumerate(c["layers"]):
        p, m = f"l{i}.mix.", L["mixer"]
        w[f"l{i}.norm1"] = 0.2 * r(H)
        if L["type"] == "attention":
            # logits of a few units: the window's edge, the cap and the sink are all visible in the output
            w[p + "q"], w[p + "k"] = 2.0 * lin(m["heads"] * m["dim"], H), 2.0 * lin(m["kv_heads"] * m["dim"], H)
            w[p + "sink"] = 2.0 + r(m["heads"])
            out = m["heads"] * m["dim"]
        elif L["type"] == "gla":
            hk, hv = m["heads"] * m["dim"], m["heads"] * m["vdim"]
            for n, o in (("q", hk), ("k", hk), ("v", hv), ("g", hv), ("a1", m["rank"])):
                w[p + n] = lin(o, H)
            w[p + "a2"], w[p + "a2.b"], w[p + "norm"] = 2.0 * lin(hk, m["rank"]), 1.0 + 2.0 * r(hk), 1.0 + 0.3 * r(m["vdim"])
            out = hv
        else:
            W, b = m["width"], m["width"] // m["blocks"]
            for n in ("y", "x"):
                w[p + n], w[p + n + ".b"] = lin(W, H), 0.3 * r(W)
            w[p + "conv"], w[p + "conv.b"] = 0.6 * r(W, m["conv"]), 0.3 * r(W)
            for n in ("ra", "ri"):
                w[p + n], w[p + n + ".b"] = r(m["blocks"], b, b) * b ** -0.5, 0.5 * r(m["blocks"], b)
            w[p + "lam"] = -3.0 + 1.5 * r(W)
            out = W
        w[p + "o"] = lin(H, out)
        if L["mlp"]:
            f = L["mlp"]["ff"]
            w[f"l{i}.mlp.gate"], w[f"l{i}.mlp.up"], w[f"l{i}.mlp.down"] = lin(f, H), lin(f, H), lin(H, f)
    return {n: t.to(dtype).contiguous() for n, t in w.items()}


def write(directory, c: dict, w: Dict[str, torch.Tensor]) -> str:
    """A checkpoint folder (without the rank, which a checkpoint's shapes give)."""
    from blitz_scale_b200.models.convert import write_safetensors
    d = Path(directory)
    d.mkdir(parents=True, exist_ok=True)
    c = json.loads(json.dumps(c))
    for L in c["layers"]:
        L["mixer"].pop("rank", None)
    (d / "config.json").write_text(json.dumps(c))
    write_safetensors(d / "model.safetensors", w)
    return str(d)


CASES = {
    # sizes the tensor-core kernels take; a loop at the start
    "regular": config([gla(dim=32, vdim=64), attention(), rglru(), gla(heads=2, dim=64, vdim=128, tau=4.0), attention(size=70, keep_first=1)],
                      width=256, vocab=304, ff=[192] * 5, loop=(0, 3, 2)),
    "head128": config([attention(heads=8, kv_heads=2, dim=128, size=100, keep_first=5, rot_dims=64, softcap=15.0), gla(dim=64, vdim=64)],
                      width=192, vocab=264, ff=[128, 0]),
    # nothing a multiple of 8, layers without a feed-forward, a loop over everything
    "odd": config([rglru(width=90, blocks=5, conv=3), gla(heads=3, dim=12, vdim=22, tau=2.0, rank=5),
                   attention(heads=6, kv_heads=3, dim=20, size=17, keep_first=2, rot_dims=12, softcap=9.0)],
                  width=121, vocab=157, ff=[51, 0, 30], loop=(0, 3, 2), residual_mult=1.3),
    # values equal to 1: one head, one block, one tap, one pass, rank 1, a window of 1, one kept token
    "ones": config([gla(heads=1, dim=16, vdim=16, tau=1.0, rank=1), attention(heads=1, kv_heads=1, dim=32, size=1, keep_first=1, rot_dims=2),
                    rglru(width=64, blocks=1, conv=1)], width=64, vocab=96, ff=[64, 64, 64], loop=(1, 2, 1), residual_mult=1.0),
    # no loop, no kept tokens, no rotation
    "plain": config([attention(heads=3, kv_heads=3, dim=64, size=24, keep_first=0, rot_dims=0), rglru(width=128, blocks=2, conv=5)],
                    width=160, vocab=128, ff=[96, 96]),
}
