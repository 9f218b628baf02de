"""Small Norusun configurations and random weights for the tests: sizes, head counts, layer orders and constants of their own,
some of them on purpose odd (nothing a multiple of 8) or equal to 1."""
from __future__ import annotations

import json
from typing import Dict

import torch

from komulorn_cases import write  # noqa: F401  (a checkpoint folder)


def wkv(heads=5, dim=40, rank=12):
    return "wkv", {"heads": heads, "dim": dim}, rank


def latent(heads=5, dim=48, rot_dim=16, vdim=72, q_rank=88, kv_rank=104, base=3000.0, window=37, scale=None):
    return "latent_attention", {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
                                "rot": {"base": base, "dims": rot_dim}, "mask": {"size": window},
                                "scale": 0.8 * (dim + rot_dim) ** -0.5 if scale is None else scale}, 0


def left(heads=6, kv_heads=3, dim=64, vdim=64, rot_dims=24, base=700.0, chunk=50, scale=None):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": {"base": base, "dims": rot_dims}, "mask": {"size": chunk},
            "scale": 1.2 * dim ** -0.5 if scale is None else scale}


def right(heads=6, vdim=40, state=56, groups=3, norm_groups=4, conv=3):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": norm_groups, "conv": conv}


def parallel(a=None, b=None):
    return "parallel", {"left": a or left(), "right": b or right()}, 0


def dense(ff=136, limit=1.5):
    return {"kind": "dense", "ff": ff, "limit": limit}


def config(mixers, mlps, width=200, vocab=211, eps=0.06, streams=3, taps=4) -> dict:
    out = {"architecture": "Norusun", "canon": {"taps": taps}, "norm": {"eps": eps}, "vocab": vocab, "width": width, "streams": streams,
           "layers": [{"type": kind, "mixer": m, "mlp": f} for (kind, m, _), f in zip(mixers, mlps)]}
    out = json.loads(json.dumps(out))
    RANKS[json.dumps(out)] = [rank for _, _, rank in mixers]
    return out


RANKS: Dict[str, list] = {}     # ranks of the decay projections, which a configuration does not say


def weights(c: dict, seed: int = 11, dtype=torch.bfloat16) -> Dict[str, torch.Tensor]:
    """Checkpoint tensors; activations of order one, coefficients, biases, sinks and decays large enough to matter."""
    g = torch.Generator().manual_seed(seed)
    r = lambda *s: torch.randn(*s, generator=g)
    lin = lambda o, i: r(o, i) * i ** -0.5
    H, S, taps, w = c["width"], c["streams"], c["canon"]["taps"], {}
    one = lambda: torch.tensor(1.2) + 0.15 * r(())
    w["embed"], w["final.norm"], w["head"] = r(c["vocab"], H), one(), 3.0 * lin(c["vocab"], H)
    for i, (L, rank) in enumerate(zip(c["layers"], RANKS[json.dumps(c)])):
        p, m, f, q = f"l{i}.mix.", L["mixer"], L["mlp"], f"l{i}.mlp."
        for k in (1, 2) if f else (1,):
            w[f"l{i}.norm{k}"] = one()
            w[f"l{i}.hc{k}.in"] = 1.0 / S + 0.25 * r(S)
            w[f"l{i}.hc{k}.out"] = 0.8 + 0.3 * r(S)
            w[f"l{i}.hc{k}.mix"] = 0.8 * torch.eye(S) + 0.25 * r(S, S)
        w[f"l{i}.canon1"] = 0.3 * r(H, taps)
        if L["type"] == "wkv":
            n = m["heads"] * m["dim"]
            for s in "rkvgw":
                w[p + "mu." + s] = 0.5 + 0.4 * r(H)
            for s in "rkvg":
                w[p + s] = lin(n, H)
            w[p + "w1"], w[p + "w2"], w[p + "w0"] = 1.5 * lin(rank, H), 1.5 * lin(n, rank), -1.5 + 0.8 * r(n)
            w[p + "u"], w[p + "norm"], w[p + "o"] = 0.5 + 1.2 * r(m["heads"], m["dim"]), 1.0 + 0.3 * r(n), lin(H, n)
        elif L["type"] == "latent_attention":
            h, d, rd = m["heads"], m["dim"], m["rot_dim"]
            w[p + "dq"], w[p + "dkv"] = lin(m["q_rank"], H), 1.5 * lin(m["kv_rank"] + rd, H)
            w[p + "dq.norm"], w[p + "dkv.norm"] = 1.0 + 0.3 * r(m["q_rank"]), 1.0 + 0.3 * r(m["kv_rank"])
            w[p + "uq"], w[p + "uk"] = 1.6 * lin(h * (d + rd), m["q_rank"]), 1.3 * lin(h * d, m["kv_rank"])
            w[p + "uv"], w[p + "sink"] = 1.2 * lin(h * m["vdim"], m["kv_rank"]), 3.0 + 1.5 * r(h)
            w[p + "o"] = 2.0 * lin(H, h * m["vdim"])
        else:
            a, b = m["left"], m["right"]
            for n, o in (("q", a["heads"] * a["dim"]), ("k", a["kv_heads"] * a["dim"]), ("v", a["kv_heads"] * a["vdim"])):
                w[p + "left." + n] = lin(o, H)
            for n, k in (("q", a["heads"]), ("k", a["kv_heads"])):     # heads of unequal size, which a norm over all of them keeps
                w[p + "left." + n] *= (0.7 * r(k)).exp().repeat_interleave(a["dim"])[:, None]
            w[p + "left.q.norm"] = 1.6 + 0.4 * r(a["heads"] * a["dim"])
            w[p + "left.k.norm"] = 1.5 + 0.4 * r(a["kv_heads"] * a["dim"])
            w[p + "left.pb"], w[p + "left.o"] = -1.5 + 1.5 * r(a["heads"]), lin(H, a["heads"] * a["vdim"])
            n, ch = b["heads"] * b["vdim"], b["heads"] * b["vdim"] + 2 * b["groups"] * b["state"]
            w[p + "right.in"] = 1.3 * lin(n + ch + b["heads"], H)
            w[p + "right.conv"], w[p + "right.conv.b"] = r(ch, b["conv"]) * b["conv"] ** -0.5 + 0.3, 0.4 * r(ch)
            w[p + "right.dt_bias"], w[p + "right.A_log"], w[p + "right.D"] = -1.0 + 0.7 * r(b["heads"]), -0.5 + 0.7 * r(b["heads"]), 1.0 + 0.7 * r(b["heads"])
            w[p + "right.norm"], w[p + "right.o"] = 1.0 + 0.3 * r(n), lin(H, n)
            w[p + "left.out"], w[p + "right.out"] = 1.2 + 0.4 * r(H), 1.2 + 0.4 * r(H)
        if f:
            for n, o, k in (("gate", f["ff"], H), ("up", f["ff"], H), ("down", H, f["ff"])):
                w[q + n], w[q + n + ".b"] = 1.4 * lin(o, k), 0.6 * r(o)
    return {n: t.to(dtype).contiguous() for n, t in w.items()}


CASES = {
    # sizes the tensor-core kernels take; every mixer, with and without a feed-forward
    "regular": config([wkv(), latent(), parallel(), wkv(heads=2, dim=64, rank=24), parallel(left(heads=4, kv_heads=4, chunk=16), right(groups=1, norm_groups=6))],
                      [None, dense(), dense(ff=72, limit=0.8), dense(), None]),
    # values of another size than keys, many query heads on a key head, whole rotation, one stream, one tap (only the token itself)
    "values": config([parallel(left(heads=12, kv_heads=1, dim=128, vdim=96, rot_dims=128, chunk=130), right(heads=4, vdim=64, state=128, groups=4, norm_groups=1, conv=4)),
                      latent(heads=2, dim=96, rot_dim=32, vdim=128, q_rank=64, kv_rank=256, window=64), wkv(heads=1, dim=128, rank=40)],
                     [dense(ff=64), dense(ff=200, limit=3.0), None], width=136, vocab=152, streams=1, taps=1),
    # a latent of several chunks of value columns, expanded heads larger than the prompt kernel takes, many streams and taps
    "wide": config([latent(heads=20, dim=120, rot_dim=40, vdim=16, q_rank=40, kv_rank=320, window=129, scale=0.05), wkv(heads=7, dim=32, rank=8),
                    parallel(left(heads=4, kv_heads=2, dim=40, vdim=24, rot_dims=8, chunk=200), right(heads=2, vdim=128, state=64, groups=2, norm_groups=2, conv=6)),
                    latent(heads=72, dim=8, rot_dim=16, vdim=8, q_rank=64, kv_rank=136, window=200, scale=0.1)],
                   [dense(ff=96), None, None, dense(ff=40)], width=96, vocab=128, streams=5, taps=6),
    # nothing a multiple of 8
    "odd": config([wkv(heads=3, dim=13, rank=5), latent(heads=3, dim=13, rot_dim=6, vdim=11, q_rank=35, kv_rank=21, window=9),
                   parallel(left(heads=9, kv_heads=3, dim=22, vdim=13, rot_dims=10, chunk=7), right(heads=5, vdim=7, state=9, groups=5, norm_groups=5, conv=2))],
                  [dense(ff=51), dense(ff=33), dense(ff=9)], width=121, vocab=157, streams=2, taps=3),
    # values equal to 1: one head, one group, one position of a window and of a chunk, one pair of rotated dimensions
    "ones": config([parallel(left(heads=1, kv_heads=1, dim=16, vdim=8, rot_dims=2, chunk=1, scale=0.2), right(heads=1, vdim=8, state=8, groups=1, norm_groups=1, conv=1)),
                    latent(heads=1, dim=8, rot_dim=2, vdim=8, q_rank=8, kv_rank=8, window=1), wkv(heads=1, dim=8, rank=1)],
                   [dense(ff=8), None, dense(ff=16)], width=64, vocab=96, streams=2, taps=2, eps=1e-6),
}
