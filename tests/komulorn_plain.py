"""Plain, slow Komulorn forward: the oracle of the tests of that design.

One function per mechanism, written from the design's equations on dense tensors: no pages, no sorted experts, no
batches and no code of the package.  `Plain(config, weights)` takes the parsed config.json and a dict of tensors under
their checkpoint names; everything is computed in `dtype` (float64 by default).

`flaws` plants a mistake (a name from FLAWS) so that a test can check that its inputs would show it.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

FLAWS = ("no_bias_q", "no_bias_k", "no_bias_v", "interleaved_rotation", "all_dims_rotated", "no_yarn", "yarn_unclipped",
         "no_yarn_gain", "no_gate", "own_kv_recomputed", "far_key_lost", "kv_unrotated", "weight_on_output", "no_weight",
         "renormalized", "one_expert_less", "relu_not_squared", "no_shared", "no_shared_gate", "no_softcap", "scale_by_dim")


def rms_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def yarn_frequencies(dims: int, base: float, sc: Optional[dict], flaws=()):
    """(list of dims / 2 frequencies, gain of cos and sin)."""
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not sc or "no_yarn" in flaws:
        return f, 1.0
    at = lambda turns: dims * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = math.floor(at(sc["fast"])), math.ceil(at(sc["slow"]))
    if "yarn_unclipped" not in flaws:
        lo, hi = max(lo, 0), min(hi, dims - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / sc["factor"] * ramp + fi * (1.0 - ramp))
    return out, 1.0 if "no_yarn_gain" in flaws else 0.1 * math.log(sc["factor"]) + 1.0


def rotate_half(x: torch.Tensor, rot: Optional[dict], flaws=()) -> torch.Tensor:
    """x [T, heads, d]: dimensions i and i + dims / 2 of the first `dims` form a pair."""
    if not rot:
        return x
    dims = x.shape[-1] // 2 * 2 if "all_dims_rotated" in flaws else rot["dims"]
    freq, gain = yarn_frequencies(dims, rot["base"], rot.get("scaling"), flaws)
    out = x.clone()
    pos = torch.arange(x.shape[0], dtype=x.dtype)
    for i, f in enumerate(freq):
        c, s = torch.cos(pos * f)[:, None] * gain, torch.sin(pos * f)[:, None] * gain
        iu, iv = (2 * i, 2 * i + 1) if "interleaved_rotation" in flaws else (i, i + dims // 2)
        u, v = x[..., iu], x[..., iv]
        out[..., iu] = u * c - v * s
        out[..., iv] = v * c + u * s
    return out


def keys_values(h, w, mx: dict, flaws=()):
    """What a layer's cache holds: rotated keys [T, G, dim] and values [T, G, vdim]."""
    T, G = h.shape[0], mx["kv_heads"]
    k, v = h @ w("k").T, h @ w("v").T
    if "no_bias_k" not in flaws:
        k = k + w("k.b")
    if "no_bias_v" not in flaws:
        v = v + w("v.b")
    k = k.view(T, G, mx["dim"])
    return k if "kv_unrotated" in flaws else rotate_half(k, mx.get("rot"), flaws), v.view(T, G, mx["vdim"])


def attention(h, w, mx: dict, k, v, flaws=()) -> torch.Tensor:
    T, H, G = h.shape[0], mx["heads"], mx["kv_heads"]
    q = h @ w("q").T
    if "no_bias_q" not in flaws:
        q = q + w("q.b")
    q = rotate_half(q.view(T, H, mx["dim"]), mx.get("rot"), flaws)
    scale = mx["dim"] ** -0.5 if "scale_by_dim" in flaws else mx["scale"]
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    see = j <= i
    if "far_key_lost" in flaws:
        see = see & ((i - j < 128) | (i < 128))
    gate = torch.sigmoid(h @ w("g").T)
    out = torch.empty(T, H, mx["vdim"], dtype=h.dtype)
    for hd in range(H):
        g = hd // (H // G)
        s = ((q[:, hd] @ k[:, g].T) * scale).masked_fill(~see, float("-inf"))
        out[:, hd] = torch.softmax(s, -1) @ v[:, g]
        if "no_gate" not in flaws:
            out[:, hd] *= gate[:, hd:hd + 1]
    return out.reshape(T, -1) @ w("o").T


def expert(h, up, down, flaws=()) -> torch.Tensor:
    a = torch.relu(h @ up.T)
    return (a if "relu_not_squared" in flaws else a * a) @ down.T


def experts(h, w, mlp: dict, flaws=(), margin: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Each token through its best experts, and through the shared one.  `margin` [T] is lowered to how far a token's router
    logits are from another choice."""
    top = mlp["router"]["top"] - ("one_expert_less" in flaws)
    z = h @ w("router").T
    s = torch.sigmoid(z)
    if margin is not None and mlp["router"]["top"] < z.shape[1]:
        best = z.sort(-1, descending=True).values
        margin.copy_(torch.minimum(margin, best[:, mlp["router"]["top"] - 1] - best[:, mlp["router"]["top"]]))
    val, idx = torch.topk(s, top, dim=-1)
    if "renormalized" in flaws:
        val = val / val.sum(-1, keepdim=True)
    if "no_weight" in flaws:
        val = torch.ones_like(val)
    out = torch.zeros_like(h)
    for e in idx.unique().tolist():
        t, k = (idx == e).nonzero(as_tuple=True)
        wt, x = val[t, k][:, None], h[t]
        y = expert(x if "weight_on_output" in flaws else wt * x, w(f"e{e}.up"), w(f"e{e}.down"), flaws)
        out[t] += wt * y if "weight_on_output" in flaws else y
    if mlp.get("shared") and "no_shared" not in flaws:
        y = expert(h, w("shared.up"), w("shared.down"), flaws)
        if "no_shared_gate" not in flaws:
            y = y * torch.sigmoid(h @ w("shared.sg").T)
        out = out + y
    return out


class Plain:
    def __init__(self, config: dict, weights: Dict[str, torch.Tensor], dtype=torch.float64, flaws=()):
        self.c, self.dtype, self.flaws = config, dtype, tuple(flaws)
        assert all(f in FLAWS for f in self.flaws)
        self.w = {n: t.to(dtype) for n, t in weights.items()}

    def run(self, tokens: List[int], keep: Optional[list] = None) -> torch.Tensor:
        """Logits at every position; `keep` collects the residual stream after every layer."""
        c, eps, fl = self.c, self.c["norm"]["eps"], self.flaws
        x = self.w["embed"][torch.tensor(tokens)]
        self.margin = torch.full((len(tokens),), math.inf, dtype=self.dtype)    # of the closest router decision
        cache: Dict[int, tuple] = {}
        for i, L in enumerate(c["layers"]):
            mix = lambda n, i=i: self.w[f"l{i}.mix.{n}"]
            mx = L["mixer"]
            h = rms_norm(x, self.w[f"l{i}.norm1"], eps)
            src = mx.get("kv_from")
            if src is None:
                cache[i] = keys_values(h, mix, mx, fl)
            elif "own_kv_recomputed" in fl:          # the other layer's projections on this layer's input
                cache[i] = keys_values(h, lambda n, j=src: self.w[f"l{j}.mix.{n}"], mx, fl)
            else:
                cache[i] = cache[src]
            x = x + attention(h, mix, mx, *cache[i], fl)
            if L.get("mlp"):
                h = rms_norm(x, self.w[f"l{i}.norm2"], eps)
                x = x + experts(h, lambda n, i=i: self.w[f"l{i}.mlp.{n}"], L["mlp"], fl, self.margin)
            if keep is not None:
                keep.append(x.clone())
        z = rms_norm(x, self.w["final.norm"], eps) @ self.w["head"].T
        cap = c.get("logit_softcap")
        return cap * torch.tanh(z / cap) if cap and "no_softcap" not in fl else z

    def greedy(self, prompt: List[int], n: int) -> List[int]:
        toks = list(prompt)
        for _ in range(n):
            toks.append(int(self.run(toks)[-1].argmax()))
        return toks[len(prompt):]
