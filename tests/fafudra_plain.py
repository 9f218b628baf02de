"""Plain, slow Fafudra forward: the oracle of the hybrid-model tests.

One function per mechanism, written from the design's equations on dense tensors: no pages, no chunks, no batches and
no code of the package.  `Plain(config, weights)` takes the parsed config.json and a dict of tensors under their
checkpoint names; everything is computed in `dtype` (float64 by default), token by token where a recurrence is.

`flaws` plants a mistake (a name from FLAWS) so that a test can check that its inputs would show it.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

FLAWS = ("window_long", "window_short", "no_sink", "sink_scaled", "no_first", "first_short", "no_softcap", "value_rotated",
         "half_split_rotation", "no_embedding_in_loop", "no_step", "shared_pass_state", "no_decay", "state_16bit")


def rms_norm(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rotate_pairs(x: torch.Tensor, pos: torch.Tensor, dims: int, base: float, half_split: bool = False) -> torch.Tensor:
    """x [T, heads, d]; dimensions 2i and 2i + 1 of the first `dims` form a pair."""
    out = x.clone()
    for i in range(dims // 2):
        a = pos.to(x.dtype) * base ** (-2.0 * i / dims)
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        iu, iv = (i, i + dims // 2) if half_split else (2 * i, 2 * i + 1)
        u, v = x[..., iu], x[..., iv]
        out[..., iu] = u * c - v * s
        out[..., iv] = v * c + u * s
    return out


def visible(n: int, size: int, first: int) -> torch.Tensor:
    """[n, n]: row i may look at column j."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    return (j <= i) & ((i - j < size) | (j < first))


def attention(h, w, mx: dict, flaws=()) -> torch.Tensor:
    T, H, G, d = h.shape[0], mx["heads"], mx["kv_heads"], mx["dim"]
    q = (h @ w("q").T).view(T, H, d)
    k_raw = (h @ w("k").T).view(T, G, d)
    pos = torch.arange(T)
    hs = "half_split_rotation" in flaws
    q = rotate_pairs(q, pos, mx["rot"]["dims"], mx["rot"]["base"], hs)
    k = rotate_pairs(k_raw, pos, mx["rot"]["dims"], mx["rot"]["base"], hs)
    v = k if "value_rotated" in flaws else k_raw
    size, first = mx["mask"]["size"], mx["mask"]["keep_first"]
    size += ("window_long" in flaws) - ("window_short" in flaws)
    if "no_first" in flaws:
        first = 0
    if "first_short" in flaws:
        first = max(0, first - 1)
    see = visible(T, size, first)
    out = torch.empty(T, H, d, dtype=h.dtype)
    for hd in range(H):
        g = hd // (H // G)
        s = (q[:, hd] @ k[:, g].T) * mx["scale"]
        if "no_softcap" not in flaws:
            s = mx["softcap"] * torch.tanh(s / mx["softcap"])
        s = s.masked_fill(~see, float("-inf"))
        sink = w("sink")[hd] * (mx["scale"] if "sink_scaled" in flaws else 1.0)
        m = torch.maximum(s.max(-1).values, sink)
        e = torch.exp(s - m[:, None])
        den = e.sum(-1)
        if "no_sink" not in flaws:
            den = den + torch.exp(sink - m)
        out[:, hd] = (e / den[:, None]) @ v[:, g]
    return out.reshape(T, H * d) @ w("o").T


def gla(h, w, mx: dict, eps: float, flaws=(), state: Optional[torch.Tensor] = None) -> torch.Tensor:
    T, H, dk, dv = h.shape[0], mx["heads"], mx["dim"], mx["vdim"]
    q = (h @ w("q").T).view(T, H, dk) * dk ** -0.5
    k = (h @ w("k").T).view(T, H, dk)
    v = (h @ w("v").T).view(T, H, dv)
    z = ((h @ w("a1").T) @ w("a2").T + w("a2.b")).view(T, H, dk)
    alpha = torch.sigmoid(z) ** (1.0 / mx["tau"])
    if "no_decay" in flaws:
        alpha = torch.ones_like(alpha)
    S = torch.zeros(H, dk, dv, dtype=h.dtype) if state is None else state
    out = torch.empty(T, H, dv, dtype=h.dtype)
    for t in range(T):
        S.mul_(alpha[t][:, :, None]).add_(k[t][:, :, None] * v[t][:, None, :])
        if "state_16bit" in flaws:
            S.copy_(S.to(torch.bfloat16))
        out[t] = torch.einsum("hkv,hk->hv", S, q[t])
    o = rms_norm(out, eps) * w("norm")
    return (o.reshape(T, H * dv) * silu(h @ w("g").T)) @ w("o").T


def rglru(h, w, mx: dict, state: Optional[torch.Tensor] = None) -> torch.Tensor:
    T, W, nb = h.shape[0], mx["width"], mx["blocks"]
    taps = w("conv").shape[1]
    y = gelu_tanh(h @ w("y").T + w("y.b"))
    x = h @ w("x").T + w("x.b")
    padded = torch.cat([torch.zeros(taps - 1, W, dtype=h.dtype), x], 0)
    u = w("conv.b").expand(T, W).clone()
    for j in range(taps):
        u = u + padded[j:j + T] * w("conv")[:, j]
    ub = u.view(T, nb, W // nb)
    r = torch.sigmoid(torch.einsum("tbi,boi->tbo", ub, w("ra")) + w("ra.b")).reshape(T, W)
    i = torch.sigmoid(torch.einsum("tbi,boi->tbo", ub, w("ri")) + w("ri.b")).reshape(T, W)
    softplus = torch.logaddexp(w("lam"), torch.zeros((), dtype=h.dtype))
    a = torch.exp(-8.0 * r * softplus)
    S = torch.zeros(W, dtype=h.dtype) if state is None else state
    out = torch.empty(T, W, dtype=h.dtype)
    for t in range(T):
        S.copy_(a[t] * S + torch.sqrt(1.0 - a[t] ** 2) * i[t] * u[t])
        out[t] = S
    return (out * y) @ w("o").T


def feed_forward(h, w) -> torch.Tensor:
    return (silu(h @ w("gate").T) * (h @ w("up").T)) @ w("down").T


class Plain:
    def __init__(self, config: dict, weights: Dict[str, torch.Tensor], dtype=torch.float64, flaws=()):
        self.c, self.dtype, self.flaws = config, dtype, tuple(flaws)
        assert all(f in FLAWS for f in self.flaws)
        self.w = {n: t.to(dtype) for n, t in weights.items()}

    def order(self) -> List[tuple]:
        """(layer, pass or None) of every layer run."""
        n, lp = len(self.c["layers"]), self.c.get("loop")
        if not lp:
            return [(i, None) for i in range(n)]
        a, b = lp["start"], lp["stop"]
        return ([(i, None) for i in range(a)] + [(i, t) for t in range(lp["times"]) for i in range(a, b)]
                + [(i, None) for i in range(b, n)])

    def run(self, tokens: List[int], keep: Optional[list] = None) -> torch.Tensor:
        """Logits at every position; `keep` collects the residual stream after every layer run."""
        c, eps = self.c, self.c["norm"]["eps"]
        x0 = self.w["embed"][torch.tensor(tokens)]
        x = x0.clone()
        shared: Dict[int, torch.Tensor] = {}
        for i, t in self.order():
            if t is not None and i == c["loop"]["start"]:
                if t > 0 and "no_embedding_in_loop" not in self.flaws:
                    x = x + x0
                if "no_step" not in self.flaws:
                    x = x + self.w["loop.step"][t]
            L = c["layers"][i]
            h = rms_norm(x, eps) * (1.0 + self.w[f"l{i}.norm1"])
            mix = lambda n, i=i: self.w[f"l{i}.mix.{n}"]
            mx = L["mixer"]
            state = None
            if "shared_pass_state" in self.flaws and L["type"] == "gla":
                state = shared.setdefault(i, torch.zeros(mx["heads"], mx["dim"], mx["vdim"], dtype=self.dtype))
            if L["type"] == "attention":
                y = attention(h, mix, mx, self.flaws)
            elif L["type"] == "gla":
                y = gla(h, mix, mx, eps, self.flaws, state)
            else:
                y = rglru(h, mix, mx)
            if L.get("mlp"):
                y = y + feed_forward(h, lambda n, i=i: self.w[f"l{i}.mlp.{n}"])
            x = x + c["residual_mult"] * y
            if keep is not None:
                keep.append(x.clone())
        return (rms_norm(x, eps) * (1.0 + self.w["final.norm"])) @ self.w["embed"].T

    def greedy(self, prompt: List[int], n: int) -> List[int]:
        toks = list(prompt)
        for _ in range(n):
            toks.append(int(self.run(toks)[-1].argmax()))
        return toks[len(prompt):]
