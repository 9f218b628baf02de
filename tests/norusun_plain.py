"""Plain, slow Norusun forward: the oracle of the tests of that design.

One function per mechanism, written from the design's equations on dense tensors, token by token where there is a state: no
pages, no slots, no latent cache, no chunks, no batches and no code of the package.  `Plain(config, weights)` takes the parsed
config.json and a dict of tensors under their checkpoint names; everything is computed in `dtype` (float64 by default).

`flaws` plants a mistake (a name from FLAWS) so that a test can check that its inputs would show it.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch
import torch.nn.functional as F

FLAWS = ("no_gain", "eps_outside", "conv_reversed", "conv_no_residual", "conv_early", "conv_lost",
         "mix_transposed", "no_mix", "out_ones", "in_ones", "new_streams_read", "last_stream_only",
         "no_shift", "mu_swapped", "no_bonus", "bonus_everywhere", "no_decay", "decay_before", "decay_once", "no_decay_tanh", "no_decay_bias",
         "no_head_norm", "whole_norm", "no_wkv_gate",
         "no_latent_norm", "no_query_latent_norm", "half_rotation", "no_rotation", "rotated_first", "window_off_by_one", "no_window",
         "no_sink", "sink_scaled", "scale_by_dim",
         "norm_per_head", "no_query_norm", "no_key_norm", "norm_after_rotation", "pair_rotation", "whole_rotation", "chunk_off_by_one",
         "no_chunks", "softmax", "no_weight_bias", "weights_normalised", "kv_head_interleaved",
         "no_conv", "no_conv_bias", "no_silu", "no_dt_bias", "dt_not_on_input", "group_interleaved", "no_skip", "gate_after_norm",
         "one_norm_group", "state_before", "sum_not_half", "no_out_norm",
         "no_limit", "up_one_sided", "plain_silu", "no_plus_one", "no_up_bias", "no_down_bias")


def rms(x: torch.Tensor, eps: float, flaws=()) -> torch.Tensor:
    if "eps_outside" in flaws:
        return x / (torch.sqrt((x * x).mean(-1, keepdim=True)) + eps)
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def scalar_norm(x, g, eps: float, flaws=()) -> torch.Tensor:
    return rms(x, eps, flaws) * (1.0 if "no_gain" in flaws else g)


def causal_conv(x: torch.Tensor, w: torch.Tensor, flaws=()) -> torch.Tensor:
    """x [T, channels], w [channels, taps]; the last column weighs the current token, zeros before the start."""
    T, taps = x.shape[0], w.shape[1]
    out = torch.zeros_like(x)
    for j in range(taps):
        back = j if "conv_reversed" in flaws else taps - 1 - j
        if "conv_early" in flaws:
            back += 1
        if "conv_lost" in flaws and back == taps - 1 and taps > 1:
            continue
        if back < T:
            out[back:] += w[:, j] * x[:T - back]
    return out


def streams_in(xs: torch.Tensor, a: torch.Tensor, flaws=()) -> torch.Tensor:
    """xs [streams, T, width] -> the sublayer's input."""
    return xs.sum(0) if "in_ones" in flaws else torch.einsum("s,stw->tw", a, xs)


def streams_out(xs: torch.Tensor, mix: torch.Tensor, out: torch.Tensor, y: torch.Tensor, flaws=()) -> torch.Tensor:
    """Stream t becomes sum_s mix[s, t] x_s + out[t] y."""
    if "mix_transposed" in flaws:
        mix = mix.T
    if "no_mix" in flaws:
        mix = torch.eye(len(mix), dtype=mix.dtype)
    if "out_ones" in flaws:
        out = torch.ones_like(out)
    if "new_streams_read" in flaws:      # one after the other, later ones from already changed ones
        xs = xs.clone()
        for t in range(len(xs)):
            xs[t] = torch.einsum("s,stw->tw", mix[:, t], xs) + out[t] * y
        return xs
    return torch.einsum("su,stw->utw", mix, xs) + out[:, None, None] * y


def rotate(x: torch.Tensor, dims: int, base: float, interleaved: bool) -> torch.Tensor:
    """x [T, ..., d]: pairs (2i, 2i + 1) or (i, i + dims / 2) of the first `dims` dimensions turn by p base^(-2i / dims)."""
    out = x.clone()
    pos = torch.arange(x.shape[0], dtype=x.dtype).view(-1, *([1] * (x.dim() - 2)))
    for i in range(dims // 2):
        a = pos * base ** (-2.0 * i / dims)
        c, s = torch.cos(a), torch.sin(a)
        iu, iv = (2 * i, 2 * i + 1) if interleaved else (i, i + dims // 2)
        u, v = x[..., iu], x[..., iv]
        out[..., iu] = u * c - v * s
        out[..., iv] = v * c + u * s
    return out


# ---------------------------------------------------------------------------------------------- time mixing
def shifted(h: torch.Tensor) -> torch.Tensor:
    return torch.cat([torch.zeros_like(h[:1]), h[:-1]])


def wkv_recurrence(r, k, v, decay, u, flaws=()) -> torch.Tensor:
    """r, k, v, decay [T, heads, dim], u [heads, dim]: o [T, heads, dim]."""
    T, H, n = r.shape
    S = torch.zeros(H, n, v.shape[2], dtype=r.dtype)
    out = torch.empty(T, H, v.shape[2], dtype=r.dtype)
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        bonus = 1.0 if "no_bonus" in flaws else u[:, :, None]
        if "decay_before" in flaws:
            S = decay[t][:, :, None] * S
        out[t] = torch.einsum("hkv,hk->hv", S + bonus * kv, r[t])
        if "bonus_everywhere" in flaws:
            kv = bonus * kv
        S = (S if "decay_before" in flaws else decay[t][:, :, None] * S) + kv
    return out


def wkv(h, w, mx: dict, eps: float, flaws=()) -> torch.Tensor:
    T, H, n = h.shape[0], mx["heads"], mx["dim"]
    prev = h if "no_shift" in flaws else shifted(h)

    def mixed(s):
        mu = w("mu." + s)
        return h + (prev - h) * (1.0 - mu if "mu_swapped" in flaws else mu)
    r, k, v = ((mixed(s) @ w(s).T).view(T, H, n) for s in "rkv")
    gate = F.silu(mixed("g") @ w("g").T)
    low = mixed("w") @ w("w1").T
    z = (low if "no_decay_tanh" in flaws else torch.tanh(low)) @ w("w2").T
    if "no_decay_bias" not in flaws:
        z = z + w("w0")
    decay = torch.exp(-torch.exp(z)).view(T, H, n)
    if "no_decay" in flaws:
        decay = torch.ones_like(decay)
    if "decay_once" in flaws:
        decay = torch.exp(z).clamp(max=1.0).view(T, H, n)
    o = wkv_recurrence(r, k, v, decay, w("u"), flaws)
    if "whole_norm" in flaws:
        o = rms(o.reshape(T, -1), eps).view(T, H, n)
    elif "no_head_norm" not in flaws:
        o = rms(o, eps, flaws)
    o = o.reshape(T, -1) * w("norm")
    return (o if "no_wkv_gate" in flaws else o * gate) @ w("o").T


# ---------------------------------------------------------------------------------------------- latent attention
def sink_attention(q, k, v, scale: float, window: int, sink, flaws=()) -> torch.Tensor:
    """One head: softmax over the last `window` keys with e^sink in the denominator."""
    T = q.shape[0]
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    see = j <= i
    if "no_window" not in flaws:
        see = see & (i - j < window + ("window_off_by_one" in flaws))
    s = ((q @ k.T) * scale).masked_fill(~see, float("-inf"))
    if "no_sink" in flaws:
        return torch.softmax(s, -1) @ v
    sk = (sink * scale if "sink_scaled" in flaws else sink).expand(T, 1)
    return torch.softmax(torch.cat([s, sk], 1), -1)[:, :T] @ v


def latent_attention(h, w, mx: dict, eps: float, flaws=()) -> torch.Tensor:
    T, H, d, r, nv, rank = h.shape[0], mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"], mx["kv_rank"]
    turn = lambda x: x if "no_rotation" in flaws else rotate(x, r, mx["rot"]["base"], "half_rotation" not in flaws)
    cq = h @ w("dq").T
    if "no_query_latent_norm" not in flaws:
        cq = rms(cq, eps, flaws) * w("dq.norm")
    q = (cq @ w("uq").T).view(T, H, d + r)
    ckv = h @ w("dkv").T
    c, kr = ckv[:, :rank], turn(ckv[:, rank:])
    if "no_latent_norm" not in flaws:
        c = rms(c, eps, flaws) * w("dkv.norm")
    k, v = (c @ w("uk").T).view(T, H, d), (c @ w("uv").T).view(T, H, nv)
    qn, qr = (q[..., r:], turn(q[..., :r])) if "rotated_first" in flaws else (q[..., :d], turn(q[..., d:]))
    scale = d ** -0.5 if "scale_by_dim" in flaws else mx["scale"]
    out = torch.empty(T, H, nv, dtype=h.dtype)
    for hd in range(H):
        out[:, hd] = sink_attention(torch.cat([qn[:, hd], qr[:, hd]], -1), torch.cat([k[:, hd], kr], -1), v[:, hd], scale,
                                    mx["mask"]["size"], w("sink")[hd], flaws)
    return out.reshape(T, -1) @ w("o").T


# ---------------------------------------------------------------------------------------------- attention without softmax
def sigmoid_attention(q, k, v, scale: float, chunk: int, bias, flaws=()) -> torch.Tensor:
    """One head: the keys of the position's own chunk, each weighed by the sigmoid of its score."""
    T = q.shape[0]
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    see = j <= i
    if "no_chunks" not in flaws:
        one = "chunk_off_by_one" in flaws
        see = see & ((i + one) // chunk == (j + one) // chunk)
    s = (q @ k.T) * scale
    if "no_weight_bias" not in flaws:
        s = s + bias
    if "softmax" in flaws:
        return torch.softmax(s.masked_fill(~see, float("-inf")), -1) @ v
    a = torch.sigmoid(s) * see
    if "weights_normalised" in flaws:
        a = a / a.sum(-1, keepdim=True)
    return a @ v


def chunked_attention(h, w, mx: dict, eps: float, flaws=()) -> torch.Tensor:
    T, H, G, d = h.shape[0], mx["heads"], mx["kv_heads"], mx["dim"]
    q, k, v = h @ w("q").T, h @ w("k").T, (h @ w("v").T).view(T, G, mx["vdim"])
    dims = d if "whole_rotation" in flaws else mx["rot"]["dims"]
    turn = lambda x: rotate(x, dims, mx["rot"]["base"], "pair_rotation" in flaws)

    def normed(x, heads, name):
        if f"no_{name}_norm" in flaws:
            return turn(x.view(T, heads, d))
        weight = w("q.norm" if name == "query" else "k.norm")
        if "norm_per_head" in flaws:
            return turn(rms(x.view(T, heads, d), eps) * weight.view(heads, d))
        if "norm_after_rotation" in flaws:
            return (rms(turn(x.view(T, heads, d)).reshape(T, -1), eps) * weight).view(T, heads, d)
        return turn((rms(x, eps, flaws) * weight).view(T, heads, d))
    q, k = normed(q, H, "query"), normed(k, G, "key")
    out = torch.empty(T, H, mx["vdim"], dtype=h.dtype)
    for hd in range(H):
        g = hd % G if "kv_head_interleaved" in flaws else hd // (H // G)
        out[:, hd] = sigmoid_attention(q[:, hd], k[:, g], v[:, g], mx["scale"], mx["mask"]["size"], w("pb")[hd], flaws)
    return out.reshape(T, -1) @ w("o").T


# ---------------------------------------------------------------------------------------------- state space
def ssd_recurrence(x, B, C, dt, rate, skip, flaws=()) -> torch.Tensor:
    """x [T, heads, vdim], B and C [T, groups, state], dt [T, heads]: S <- e^(-rate dt) S + dt B x^T, y = S^T C + skip x."""
    T, H, P = x.shape
    G = B.shape[1]
    group = [h % G if "group_interleaved" in flaws else h // (H // G) for h in range(H)]
    S = torch.zeros(H, B.shape[2], P, dtype=x.dtype)
    y = torch.empty(T, H, P, dtype=x.dtype)
    for t in range(T):
        before = S
        step = torch.ones_like(dt[t]) if "dt_not_on_input" in flaws else dt[t]
        S = torch.exp(-rate * dt[t])[:, None, None] * S + step[:, None, None] * B[t, group][:, :, None] * x[t][:, None, :]
        y[t] = torch.einsum("hnp,hn->hp", before if "state_before" in flaws else S, C[t, group])
        if "no_skip" not in flaws:
            y[t] += skip[:, None] * x[t]
    return y


def state_space(h, w, mx: dict, eps: float, flaws=()) -> torch.Tensor:
    T, H, P, N, G = h.shape[0], mx["heads"], mx["vdim"], mx["state"], mx["groups"]
    inner = H * P
    z, xbc, dt = torch.split(h @ w("in").T, [inner, inner + 2 * G * N, H], -1)
    if "no_conv" not in flaws:
        xbc = causal_conv(xbc, w("conv"))
        if "no_conv_bias" not in flaws:
            xbc = xbc + w("conv.b")
    if "no_silu" not in flaws:
        xbc = F.silu(xbc)
    x, B, C = torch.split(xbc, [inner, G * N, G * N], -1)
    dt = F.softplus(dt if "no_dt_bias" in flaws else dt + w("dt_bias"), threshold=1e9)
    y = ssd_recurrence(x.reshape(T, H, P), B.reshape(T, G, N), C.reshape(T, G, N), dt, torch.exp(w("A_log")), w("D"), flaws).reshape(T, -1)
    groups = 1 if "one_norm_group" in flaws else mx["norm_groups"]
    norm = lambda a: rms(a.view(T, groups, -1), eps, flaws).reshape(T, -1) * w("norm")
    y = norm(y) * F.silu(z) if "gate_after_norm" in flaws else norm(y * F.silu(z))
    return y @ w("o").T


def side_by_side(h, w, mx: dict, eps: float, flaws=()) -> torch.Tensor:
    a = chunked_attention(h, lambda n: w("left." + n), mx["left"], eps, flaws)
    b = state_space(h, lambda n: w("right." + n), mx["right"], eps, flaws)
    if "no_out_norm" not in flaws:
        a, b = rms(a, eps, flaws) * w("left.out"), rms(b, eps, flaws) * w("right.out")
    return (a + b) * (1.0 if "sum_not_half" in flaws else 0.5)


# ---------------------------------------------------------------------------------------------- feed-forward
def clamped_ff(h, w, limit: float, flaws=()) -> torch.Tensor:
    g, u = h @ w("gate").T + w("gate.b"), h @ w("up").T
    if "no_up_bias" not in flaws:
        u = u + w("up.b")
    if "no_limit" not in flaws:
        g = g.clamp(max=limit)
        u = u.clamp(max=limit) if "up_one_sided" in flaws else u.clamp(-limit, limit)
    y = g * torch.sigmoid((1.0 if "plain_silu" in flaws else 1.702) * g) * (u + (0.0 if "no_plus_one" in flaws else 1.0))
    return y @ w("down").T + (0.0 if "no_down_bias" in flaws else w("down.b"))


MIXERS = {"wkv": wkv, "latent_attention": latent_attention, "parallel": side_by_side}


class Plain:
    """`rounded`: a shorter type that what enters and leaves every sublayer is rounded to, for an idea of how much rounding alone
    changes a position's logits."""

    def __init__(self, config: dict, weights: Dict[str, torch.Tensor], dtype=torch.float64, flaws=(), rounded=None):
        self.c, self.dtype, self.flaws, self.rounded = config, dtype, tuple(flaws), rounded
        assert all(f in FLAWS for f in self.flaws)
        self.w = {n: t.to(dtype) for n, t in weights.items()}

    def run(self, tokens: List[int], keep: Optional[list] = None) -> torch.Tensor:
        """Logits at every position; `keep` collects the sum of the streams after every layer."""
        c, eps, fl = self.c, self.c["norm"]["eps"], self.flaws
        short = lambda t: t if self.rounded is None else t.to(self.rounded).to(t.dtype)
        x = self.w["embed"][torch.tensor(tokens)]
        xs = torch.stack([x] * c["streams"])
        for i, L in enumerate(c["layers"]):
            mix = lambda n, i=i: self.w[f"l{i}.mix.{n}"]
            mlp = lambda n, i=i: self.w[f"l{i}.mlp.{n}"]
            for q in (1, 2):
                if q == 2 and not L.get("mlp"):
                    continue
                hc = {n: self.w[f"l{i}.hc{q}.{n}"] for n in ("in", "out", "mix")}
                h = short(scalar_norm(streams_in(xs, hc["in"], fl), self.w[f"l{i}.norm{q}"], eps, fl))
                if q == 2:
                    y = clamped_ff(h, mlp, L["mlp"]["limit"], fl)
                else:
                    conv = causal_conv(h, self.w[f"l{i}.canon1"], fl)
                    h = short(conv if "conv_no_residual" in fl else h + conv)
                    y = MIXERS[L["type"]](h, mix, L["mixer"], eps, fl)
                xs = streams_out(xs, hc["mix"], hc["out"], short(y), fl)
            if keep is not None:
                keep.append(xs.sum(0))
        x = xs[-1] if "last_stream_only" in fl else xs.sum(0)
        return scalar_norm(x, self.w["final.norm"], eps, fl) @ self.w["head"].T

    def greedy(self, prompt: List[int], n: int) -> List[int]:
        toks = list(prompt)
        for _ in range(n):
            toks.append(int(self.run(toks)[-1].argmax()))
        return toks[len(prompt):]
