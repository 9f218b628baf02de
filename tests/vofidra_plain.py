"""Plain, slow Vofidra forward: the oracle of the tests of that design.

One function per mechanism, written from the design's equations on dense tensors: no pages, no latent cache, no absorbed
projections, no sorted experts, no batches and no code of the package.  `Plain(config, weights)` takes the parsed
config.json and a dict of tensors under their checkpoint names; everything is computed in `dtype` (float64 by default).

`flaws` plants a mistake (a name from FLAWS) so that a test can check that its inputs would show it.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

FLAWS = ("no_alpha", "no_norm_bias", "no_tanh", "mix_transposed", "no_mix", "out_ones", "in_ones", "new_streams_read", "last_stream_only",
         "no_query_norm", "no_key_norm", "no_temperature", "temperature_from_p", "bias_scaled", "no_bias", "bias_off_by_one",
         "bias_not_logarithmic", "far_key_lost", "kv_head_interleaved",
         "no_latent_norm", "no_query_latent_norm", "no_rotation", "interleaved_rotation", "rotated_first", "rotated_key_normed",
         "no_gate", "scale_by_dim",
         "no_correction", "weights_corrected", "not_renormalized", "no_groups", "dropped_groups_zero", "identity_nothing",
         "identity_unweighted", "one_expert_less", "group_by_sum", "no_softcap")


def dyt(x: torch.Tensor, w: torch.Tensor, b: torch.Tensor, alpha: torch.Tensor, flaws=()) -> torch.Tensor:
    """tanh(alpha x) w + b"""
    z = x if "no_alpha" in flaws else alpha * x
    y = (z if "no_tanh" in flaws else torch.tanh(z)) * w
    return y if "no_norm_bias" in flaws else y + b


def rms_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


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


def rotate_half(x: torch.Tensor, dims: int, base: float, flaws=()) -> torch.Tensor:
    """x [T, ..., d]: dimensions i and i + dims / 2 of the first `dims` form a pair."""
    if "no_rotation" in flaws:
        return x
    out = x.clone()
    pos = torch.arange(x.shape[0], dtype=x.dtype).view(-1, *([1] * (x.dim() - 2)))
    for i in range(dims // 2):
        a = pos * base ** (-2.0 * i / dims)
        c, s = torch.cos(a), torch.sin(a)
        iu, iv = (2 * i, 2 * i + 1) if "interleaved_rotation" in flaws else (i, i + dims // 2)
        u, v = x[..., iu], x[..., iv]
        out[..., iu] = u * c - v * s
        out[..., iv] = v * c + u * s
    return out


def softmax_values(q, k, v, scale: float, bias: Optional[torch.Tensor] = None, flaws=()) -> torch.Tensor:
    """One head: q, k [T, d], v [T, n], causal; `bias` [T, T] is added to the scaled scores."""
    T = q.shape[0]
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    see = j <= i
    if "far_key_lost" in flaws:
        see = see & ((i - j < 128) | (i < 128))
    s = (q @ k.T) * scale
    if bias is not None and "no_bias" not in flaws:
        s = s + (scale * bias if "bias_scaled" in flaws else bias)
    return torch.softmax(s.masked_fill(~see, float("-inf")), -1) @ v


def bucket(n: int, rows: int, far: int, flaws=()) -> int:
    """Distances below rows / 2 have a row each, longer ones share rows on a logarithmic scale up to distance `far`."""
    if "bias_off_by_one" in flaws:
        n += 1
    half = rows // 2
    if n < half:
        return n
    if "bias_not_logarithmic" in flaws:
        return min(rows - 1, half + (n - half) * (rows - half) // (far - half))
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (rows - half)))


def temperature(T: int, spec: Optional[dict], dtype, flaws=()) -> torch.Tensor:
    if not spec or "no_temperature" in flaws:
        return torch.ones(T, dtype=dtype)
    one = 0 if "temperature_from_p" in flaws else 1
    return torch.tensor([1.0 + spec["coef"] * math.log((p + one) // spec["every"] + 1) for p in range(T)], dtype=dtype)


def attention(h, w, mx: dict, eps: float, flaws=()) -> torch.Tensor:
    T, H, G, d = h.shape[0], mx["heads"], mx["kv_heads"], mx["dim"]
    q, k, v = (h @ w("q").T).view(T, H, d), (h @ w("k").T).view(T, G, d), (h @ w("v").T).view(T, G, mx["vdim"])
    if "no_query_norm" not in flaws:
        q = rms_norm(q, w("q.norm"), eps)
    if "no_key_norm" not in flaws:
        k = rms_norm(k, w("k.norm"), eps)
    q = q * temperature(T, mx.get("q_temp"), h.dtype, flaws)[:, None, None]
    scale = d ** -0.5 if "scale_by_dim" in flaws else mx["scale"]
    rel = w("rel")
    rows = torch.tensor([bucket(n, rel.shape[0], mx["bias_max"], flaws) for n in range(T)])
    dist = (torch.arange(T)[:, None] - torch.arange(T)[None, :]).clamp(min=0)
    out = torch.empty(T, H, mx["vdim"], dtype=h.dtype)
    for hd in range(H):
        g = hd % G if "kv_head_interleaved" in flaws else hd // (H // G)
        out[:, hd] = softmax_values(q[:, hd], k[:, g], v[:, g], scale, rel[rows, hd][dist], flaws)
    return out.reshape(T, -1) @ w("o").T


def latent_attention(h, w, mx: dict, eps: float, flaws=()) -> torch.Tensor:
    T, H, d, r, nv, rank = h.shape[0], mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"], mx["kv_rank"]
    base = mx["rot"]["base"]
    cq = h @ w("dq").T
    if "no_query_latent_norm" not in flaws:
        cq = rms_norm(cq, w("dq.norm"), eps)
    q = (cq @ w("uq").T).view(T, H, d + r)
    ckv = h @ w("dkv").T
    c, kr = ckv[:, :rank], ckv[:, rank:]
    if "no_latent_norm" not in flaws:
        c = rms_norm(c, w("dkv.norm"), eps)
    if "rotated_key_normed" in flaws:
        kr = rms_norm(kr, torch.ones(r, dtype=h.dtype), eps)
    k, v = (c @ w("uk").T).view(T, H, d), (c @ w("uv").T).view(T, H, nv)
    kr = rotate_half(kr, r, base, flaws)
    if "rotated_first" in flaws:
        qr, qn = rotate_half(q[..., :r], r, base, flaws), q[..., r:]
    else:
        qn, qr = q[..., :d], rotate_half(q[..., d:], r, base, flaws)
    gate = torch.sigmoid(h @ w("g").T)
    scale = d ** -0.5 if "scale_by_dim" in flaws else mx["scale"]
    out = torch.empty(T, H, nv, dtype=h.dtype)
    for hd in range(H):
        out[:, hd] = softmax_values(torch.cat([qn[:, hd], qr[:, hd]], -1), torch.cat([k[:, hd], kr], -1), v[:, hd], scale, None, flaws)
        if "no_gate" not in flaws:
            out[:, hd] *= gate[:, hd:hd + 1]
    return out.reshape(T, -1) @ w("o").T


def gated_ff(h, gate, up, down) -> torch.Tensor:
    z = h @ gate.T
    return (z * torch.sigmoid(z) * (h @ up.T)) @ down.T


def route(z: torch.Tensor, correction: torch.Tensor, router: dict, flaws=()):
    """Router logits of one token -> (expert, weight) pairs, and how far the choice is from another one."""
    n = z.numel()
    top = router["top"] - ("one_expert_less" in flaws)
    s = torch.softmax(z, -1)
    choice = s if "no_correction" in flaws else s + correction
    margin = math.inf
    groups = router.get("groups")
    if groups and "no_groups" not in flaws:
        size = n // groups["count"]
        per = choice.view(groups["count"], size)
        gs = per.sum(-1) if "group_by_sum" in flaws else per.max(-1).values
        order = gs.sort(descending=True)
        if groups["keep"] < groups["count"]:
            margin = float(order.values[groups["keep"] - 1] - order.values[groups["keep"]])
        keep = torch.zeros(groups["count"], dtype=torch.bool)
        keep[order.indices[:groups["keep"]]] = True
        lost = 0.0 if "dropped_groups_zero" in flaws else float("-inf")
        choice = choice.masked_fill(~keep.repeat_interleave(size), lost)
    order = choice.sort(descending=True)
    if top < n:
        margin = min(margin, float(order.values[top - 1] - order.values[top]))
    idx = order.indices[:top]
    wt = (choice if "weights_corrected" in flaws else s)[idx]
    if "not_renormalized" not in flaws:
        wt = wt / (wt.sum() + 1e-20)
    return list(zip(idx.tolist(), wt)), margin


def experts(h, w, mlp: dict, flaws=(), margin: Optional[torch.Tensor] = None) -> torch.Tensor:
    """`margin` [T] is lowered to how far a token's choice scores are from another choice."""
    r = mlp["router"]
    z = h @ w("router").T
    out = torch.zeros_like(h)
    rows: Dict[int, list] = {}
    for t in range(h.shape[0]):
        pairs, m = route(z[t], w("correction"), r, flaws)
        if margin is not None:
            margin[t] = min(float(margin[t]), m)
        for e, wt in pairs:
            rows.setdefault(e, []).append((t, wt))
    for e, tw in rows.items():
        t = torch.tensor([a for a, _ in tw])
        wt = torch.stack([b for _, b in tw])[:, None]
        if e >= r["experts"]:
            if "identity_nothing" not in flaws:
                out[t] += h[t] * (1.0 if "identity_unweighted" in flaws else wt)
        else:
            out[t] += wt * gated_ff(h[t], w(f"e{e}.gate"), w(f"e{e}.up"), w(f"e{e}.down"))
    return out


class Plain:
    def __init__(self, config: dict, weights: Dict[str, torch.Tensor], dtype=torch.float64, flaws=()):
        self.c, self.dtype, self.flaws = config, dtype, tuple(flaws)
        assert all(f in FLAWS for f in self.flaws)
        self.w = {n: t.to(dtype) for n, t in weights.items()}

    def norm(self, name: str, x: torch.Tensor) -> torch.Tensor:
        return dyt(x, self.w[name], self.w[name + ".b"], self.w[name + ".alpha"], self.flaws)

    def run(self, tokens: List[int], keep: Optional[list] = None) -> torch.Tensor:
        """Logits at every position; `keep` collects the sum of the streams after every layer."""
        c, eps, fl = self.c, self.c["norm"]["eps"], self.flaws
        x = self.w["embed"][torch.tensor(tokens)]
        xs = torch.stack([x] * c["streams"])
        self.margin = torch.full((len(tokens),), math.inf, dtype=self.dtype)    # of the closest router decision
        for i, L in enumerate(c["layers"]):
            mix = lambda n, i=i: self.w[f"l{i}.mix.{n}"]
            mlp = lambda n, i=i: self.w[f"l{i}.mlp.{n}"]
            for q in (1, 2):
                hc = {n: self.w.get(f"l{i}.hc{q}.{n}") for n in ("in", "out", "mix")}
                if q == 2 and not L.get("mlp"):
                    continue
                h = self.norm(f"l{i}.norm{q}", streams_in(xs, hc["in"], fl))
                if q == 2 and L["mlp"]["kind"] == "dense":
                    y = gated_ff(h, mlp("gate"), mlp("up"), mlp("down"))
                elif q == 2:
                    y = experts(h, mlp, L["mlp"], fl, self.margin)
                else:
                    y = {"attention": attention, "latent_attention": latent_attention}[L["type"]](h, mix, L["mixer"], eps, fl)
                xs = streams_out(xs, hc["mix"], hc["out"], y, fl)
            if keep is not None:
                keep.append(xs.sum(0))
        x = xs[-1] if "last_stream_only" in fl else xs.sum(0)
        z = self.norm("final.norm", x) @ self.w["head"].T
        cap = c.get("logit_softcap")
        return cap * torch.tanh(z / cap) if cap and "no_softcap" not in fl else z

    def greedy(self, prompt: List[int], n: int) -> List[int]:
        toks = list(prompt)
        for _ in range(n):
            toks.append(int(self.run(toks)[-1].argmax()))
        return toks[len(prompt):]
