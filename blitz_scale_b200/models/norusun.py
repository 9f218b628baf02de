"""Norusun: pre-norm layers over several residual streams (hyper-connections, RMS norms with one number each) whose mixers read their
input plus a short causal convolution of it.  Mixers: linear attention with a token shift, a decay that depends on the token and a
bonus for the current token; latent attention in a sliding window with a sink; attention in chunks whose weights are sigmoids,
side by side with a state-space recurrence.  Gated feed-forwards with biases and a clamped unit; an untied head.

This file is what is specific to the design: how its config.json and its tensor names map onto the records of
hybrid_config.py.  Linear weights come as [out, in] and are stored as [in, out].
"""
from __future__ import annotations

from typing import Dict, Iterable, Mapping, Optional, Tuple

import torch

from .hybrid_config import (AttentionMixer, ClampedUnit, HybridConfig, LatentAttentionMixer, LayerSpec, ParallelMixer, SSDMixer,
                            WKVMixer)
from .weights import WeightSegment

ARCHITECTURE = "Norusun"


def _whole(x) -> int:
    if int(x) != x:
        raise ValueError(f"{x} is not a whole number")
    return int(x)


def _mixer(i: int, kind: str, m: dict, width: int, shapes: Mapping[str, Tuple[int, ...]]):
    p = f"l{i}.mix."
    if kind == "wkv":
        rank = shapes[p + "w1"][0] if p + "w1" in shapes else m["rank"]
        return WKVMixer(hidden=width, heads=m["heads"], dim=m["dim"], rank=rank)
    if kind == "latent_attention":
        if m["rot"]["dims"] != m["rot_dim"]:
            raise ValueError(f"layer {i}: the rotated part has {m['rot_dim']} dimensions, the rotation {m['rot']['dims']}")
        rank = m["q_rank"] if "q_rank" in m else shapes[p + "dq"][0]
        return LatentAttentionMixer(heads=m["heads"], dim=m["dim"], rot_dim=m["rot_dim"], vdim=m["vdim"], q_rank=rank, kv_rank=m["kv_rank"],
                                    scale=float(m["scale"]), rot_base=float(m["rot"]["base"]), gate=False, interleaved=True,
                                    window=_whole(m["mask"]["size"]), sink=True)
    if kind == "parallel":
        a, s = m["left"], m["right"]
        left = AttentionMixer(heads=a["heads"], kv_heads=a["kv_heads"], dim=a["dim"], value_dim=a["vdim"], scale=float(a["scale"]),
                              rot_dims=a["rot"]["dims"], rot_base=float(a["rot"]["base"]), interleaved=False, window=_whole(a["mask"]["size"]),
                              whole_norm=True, chunked=True, sigmoid=True)
        right = SSDMixer(heads=s["heads"], vdim=s["vdim"], state=s["state"], groups=s["groups"], taps=s["conv"], norm_groups=s["norm_groups"])
        return ParallelMixer(width, left, right)
    raise ValueError(f"layer {i}: unknown mixer {kind!r}")


def _layer(i: int, L: dict, width: int, shapes: Mapping[str, Tuple[int, ...]]) -> LayerSpec:
    mixer, f = _mixer(i, L["type"], L["mixer"], width, shapes), L.get("mlp")
    if not f:
        return LayerSpec(mixer)
    if f.get("kind", "dense") != "dense":
        raise ValueError(f"layer {i}: unknown feed-forward {f['kind']!r}")
    return LayerSpec(mixer, ff_after=f["ff"], unit=ClampedUnit(float(f["limit"])))


def parse_config(c: dict, shapes: Optional[Mapping[str, Tuple[int, ...]]] = None, name: str = "norusun") -> HybridConfig:
    """config.json -> HybridConfig.  `shapes`: tensor shapes of the checkpoint, for the one size that config.json does not carry
    (the rank of a decay projection; without a checkpoint it is read from the mixer's "rank")."""
    return HybridConfig(name=name, vocab=c["vocab"], hidden=c["width"],
                        layer_specs=tuple(_layer(i, L, c["width"], shapes or {}) for i, L in enumerate(c["layers"])),
                        rms_eps=float(c["norm"]["eps"]), norm_offset=0.0, tied=False, design="norusun", norm_scalar=True,
                        mix_taps=c["canon"]["taps"], streams=c["streams"])


def _tensors(seg: WeightSegment):
    """(checkpoint name, view of the segment, how) of every tensor.  how: False as it is, True transposed, a tuple: by head (see
    `to_segment`); a list of views holds the tensor's rows piece by piece, each transposed."""
    cfg: HybridConfig = seg.cfg

    def attention(m, p, d, cols, w_in, out):
        for n in ("q", "k", "v"):
            at, width = cols[d[1] + n]
            yield p + n, w_in[:, at:at + width], True
        yield p + "q.norm", seg[d[0] + d[1] + "q_norm"], False
        yield p + "k.norm", seg[d[0] + d[1] + "k_norm"], False
        yield p + "pb", seg[d[0] + d[1] + "weight_b"].view(-1), False
        yield p + "o", out[:m.out_width], True

    def state_space(m, p, d, cols, w_in, out):
        t = lambda n: seg[d[0] + d[1] + n]
        yield p + "in", [w_in[:, at:at + width] for at, width in (cols[d[1] + n] for n in ("z", "xbc", "dt"))], True
        yield p + "conv", t("conv"), True
        for n, at in (("conv.b", "conv_b"), ("dt_bias", "dt_bias"), ("A_log", "A_log"), ("D", "D"), ("norm", "o_norm")):
            yield p + n, t(at), False
        yield p + "o", out[:m.out_width], True

    yield "embed", seg["embed"], False
    yield "head", seg["lm_head"][:, :cfg.vocab], True
    yield "final.norm", seg["final_norm"].view(()), False
    for l, s in enumerate(cfg.layer_specs):
        d, p, m = f"layers.{l}.", f"l{l}.", s.mixer
        for q in s.sublayers:
            yield f"{p}norm{q}", seg[f"{d}norm{q}"].view(()), False
            for n in ("in", "out", "mix"):
                yield f"{p}hc{q}.{n}", seg[f"{d}hc{q}_{n}"], False
        yield p + "canon1", seg[d + "mix_conv"], True
        cols, w_in, out, x = s.in_columns()[0], seg[d + "in"], seg[d + "out"], p + "mix."
        if m.kind == "wkv":
            for i, n in enumerate(m.MIXES):
                yield f"{x}mu.{n}", seg[d + "mu"][i], False
            blocks = seg[d + "rkvg"].view(4, cfg.hidden, m.out_width)
            for i in range(4):
                yield x + m.MIXES[i], blocks[i], True
            yield x + "w1", seg[d + "w1"][:, :m.rank], True
            yield x + "w2", seg[d + "w2"], True
            yield x + "w0", seg[d + "w0"], False
            yield x + "u", seg[d + "bonus"].view(m.heads, m.dim), False
            yield x + "norm", seg[d + "o_norm"], False
            yield x + "o", out[:m.out_width], True
        elif m.kind == "latent":
            for n in ("dq", "dkv"):
                at, width = cols[n]
                yield x + n, w_in[:, at:at + width], True
                yield f"{x}{n}.norm", seg[f"{d}{n}_norm"], False
            yield x + "uq", seg[d + "uq"], True
            yield x + "uk", seg[d + "uk"], False
            # [heads * rank, vdim] by head, [heads * vdim, rank] in the checkpoint
            yield x + "uv", seg[d + "uv"].view(m.heads, m.kv_rank, m.vdim), (m.heads, m.vdim, m.kv_rank)
            yield x + "sink", seg[d + "sink"], False
            yield x + "o", out[:m.out_width], True
        else:
            yield from attention(m.left, x + "left.", (d, "l_"), cols, w_in, out)
            yield from state_space(m.right, x + "right.", (d, "r_"), cols, w_in, seg[d + "r_out"])
            yield x + "left.out", seg[d + "l_out_norm"], False
            yield x + "right.out", seg[d + "r_out_norm"], False
        if s.ff_after:
            n, pad = s.ff_after, s.ff_after_pad
            for k, at in (("gate", 0), ("up", pad)):
                yield f"{p}mlp.{k}", seg[d + "gate_up"][:, at:at + n], True
                yield f"{p}mlp.{k}.b", seg[d + "gate_up_b"][at:at + n], False
            yield p + "mlp.down", seg[d + "down"][:n], True
            yield p + "mlp.down.b", seg[d + "down_b"], False


def to_segment(reader, cfg: HybridConfig, dtype=torch.bfloat16) -> WeightSegment:
    """Segment on the host from a checkpoint reader (`get(name)`)."""
    seg = WeightSegment(cfg, 1, 0, dtype, device="cpu")
    seg.buffer.zero_()
    for name, dst, how in _tensors(seg):
        src = reader.get(name).to(dtype)
        if isinstance(how, tuple):
            want = (how[0] * how[1], how[2])
        elif isinstance(dst, list):
            want = (sum(v.shape[1] for v in dst), dst[0].shape[0])
        else:
            want = tuple(dst.t().shape if how else dst.shape)
        if tuple(src.shape) != want:
            raise ValueError(f"checkpoint tensor {name} has shape {tuple(src.shape)}, the configuration says {want}")
        if isinstance(how, tuple):
            dst.copy_(src.view(how).transpose(1, 2))
        elif isinstance(dst, list):
            for v, piece in zip(dst, src.split([v.shape[1] for v in dst])):
                v.copy_(piece.t())
        else:
            dst.copy_(src.t() if how else src)
    cfg.derive_(seg)
    return seg


def from_segment(seg: WeightSegment) -> Dict[str, torch.Tensor]:
    """Inverse mapping: checkpoint tensors of a segment."""
    out = {}
    for name, v, how in _tensors(seg):
        if isinstance(v, list):
            v = torch.cat(v, 1)
        if isinstance(how, tuple):
            v = v.transpose(1, 2).reshape(how[0] * how[1], how[2])
        out[name] = (v.t() if how is True else v).clone(memory_format=torch.contiguous_format)
    return out


def shape_config(name: str, vocab: int, hidden: int, pattern: Iterable[str], ff: int, *, wkv: Tuple[int, int, int], latent: dict, heads: int,
                 kv_heads: int, dim: int, chunk: int, ssd: dict, streams: int, taps: int, vdim: int = 0, rot_dims: int = 0,
                 limit: float = 7.0, gb: float = 0.0) -> HybridConfig:
    """A registry shape: one set of sizes per mixer, `pattern` names the layers' mixers; wkv: heads, head size, rank.  The layers with
    the linear attention have no feed-forward."""
    left = AttentionMixer(heads, kv_heads, dim, dim ** -0.5, rot_dims or dim, 5e5, interleaved=False, window=chunk, value_dim=vdim,
                          whole_norm=True, chunked=True, sigmoid=True)
    kinds = {"wkv": WKVMixer(hidden, *wkv), "parallel": ParallelMixer(hidden, left, SSDMixer(**ssd)),
             "latent_attention": LatentAttentionMixer(**latent, scale=(latent["dim"] + latent["rot_dim"]) ** -0.5, rot_base=5e5, gate=False,
                                                      interleaved=True, sink=True)}
    specs = tuple(LayerSpec(kinds[k]) if k == "wkv" else LayerSpec(kinds[k], ff_after=ff, unit=ClampedUnit(limit)) for k in pattern)
    return HybridConfig(name, vocab, hidden, specs, None, 1e-5, 1.0, gb, norm_offset=0.0, tied=False, design="norusun", norm_scalar=True,
                        mix_taps=taps, streams=streams)
