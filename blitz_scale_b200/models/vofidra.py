"""Vofidra: pre-norm layers over several residual streams (hyper-connections, dynamic-tanh norms); attention with normed
queries and keys, a query temperature and a learned bias by distance; latent attention with a cached latent, a shared rotated
key part and a gate per head; gated feed-forwards, dense or a mixture of experts (softmax scores with a correction, groups,
identity experts); an untied head with soft-capped logits.

This file is what is specific to the design: how its config.json and its tensor names map onto the records of
hybrid_config.py.  Linear weights come as [out, in] and are stored as [in, out].
"""
from __future__ import annotations

from typing import Dict, Mapping, Optional, Tuple

import torch

from .hybrid_config import (AttentionMixer, DistanceBias, ExpertsSpec, HybridConfig, LatentAttentionMixer, LayerSpec,
                            QueryTemperature)
from .weights import WeightSegment

ARCHITECTURE = "Vofidra"


def _mixer(i: int, kind: str, m: dict, shapes: Mapping[str, Tuple[int, ...]]):
    if kind == "attention":
        t = m.get("q_temp")
        return AttentionMixer(heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], value_dim=m["vdim"], scale=float(m["scale"]),
                              rot_dims=0, rot_base=1.0, qk_norm=True,
                              q_temp=QueryTemperature(float(t["coef"]), _whole(t["every"])) if t else None,
                              rel=DistanceBias(shapes[f"l{i}.mix.rel"][0], _whole(m["bias_max"])))
    if kind == "latent_attention":
        rot = m.get("rot") or {"dims": 0, "base": 1.0}
        if rot["dims"] != m["rot_dim"]:
            raise ValueError(f"layer {i}: the rotated part has {m['rot_dim']} dimensions, the rotation {rot['dims']}")
        rank = m["q_rank"] if "q_rank" in m else shapes[f"l{i}.mix.dq"][0]
        return LatentAttentionMixer(heads=m["heads"], dim=m["dim"], rot_dim=m["rot_dim"], vdim=m["vdim"], q_rank=rank,
                                    kv_rank=m["kv_rank"], scale=float(m["scale"]), rot_base=float(rot["base"]))
    raise ValueError(f"layer {i}: unknown mixer {kind!r}")


def _whole(x) -> int:
    if int(x) != x:
        raise ValueError(f"{x} is not a whole number")
    return int(x)


def _layer(i: int, L: dict, shapes: Mapping[str, Tuple[int, ...]]) -> LayerSpec:
    mixer, f = _mixer(i, L["type"], L["mixer"], shapes), L.get("mlp")
    if not f:
        return LayerSpec(mixer)
    if f["kind"] == "dense":
        return LayerSpec(mixer, ff_after=f["ff"])
    if f["kind"] != "moe":
        raise ValueError(f"layer {i}: unknown feed-forward {f['kind']!r}")
    r = f["router"]
    groups = r.get("groups") or {"count": 0, "keep": 0}
    return LayerSpec(mixer, moe=ExpertsSpec(experts=r["experts"], top=r["top"], ff=f["expert"]["ff"], weight_on_input=False,
                                            renormalize=True, gated=True, softmax=True, correction=True,
                                            identity=r.get("identity") or 0, groups=groups["count"], keep=groups["keep"]))


def parse_config(c: dict, shapes: Optional[Mapping[str, Tuple[int, ...]]] = None, name: str = "vofidra") -> HybridConfig:
    """config.json -> HybridConfig; the rows of the distance biases are in the tensors' shapes only."""
    return HybridConfig(name=name, vocab=c["vocab"], hidden=c["width"],
                        layer_specs=tuple(_layer(i, L, shapes or {}) for i, L in enumerate(c["layers"])), rms_eps=float(c["norm"]["eps"]),
                        norm_offset=0.0, logit_softcap=float(c.get("logit_softcap") or 0.0), tied=False, design="vofidra",
                        norm="tanh", streams=c["streams"])


def _tensors(seg: WeightSegment):
    """(checkpoint name, view of the segment, transposed) of every tensor but the experts' gate and up."""
    cfg: HybridConfig = seg.cfg

    def norm(name, at):
        yield name, seg[at], False
        yield name + ".b", seg[at + "_b"], False
        yield name + ".alpha", seg[at + "_alpha"].view(()), False
    yield "embed", seg["embed"], False
    yield "head", seg["lm_head"][:, :cfg.vocab], True
    yield from norm("final.norm", "final_norm")
    for l, s in enumerate(cfg.layer_specs):
        d, p, m = f"layers.{l}.", f"l{l}.", s.mixer
        for q in s.sublayers:
            yield from norm(f"{p}norm{q}", f"{d}norm{q}")
            for n in ("in", "out", "mix"):
                yield f"{p}hc{q}.{n}", seg[f"{d}hc{q}_{n}"], False
        for n, (at, width) in s.in_columns()[0].items():
            yield p + "mix." + n, seg[d + "in"][:, at:at + width], True
        if m.kind == "latent":
            yield p + "mix.dq.norm", seg[d + "dq_norm"], False
            yield p + "mix.dkv.norm", seg[d + "dkv_norm"], False
            yield p + "mix.uq", seg[d + "uq"], True
            yield p + "mix.uk", seg[d + "uk"], False
            # [heads * rank, vdim] by head, [heads * vdim, rank] in the checkpoint
            yield p + "mix.uv", seg[d + "uv"].view(m.heads, m.kv_rank, m.vdim), (m.heads, m.vdim, m.kv_rank)
        else:
            yield p + "mix.q.norm", seg[d + "q_norm"], False
            yield p + "mix.k.norm", seg[d + "k_norm"], False
            yield p + "mix.rel", seg[d + "rel"], False
        yield p + "mix.o", seg[d + "out"][:m.out_width], True
        if s.ff_after:
            n, pad = s.ff_after, s.ff_after_pad
            yield p + "mlp.gate", seg[d + "gate_up"][:, :n], True
            yield p + "mlp.up", seg[d + "gate_up"][:, pad:pad + n], True
            yield p + "mlp.down", seg[d + "down"][:n], True
        if s.moe:
            e = s.moe
            yield p + "mlp.router", seg[d + "router"][:, :e.outputs], True
            yield p + "mlp.correction", seg[d + "correction"], False
            down = seg[d + "down"].view(e.experts, e.ff_pad, cfg.hidden)
            for i in range(e.experts):
                yield f"{p}mlp.e{i}.down", down[i, :e.ff], True


def _gates(seg: WeightSegment):
    """(checkpoint name, view [hidden, ff_pad / 32, 32], width) of the experts' gate and up matrices."""
    cfg: HybridConfig = seg.cfg
    for l, s in enumerate(cfg.layer_specs):
        if s.moe:
            both = s.moe.gate_and_up(seg[f"layers.{l}.up"].view(s.moe.experts, cfg.hidden, s.moe.up_cols))
            for i in range(s.moe.experts):
                for k, n in enumerate(("gate", "up")):
                    yield f"l{l}.mlp.e{i}.{n}", both[i, :, :, k], s.moe.ff


def to_segment(reader, cfg: HybridConfig, dtype=torch.bfloat16) -> WeightSegment:
    """Segment on the host from a checkpoint reader (`get(name)`)."""
    seg = WeightSegment(cfg, 1, 0, dtype, device="cpu")
    seg.buffer.zero_()

    def fetch(name, shape):
        src = reader.get(name)
        if tuple(src.shape) != tuple(shape):
            raise ValueError(f"checkpoint tensor {name} has shape {tuple(src.shape)}, the configuration says {tuple(shape)}")
        return src.to(dtype)
    for name, dst, how in _tensors(seg):
        if isinstance(how, tuple):
            dst.copy_(fetch(name, (how[0] * how[1], how[2])).view(how).transpose(1, 2))
        else:
            src = fetch(name, dst.t().shape if how else dst.shape)
            dst.copy_(src.t() if how else src)
    for name, dst, ff in _gates(seg):
        src = torch.zeros(dst.shape[0], dst.shape[1] * 32, dtype=dtype)
        src[:, :ff] = fetch(name, (ff, cfg.hidden)).t()
        dst.copy_(src.view(dst.shape))
    cfg.derive_(seg)
    return seg


def from_segment(seg: WeightSegment) -> Dict[str, torch.Tensor]:
    """Inverse mapping: checkpoint tensors of a segment."""
    out = {}
    for name, v, how in _tensors(seg):
        if isinstance(how, tuple):
            v = v.transpose(1, 2).reshape(how[0] * how[1], how[2])
        out[name] = (v.t() if how is True else v).clone(memory_format=torch.contiguous_format)
    for name, v, ff in _gates(seg):
        out[name] = v.reshape(v.shape[0], -1)[:, :ff].t().contiguous()
    return out


def shape_config(name: str, vocab: int, hidden: int, layers: int, *, heads: int, kv_heads: int, dim: int, latent: dict, experts: int,
                 identity: int, top: int, groups: int, keep: int, ff: int, dense_ff: int, streams: int, rel: Tuple[int, int] = (32, 512),
                 gb: float = 0.0) -> HybridConfig:
    """A registry shape: every second layer has latent attention; the first has a dense feed-forward, the others experts."""
    moe = ExpertsSpec(experts, top, ff, weight_on_input=False, renormalize=True, gated=True, softmax=True, correction=True,
                      identity=identity, groups=groups, keep=keep)
    plain = AttentionMixer(heads, kv_heads, dim, dim ** -0.5, 0, 1.0, qk_norm=True, q_temp=QueryTemperature(0.1, 2048),
                           rel=DistanceBias(*rel))
    mla = LatentAttentionMixer(**latent, scale=(latent["dim"] + latent["rot_dim"]) ** -0.5, rot_base=5e5)
    specs = tuple(LayerSpec(mla if i % 2 else plain, **(dict(moe=moe) if i else dict(ff_after=dense_ff))) for i in range(layers))
    return HybridConfig(name, vocab, hidden, specs, None, 1e-6, 1.0, gb, norm_offset=0.0, logit_softcap=30.0, tied=False,
                        design="vofidra", norm="tanh", streams=streams)
