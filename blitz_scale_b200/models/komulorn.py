"""Komulorn: pre-norm layers of attention (biased projections, YaRN rotation of part of a head, values of a size of their
own, a gate per head, layers that read another layer's key/value cache) and a mixture of experts (squared relu, sigmoid
scores that scale the expert's input, a gated shared expert), an untied head with soft-capped logits.

This file is what is specific to the design: how its config.json and its tensor names map onto the records of
hybrid_config.py.  Linear weights come as [out, in] and are stored as [in, out].
"""
from __future__ import annotations

from typing import Dict, Mapping, Optional, Tuple

import torch

from .hybrid_config import AttentionMixer, ExpertsSpec, HybridConfig, LayerSpec, YarnScaling
from .weights import WeightSegment

ARCHITECTURE = "Komulorn"


def _mixer(i: int, kind: str, m: dict) -> AttentionMixer:
    if kind != "attention":
        raise ValueError(f"layer {i}: unknown mixer {kind!r}")
    rot = m.get("rot") or {"dims": 0, "base": 1.0}
    sc = rot.get("scaling")
    yarn = YarnScaling(*(float(sc[n]) for n in ("factor", "original", "fast", "slow"))) if sc and rot["dims"] else None
    return AttentionMixer(heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], value_dim=m["vdim"], scale=float(m["scale"]),
                          rot_dims=rot["dims"], rot_base=float(rot["base"]), interleaved=False, bias=True, gate=True, yarn=yarn,
                          kv_from=m.get("kv_from"))


def _experts(i: int, m: dict) -> ExpertsSpec:
    if m.get("kind") != "moe":
        raise ValueError(f"layer {i}: unknown feed-forward {m.get('kind')!r}")
    shared = m.get("shared")
    return ExpertsSpec(experts=m["router"]["experts"], top=m["router"]["top"], ff=m["expert"]["ff"],
                       shared_ff=shared["ff"] if shared else 0)


def parse_config(c: dict, shapes: Optional[Mapping[str, Tuple[int, ...]]] = None, name: str = "komulorn") -> HybridConfig:
    """config.json -> HybridConfig (every size is in config.json; `shapes` is not needed)."""
    layers = tuple(LayerSpec(_mixer(i, L["type"], L["mixer"]), moe=_experts(i, L["mlp"]) if L.get("mlp") else None)
                   for i, L in enumerate(c["layers"]))
    return HybridConfig(name=name, vocab=c["vocab"], hidden=c["width"], layer_specs=layers, rms_eps=float(c["norm"]["eps"]),
                        norm_offset=0.0, logit_softcap=float(c.get("logit_softcap") or 0.0), tied=False, design="komulorn")


def _tensors(seg: WeightSegment):
    """(checkpoint name, view of the segment, transposed) of every tensor."""
    cfg: HybridConfig = seg.cfg
    yield "embed", seg["embed"], False
    yield "head", seg["lm_head"][:, :cfg.vocab], True
    yield "final.norm", seg["final_norm"], False
    for l, s in enumerate(cfg.layer_specs):
        d, p, m = f"layers.{l}.", f"l{l}.", s.mixer
        yield p + "norm1", seg[d + "norm1"], False
        for n, (at, width) in s.in_columns()[0].items():
            yield p + "mix." + n, seg[d + "in"][:, at:at + width], True
        for n, _ in m.tensors():
            yield p + "mix." + n.replace("_b", ".b"), seg[d + n], False
        yield p + "mix.o", seg[d + "out"][:m.out_width], True
        if s.moe:
            e = s.moe
            yield p + "norm2", seg[d + "norm2"], False
            yield p + "mlp.router", seg[d + "router"][:, :e.experts], True
            up = seg[d + "up"].view(e.experts, cfg.hidden, e.ff_pad)
            down = seg[d + "down"].view(e.experts, e.ff_pad, cfg.hidden)
            for i in range(e.experts):
                yield f"{p}mlp.e{i}.up", up[i, :, :e.ff], True
                yield f"{p}mlp.e{i}.down", down[i, :e.ff], True
            if e.shared_ff:
                yield p + "mlp.shared.up", seg[d + "shared_up"][:, :e.shared_ff], True
                yield p + "mlp.shared.down", seg[d + "shared_down"][:e.shared_ff], True
                yield p + "mlp.shared.sg", seg[d + "router"][:, e.experts:e.experts + 1], True


def to_segment(reader, cfg: HybridConfig, dtype=torch.bfloat16) -> WeightSegment:
    """Segment on the host from a checkpoint reader (`get(name)`)."""
    seg = WeightSegment(cfg, 1, 0, dtype, device="cpu")
    seg.buffer.zero_()
    for name, dst, transposed in _tensors(seg):
        src = reader.get(name)
        src = src.t() if transposed else src
        if tuple(dst.shape) != tuple(src.shape):
            raise ValueError(f"checkpoint tensor {name} has shape {tuple(src.shape)}, the configuration says {tuple(dst.shape)}")
        dst.copy_(src.to(dtype))
    return seg


def from_segment(seg: WeightSegment) -> Dict[str, torch.Tensor]:
    """Inverse mapping: checkpoint tensors of a segment."""
    return {n: (v.t() if transposed else v).clone(memory_format=torch.contiguous_format) for n, v, transposed in _tensors(seg)}


def shape_config(name: str, vocab: int, hidden: int, layers: int, *, heads: int, kv_heads: int, dim: int, vdim: int, rot_dims: int,
                 experts: int, top: int, ff: int, shared_ff: int, share: int = 2, gb: float = 0.0) -> HybridConfig:
    """A registry shape of equal layers; of every `share` neighbours the first has the keys and values."""
    yarn = YarnScaling(4.0, 4096.0, 32.0, 1.0)
    moe = ExpertsSpec(experts, top, ff, shared_ff)
    mixer = lambda i: AttentionMixer(heads, kv_heads, dim, dim ** -0.5, rot_dims, 5e5, interleaved=False, value_dim=vdim, bias=True,
                                     gate=True, yarn=yarn, kv_from=i // share * share if i % share else None)
    return HybridConfig(name, vocab, hidden, tuple(LayerSpec(mixer(i), moe=moe) for i in range(layers)), None, 1e-6, 1.0, gb,
                        norm_offset=0.0, logit_softcap=30.0, tied=False, design="komulorn")
