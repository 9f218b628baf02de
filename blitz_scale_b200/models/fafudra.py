"""Fafudra: parallel layers (mixer and feed-forward read one norm) over three mixers (windowed attention with kept
first tokens, a sink and soft-capped scores; gated linear attention; a gated linear recurrence), a block of layers that
runs several times, tied embeddings.

This file is what is specific to the design: how its config.json and its tensor names map onto the records of
hybrid_config.py.  Linear weights come as [out, in] and are stored as [in, out].
"""
from __future__ import annotations

from typing import Dict, Iterable, Mapping, Optional, Tuple

import torch

from .hybrid_config import AttentionMixer, GLAMixer, HybridConfig, LayerSpec, LoopSpec, RGLRUMixer
from .weights import WeightSegment

ARCHITECTURE = "Fafudra"


def _mixer(i: int, kind: str, m: dict, shapes: Mapping[str, Tuple[int, ...]]):
    p = f"l{i}.mix."
    if kind == "attention":
        if m["vdim"] != m["dim"]:
            raise ValueError(f"layer {i}: values are the keys, so vdim ({m['vdim']}) must equal dim ({m['dim']})")
        return AttentionMixer(heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], scale=float(m["scale"]),
                              rot_dims=m["rot"]["dims"], rot_base=float(m["rot"]["base"]), interleaved=True,
                              window=m["mask"]["size"], keep_first=m["mask"]["keep_first"],
                              softcap=float(m["softcap"]), sink=True, value_is_key=True)
    if kind == "gla":
        rank = shapes[p + "a1"][0] if p + "a1" in shapes else m["rank"]
        return GLAMixer(heads=m["heads"], dim=m["dim"], vdim=m["vdim"], tau=float(m["tau"]), rank=rank)
    if kind == "rglru":
        return RGLRUMixer(width=m["width"], blocks=m["blocks"], taps=m["conv"])
    raise ValueError(f"layer {i}: unknown mixer {kind!r}")


def parse_config(c: dict, shapes: Optional[Mapping[str, Tuple[int, ...]]] = None, name: str = "fafudra") -> HybridConfig:
    """config.json -> HybridConfig.  `shapes`: tensor shapes of the checkpoint, for the one size that config.json does
    not carry (the rank of a decay projection; without a checkpoint it is read from the mixer's "rank")."""
    layers = []
    for i, L in enumerate(c["layers"]):
        mlp = L.get("mlp")
        if mlp is not None and mlp.get("kind", "dense") != "dense":
            raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
        layers.append(LayerSpec(_mixer(i, L["type"], L["mixer"], shapes or {}), int(mlp["ff"]) if mlp else 0))
    lp = c.get("loop")
    loop = LoopSpec(lp["start"], lp["stop"], lp["times"]) if lp else None
    return HybridConfig(name=name, vocab=c["vocab"], hidden=c["width"], layer_specs=tuple(layers), loop=loop,
                        rms_eps=float(c["norm"]["eps"]), residual_mult=float(c["residual_mult"]))


def to_segment(reader, cfg: HybridConfig, dtype=torch.bfloat16) -> WeightSegment:
    """Segment on the host from a checkpoint reader (`get(name)`)."""
    seg = WeightSegment(cfg, 1, 0, dtype, device="cpu")
    seg.buffer.zero_()

    def put(dst: torch.Tensor, src: torch.Tensor) -> None:
        if tuple(dst.shape) != tuple(src.shape):
            raise ValueError(f"checkpoint tensor has shape {tuple(src.shape)}, the configuration says {tuple(dst.shape)}")
        dst.copy_(src.to(dtype))

    put(seg["embed"], reader.get("embed"))
    put(seg["lm_head"][:, :cfg.vocab], reader.get("embed").t())
    put(seg["final_norm"], reader.get("final.norm"))
    if cfg.loop is not None:
        put(seg["loop_step"], reader.get("loop.step"))
    for l, s in enumerate(cfg.layer_specs):
        d, m = f"layers.{l}.", s.mixer
        mix = lambda n, l=l: reader.get(f"l{l}.mix.{n}")
        put(seg[d + "norm1"], reader.get(f"l{l}.norm1"))
        names = {"low": "a1"}                         # projections whose checkpoint name differs
        for n, (at, width) in s.in_columns()[0].items():
            put(seg[d + "in"][:, at:at + width], mix(names.get(n, n)).t())
        if m.kind == "attention":
            put(seg[d + "sink"], mix("sink"))
        elif m.kind == "gla":
            put(seg[d + "a2"], mix("a2").t())
            put(seg[d + "a2_b"], mix("a2.b"))
            put(seg[d + "o_norm"], mix("norm"))
        else:
            for dst, src in (("y_b", "y.b"), ("x_b", "x.b"), ("conv_b", "conv.b"), ("lam", "lam")):
                put(seg[d + dst], mix(src))
            put(seg[d + "conv"], mix("conv").t())
            b = m.block
            gates = seg[d + "gates"].view(m.blocks, b, 2, b)                 # block, in, r | i, out
            bias = seg[d + "gate_b"].view(m.blocks, 2, b)
            for j, n in enumerate(("ra", "ri")):
                put(gates[:, :, j], mix(n).transpose(1, 2))
                put(bias[:, j], mix(n + ".b"))
        put(seg[d + "out"][:m.out_width], mix("o").t())
        if s.ff:
            put(seg[d + "out"][s.mix_rows:s.mix_rows + s.ff], reader.get(f"l{l}.mlp.down").t())
            put(seg[d + "gate_up"][:, :s.ff], reader.get(f"l{l}.mlp.gate").t())
            put(seg[d + "gate_up"][:, s.ff_pad:s.ff_pad + s.ff], reader.get(f"l{l}.mlp.up").t())
    return seg


def from_segment(seg: WeightSegment) -> Dict[str, torch.Tensor]:
    """Inverse mapping: checkpoint tensors of a segment."""
    cfg: HybridConfig = seg.cfg
    out = {"embed": seg["embed"].clone(), "final.norm": seg["final_norm"].clone()}
    if cfg.loop is not None:
        out["loop.step"] = seg["loop_step"].clone()
    t = lambda x: x.t().contiguous()
    for l, s in enumerate(cfg.layer_specs):
        d, p, m = f"layers.{l}.", f"l{l}.mix.", s.mixer
        out[f"l{l}.norm1"] = seg[d + "norm1"].clone()
        for n, (at, width) in s.in_columns()[0].items():
            out[p + {"low": "a1"}.get(n, n)] = t(seg[d + "in"][:, at:at + width])
        if m.kind == "attention":
            out[p + "sink"] = seg[d + "sink"].clone()
        elif m.kind == "gla":
            out[p + "a2"], out[p + "a2.b"], out[p + "norm"] = t(seg[d + "a2"]), seg[d + "a2_b"].clone(), seg[d + "o_norm"].clone()
        else:
            for src, dst in (("y_b", "y.b"), ("x_b", "x.b"), ("conv_b", "conv.b"), ("lam", "lam")):
                out[p + dst] = seg[d + src].clone()
            out[p + "conv"] = t(seg[d + "conv"])
            gates = seg[d + "gates"].view(m.blocks, m.block, 2, m.block)
            bias = seg[d + "gate_b"].view(m.blocks, 2, m.block)
            for j, n in enumerate(("ra", "ri")):
                out[p + n] = gates[:, :, j].transpose(1, 2).contiguous()
                out[p + n + ".b"] = bias[:, j].contiguous()
        out[p + "o"] = t(seg[d + "out"][:m.out_width])
        if s.ff:
            out[f"l{l}.mlp.down"] = t(seg[d + "out"][s.mix_rows:s.mix_rows + s.ff])
            out[f"l{l}.mlp.gate"] = t(seg[d + "gate_up"][:, :s.ff])
            out[f"l{l}.mlp.up"] = t(seg[d + "gate_up"][:, s.ff_pad:s.ff_pad + s.ff])
    return out


def shape_config(name: str, vocab: int, hidden: int, pattern: Iterable[str], ff: int, *, heads: int, kv_heads: int, dim: int,
                 window: int, keep_first: int = 4, gla_heads: int = 0, gla_dim: int = 0, gla_vdim: int = 0, rank: int = 16,
                 width: int = 0, blocks: int = 1, loop: Optional[Tuple[int, int, int]] = None, gb: float = 0.0) -> HybridConfig:
    """A registry shape: one set of sizes per mixer, `pattern` names the layers' mixers."""
    kinds = {"attention": AttentionMixer(heads, kv_heads, dim, dim ** -0.5, dim, 1e5, True, window, keep_first, 50.0, True, True),
             "gla": GLAMixer(gla_heads or heads, gla_dim or dim, gla_vdim or dim, 16.0, rank),
             "rglru": RGLRUMixer(width or hidden, blocks, 4)}
    return HybridConfig(name, vocab, hidden, tuple(LayerSpec(kinds[k], ff) for k in pattern),
                        LoopSpec(*loop) if loop else None, 1e-6, 0.8, gb)
