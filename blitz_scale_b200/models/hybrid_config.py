"""Shapes and constants of models whose layers differ: a list of layers over an fp32 residual stream, each with a mixer
(attention, gated linear attention, gated linear recurrence) and an optional feed-forward, with an optional block of
layers that runs several times.  The feed-forward is either a gated one beside the mixer (both read one norm) or a
mixture of experts behind it (with a norm of its own).

Everything a kernel needs is a field here, so a design is described by data: `models/fafudra.py` and
`models/komulorn.py` fill these records from a checkpoint's config.json, the registry from shapes.  `ModelConfig` (config.py) stays the record of
the uniform Llama-type models; both offer what the engine, the worker and the router read (name, vocab, hidden,
layers, eos_token, param_gb, kv_bytes_per_token).

Weight segment of such a model (one allocation, matrices ``[in, out]``, every tensor on a 256-byte boundary)::

    embed [vocab, hidden] | loop_step [times, hidden]
    L x { norm1 | in [hidden, projections] | mixer tensors | out [mixer out + ff, hidden] | gate_up [hidden, 2 ff]
          | norm2 | router [hidden, experts + 1] | up [experts x hidden, ff] | down [experts x ff, hidden]
          | shared_up [hidden, shared ff] | shared_down [shared ff, hidden] }
    final_norm [hidden] | lm_head [hidden, vocab]

A layer has two wide projections per side: ``in`` holds every projection of the mixer next to each other and ``out``
the mixer's and the feed-forward's output projections on top of each other, so that the sum of both sublayers is one
matrix product.  Experts are stacked along their input dimension, as the blocks of a block-diagonal product are; the
column behind the router's is the gate of the shared expert.  The column ranges of ``in`` and the row ranges of ``out`` start on multiples of 8 elements (16 bytes
in 16-bit types, what TMA and vector loads need); the padding is zero.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Dict, List, Optional, Tuple, Union

import torch

from .config import SegmentLayout, TensorSpec, _align


def pad8(n: int) -> int:
    return (n + 7) // 8 * 8


def _columns(widths: List[Tuple[str, int]]) -> Tuple[Dict[str, Tuple[int, int]], int]:
    """name -> (first column, width), each on a multiple of 8, and the padded total."""
    out, at = {}, 0
    for n, w in widths:
        out[n] = (at, w)
        at += pad8(w)
    return out, at


@dataclass(frozen=True)
class YarnScaling:
    """Rotary frequencies stretched for long contexts: pair i's frequency goes from f_i (pairs that turn more than `fast`
    times over the `original` context) to f_i / factor (fewer than `slow` times) along a linear ramp, and the rotated
    vectors grow by a constant."""
    factor: float
    original: float
    fast: float
    slow: float

    @property
    def gain(self) -> float:
        return 0.1 * math.log(self.factor) + 1.0

    def stretch(self, dims: int, base: float) -> List[float]:
        """What every pair's frequency is multiplied with."""
        pair_of = lambda turns: dims * math.log(self.original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
        lo, hi = max(math.floor(pair_of(self.fast)), 0), min(math.ceil(pair_of(self.slow)), dims - 1)
        ramp = [min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0) for i in range(dims // 2)]
        return [r / self.factor + (1.0 - r) for r in ramp]


@dataclass(frozen=True)
class AttentionMixer:
    heads: int
    kv_heads: int
    dim: int
    scale: float
    rot_dims: int
    rot_base: float
    interleaved: bool = True      # rotation pairs (2i, 2i + 1); False: (i, i + rot_dims / 2)
    window: int = 0               # a position sees this many positions back, itself included; 0: all
    keep_first: int = 0           # and the first ones of the sequence
    softcap: float = 0.0          # 0: none
    sink: bool = False            # learned number per head in the softmax denominator
    value_is_key: bool = False    # no value projection: values are the keys before rotation
    value_dim: int = 0            # size of a value head; 0: as `dim`
    bias: bool = False            # biases on the q, k and v projections
    gate: bool = False            # a head's output is multiplied by the sigmoid of a projection, one number per head
    yarn: Optional[YarnScaling] = None
    kv_from: Optional[int] = None  # layer whose cached keys and values are used; no k and v projections then
    kind = "attention"

    def __post_init__(self):
        if self.heads % self.kv_heads or self.rot_dims % 2 or self.rot_dims > self.dim:
            raise ValueError("attention mixer: heads must be a multiple of kv_heads, rotated dimensions even and within a head")
        if self.value_is_key and self.vdim != self.dim:
            raise ValueError("attention mixer: values that are keys have the keys' size")

    @property
    def vdim(self) -> int:
        return self.value_dim or self.dim

    @property
    def out_width(self) -> int:
        return self.heads * self.vdim

    def _qkv(self) -> List[Tuple[str, int]]:
        out = [("q", self.heads * self.dim)]
        if self.kv_from is None:
            out.append(("k", self.kv_heads * self.dim))
            if not self.value_is_key:
                out.append(("v", self.kv_heads * self.vdim))
        return out

    def projections(self) -> List[Tuple[str, int]]:
        return self._qkv() + ([("g", self.heads)] if self.gate else [])

    def tensors(self) -> List[Tuple[str, Tuple[int, ...]]]:
        return ([("sink", (self.heads,))] if self.sink else []) + ([(n + "_b", (w,)) for n, w in self._qkv()] if self.bias else [])


@dataclass(frozen=True)
class GLAMixer:
    heads: int
    dim: int
    vdim: int
    tau: float
    rank: int                     # of the decay projection
    kind = "gla"

    @property
    def out_width(self) -> int:
        return self.heads * self.vdim

    def projections(self) -> List[Tuple[str, int]]:
        k, v = self.heads * self.dim, self.heads * self.vdim
        return [("q", k), ("k", k), ("v", v), ("g", v), ("low", self.rank)]

    def tensors(self) -> List[Tuple[str, Tuple[int, ...]]]:
        k = self.heads * self.dim
        return [("a2", (self.rank, k)), ("a2_b", (k,)), ("o_norm", (self.vdim,))]

    def state_floats(self) -> int:
        return self.heads * self.dim * self.vdim


@dataclass(frozen=True)
class RGLRUMixer:
    width: int
    blocks: int
    taps: int
    kind = "rglru"

    def __post_init__(self):
        if self.width % self.blocks:
            raise ValueError("recurrent mixer: width must be a multiple of its blocks")

    @property
    def block(self) -> int:
        return self.width // self.blocks

    @property
    def out_width(self) -> int:
        return self.width

    def projections(self) -> List[Tuple[str, int]]:
        return [("y", self.width), ("x", self.width)]

    def tensors(self) -> List[Tuple[str, Tuple[int, ...]]]:
        w = self.width
        # gates: the blocks stacked along their inputs; a block's columns are its r outputs, then its i outputs
        return [("y_b", (w,)), ("x_b", (w,)), ("conv", (self.taps, w)), ("conv_b", (w,)), ("gates", (w, 2 * self.block)),
                ("gate_b", (2 * w,)), ("lam", (w,))]


Mixer = Union[AttentionMixer, GLAMixer, RGLRUMixer]


@dataclass(frozen=True)
class ExpertsSpec:
    """Mixture of experts without biases: W_down act(W_up h), act = the square of relu.  A token goes to the `top` experts
    with the largest router scores (sigmoid of the logits, optionally divided by the sum of the chosen ones); the score
    multiplies the expert's input or its output.  A shared expert runs for every token and is added, multiplied by the
    sigmoid of a projection."""
    experts: int
    top: int
    ff: int
    shared_ff: int = 0            # 0: no shared expert
    weight_on_input: bool = True
    renormalize: bool = False

    def __post_init__(self):
        if not 1 <= self.top <= self.experts or self.ff < 1:
            raise ValueError(f"{self.top} of {self.experts} experts of width {self.ff}")

    @property
    def ff_pad(self) -> int:
        return pad8(self.ff)

    @property
    def shared_pad(self) -> int:
        return pad8(self.shared_ff)

    @property
    def per_token(self) -> int:
        """Expert rows of a token, the shared expert's included."""
        return self.top + bool(self.shared_ff)

    @property
    def router_cols(self) -> int:
        return pad8(self.experts + bool(self.shared_ff))


@dataclass(frozen=True)
class LayerSpec:
    mixer: Mixer
    ff: int = 0                   # width of the gated feed-forward beside the mixer; 0: none
    moe: Optional[ExpertsSpec] = None   # experts behind the mixer, with a norm of their own

    def __post_init__(self):
        if self.ff and self.moe:
            raise ValueError("a layer has a feed-forward beside its mixer or experts behind it, not both")

    def in_columns(self) -> Tuple[Dict[str, Tuple[int, int]], int]:
        return _columns(self.mixer.projections())

    @property
    def mix_rows(self) -> int:
        """Rows of ``out`` before the feed-forward's."""
        return pad8(self.mixer.out_width)

    @property
    def ff_pad(self) -> int:
        return pad8(self.ff)

    @property
    def out_rows(self) -> int:
        return self.mix_rows + self.ff_pad


@dataclass(frozen=True)
class LoopSpec:
    start: int
    stop: int
    times: int


@dataclass(frozen=True)
class LayerRun:
    """One execution of a layer: which layer, and what is done to the stream before it."""
    layer: int
    step: int = -1                # row of loop_step added right before it (-1: none)
    add_embed: bool = False       # the embedding output is added as well


@dataclass(frozen=True)
class HybridConfig:
    name: str
    vocab: int
    hidden: int
    layer_specs: Tuple[LayerSpec, ...]
    loop: Optional[LoopSpec] = None
    rms_eps: float = 1e-6
    residual_mult: float = 1.0
    param_gb: float = 0.0
    eos_token: int = -1
    max_positions: int = 1 << 20
    norm_offset: float = 1.0      # added to the stored norm weights (1: they are stored around zero)
    logit_softcap: float = 0.0    # logits become cap * tanh(logits / cap); 0: none
    tied: bool = True             # the head is the embedding table
    design: str = "fafudra"       # module of this package that maps checkpoint names (weights of a folder)
    family = "hybrid"

    def __post_init__(self):
        for i, s in enumerate(self.layer_specs):
            j = getattr(s.mixer, "kv_from", None)
            if j is None:
                continue
            src = self.layer_specs[j].mixer if 0 <= j < i else None
            if src is None or src.kind != "attention" or src.kv_from is not None:
                raise ValueError(f"{self.name}: layer {i} takes keys and values from layer {j}, which has none of its own before it")
            same = ("kv_heads", "dim", "vdim")
            if any(getattr(src, n) != getattr(s.mixer, n) for n in same):
                raise ValueError(f"{self.name}: layers {j} and {i} share keys and values but differ in {', '.join(same)}")
        lp = self.loop
        if lp is not None and not (0 <= lp.start < lp.stop <= len(self.layer_specs) and lp.times >= 1):
            raise ValueError(f"{self.name}: loop of layers {lp.start}..{lp.stop} x {lp.times} does not fit "
                             f"{len(self.layer_specs)} layers")

    @property
    def layers(self) -> int:
        return len(self.layer_specs)

    def runs(self) -> List[LayerRun]:
        """The layer executions of one forward pass, in order.  Every one has a cache or a state of its own."""
        n, lp = self.layers, self.loop
        if lp is None:
            return [LayerRun(i) for i in range(n)]
        out = [LayerRun(i) for i in range(lp.start)]
        for t in range(lp.times):
            for i in range(lp.start, lp.stop):
                out.append(LayerRun(i, t, t > 0) if i == lp.start else LayerRun(i))
        return out + [LayerRun(i) for i in range(lp.stop, n)]

    def run_mixers(self) -> List[Mixer]:
        return [self.layer_specs[r.layer].mixer for r in self.runs()]

    def kv_runs(self) -> List[int]:
        """For every layer run the run whose keys and values it reads (its own, but for layers that share another's)."""
        latest: Dict[int, int] = {}
        out = []
        for r, run in enumerate(self.runs()):
            latest[run.layer] = r
            j = getattr(self.layer_specs[run.layer].mixer, "kv_from", None)
            out.append(r if j is None else latest[j])
        return out

    def kv_bytes_per_token(self, tp: int = 1, elem: int = 2) -> int:
        return sum(m.kv_heads * (m.dim + m.vdim) * elem for m in self.run_mixers() if m.kind == "attention" and m.kv_from is None)

    def state_bytes_per_sequence(self, elem: int = 2) -> int:
        n = 0
        for m in self.run_mixers():
            if m.kind == "gla":
                n += 4 * m.state_floats()
            elif m.kind == "rglru":
                n += 4 * m.width + elem * (m.taps - 1) * m.width
        return n

    def attention_work(self, length: int) -> Tuple[int, int]:
        """(KV heads, positions) of the attention run with the fewest heads and of the one that looks furthest back, for a
        sequence of `length` tokens: what the number of key splits is chosen from.  (0, 0) without attention."""
        a = [m for m in self.run_mixers() if m.kind == "attention"]
        if not a:
            return 0, 0
        span = max(min(length, m.window + m.keep_first) if m.window else length for m in a)
        return min(m.kv_heads for m in a), span

    @property
    def recurrent(self) -> bool:
        return any(m.kind != "attention" for m in self.run_mixers())

    @property
    def vocab_pad(self) -> int:
        return pad8(self.vocab)

    def init_(self, name: str, v: torch.Tensor, rand) -> None:
        """Random weights with activations of order one; `rand(shape)` gives normal numbers on v's device."""
        leaf = name.rsplit(".", 1)[-1]
        if leaf in ("norm1", "norm2", "final_norm"):
            x = 1.0 - self.norm_offset + 0.1 * rand(v.shape)
        elif leaf == "o_norm":
            x = 1.0 + 0.1 * rand(v.shape)
        elif leaf == "a2_b":
            x = 2.0 + rand(v.shape)                          # slow decays with some fast channels
        elif leaf == "lam":
            x = -4.0 + rand(v.shape)                         # a between about 0.8 and 0.99
        elif leaf in ("x_b", "y_b", "conv_b", "gate_b", "sink", "loop_step", "q_b", "k_b", "v_b"):
            x = 0.2 * rand(v.shape)
        elif leaf in ("up", "down"):                         # experts stacked along their inputs
            moe = self.layer_specs[int(name.split(".")[1])].moe
            n = v.shape[0] // moe.experts
            for e in range(moe.experts):
                v[e * n:(e + 1) * n].copy_((rand((n, v.shape[1])) * n ** -0.5).to(v.dtype))
            return
        elif leaf == "conv":
            x = rand(v.shape) * v.shape[0] ** -0.5
        elif leaf == "embed":
            x = rand(v.shape)
        elif leaf == "gates":
            x = rand(v.shape) * (v.shape[1] // 2) ** -0.5
        else:
            x = rand(v.shape) * v.shape[0] ** -0.5
        v.copy_(x.to(v.dtype))

    def zero_padding_(self, tensors) -> None:
        """Clear the padding columns and rows of a filled segment (name -> tensor)."""
        tensors["lm_head"][:, self.vocab:] = 0
        for l, s in enumerate(self.layer_specs):
            p = f"layers.{l}."
            cols, total = s.in_columns()
            w = tensors[p + "in"]
            for at, width in cols.values():
                w[:, at + width:at + pad8(width)] = 0
            o = tensors[p + "out"]
            o[s.mixer.out_width:s.mix_rows] = 0
            if s.ff:
                o[s.mix_rows + s.ff:] = 0
                g = tensors[p + "gate_up"]
                g[:, s.ff:s.ff_pad] = 0
                g[:, s.ff_pad + s.ff:] = 0
            if s.moe:
                e = s.moe
                tensors[p + "router"][:, e.experts + bool(e.shared_ff):] = 0
                tensors[p + "up"][:, e.ff:] = 0
                tensors[p + "down"].view(e.experts, e.ff_pad, self.hidden)[:, e.ff:] = 0
                if e.shared_ff:
                    tensors[p + "shared_up"][:, e.shared_ff:] = 0
                    tensors[p + "shared_down"][e.shared_ff:] = 0


def build_hybrid_layout(cfg: HybridConfig, tp: int = 1, elem_bytes: int = 2) -> SegmentLayout:
    if tp != 1:
        raise ValueError(f"{cfg.name}: models of this kind run on one GPU (tp = 1)")
    lay = SegmentLayout(cfg, tp, elem_bytes)
    cur = 0

    def add(name, shape):
        nonlocal cur
        n = elem_bytes
        for s in shape:
            n *= s
        lay.tensors[name] = TensorSpec(name, tuple(shape), cur, n)
        cur = _align(cur + n)

    start = cur
    add("embed", (cfg.vocab, cfg.hidden))
    if cfg.loop is not None:
        add("loop_step", (cfg.loop.times, cfg.hidden))
    lay.units.append(("embed", start, cur - start))
    for l, s in enumerate(cfg.layer_specs):
        start, p = cur, f"layers.{l}."
        add(p + "norm1", (cfg.hidden,))
        add(p + "in", (cfg.hidden, s.in_columns()[1]))
        for n, shape in s.mixer.tensors():
            add(p + n, shape)
        add(p + "out", (s.out_rows, cfg.hidden))
        if s.ff:
            add(p + "gate_up", (cfg.hidden, 2 * s.ff_pad))
        if s.moe:
            e = s.moe
            add(p + "norm2", (cfg.hidden,))
            add(p + "router", (cfg.hidden, e.router_cols))
            add(p + "up", (e.experts * cfg.hidden, e.ff_pad))
            add(p + "down", (e.experts * e.ff_pad, cfg.hidden))
            if e.shared_ff:
                add(p + "shared_up", (cfg.hidden, e.shared_pad))
                add(p + "shared_down", (e.shared_pad, cfg.hidden))
        lay.units.append((f"layer.{l}", start, cur - start))
    start = cur
    add("final_norm", (cfg.hidden,))
    add("lm_head", (cfg.hidden, cfg.vocab_pad))
    lay.units.append(("head", start, cur - start))
    lay.total_bytes = cur
    return lay
