"""Shapes and constants of models whose layers differ: a list of layers over an fp32 residual stream, or several of them,
each with a mixer (attention, latent attention, gated linear attention, gated linear recurrence, linear attention with a token
shift and a bonus, state space, or two of them side by side) and an optional feed-forward, with an optional block of layers that runs several times.  The feed-forward is a gated one beside the mixer
(both read one norm), or a gated one or a mixture of experts behind it (with a norm of its own).

Everything a kernel needs is a field here, so a design is described by data: `models/fafudra.py`, `models/komulorn.py`,
`models/vofidra.py` and `models/norusun.py` fill these records from a checkpoint's config.json, the registry from shapes.  `ModelConfig` (config.py) stays the record of
the uniform Llama-type models; both offer what the engine, the worker and the router read (name, vocab, hidden,
layers, eos_token, param_gb, kv_bytes_per_token).

Weight segment of such a model (one allocation, matrices ``[in, out]``, every tensor on a 256-byte boundary)::

    embed [vocab, hidden] | loop_step [times, hidden]
    L x { norm1 | in [hidden, projections] | mixer tensors | out [mixer out + ff, hidden] | gate_up [hidden, 2 ff]
          | norm2 | router [hidden, experts + 1] | up [experts x hidden, ff] | down [experts x ff, hidden]
          | shared_up [hidden, shared ff] | shared_down [shared ff, hidden] }
    final_norm [hidden] | lm_head [hidden, vocab]

A norm's weight is one number where `norm_scalar` says so.  Every norm of a model with the dynamic-tanh norm has two more tensors (``norm1_b`` and ``norm1_alpha``), a sublayer of a
model with several streams its coefficients (``hc1_in``, ``hc1_out``, ``hc1_mix``), a gated feed-forward behind the mixer
``gate_up`` and ``down`` (with a clamped unit also their biases), a layer whose mixer reads a convolution of its input ``mix_conv``.  Some tensors are derived from others when a segment is filled (`derive_`): forms of one matrix that
different kernels read.

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
class QueryTemperature:
    """Queries at position p are multiplied by 1 + coef * ln(floor((p + 1) / every) + 1)."""
    coef: float
    every: int

    def __post_init__(self):
        if self.every < 1:
            raise ValueError("query temperature: the step must be a positive whole number")


@dataclass(frozen=True)
class DistanceBias:
    """A table of `rows` numbers per head.  Distances below rows / 2 have a row each; longer ones share the others on a
    logarithmic scale that reaches the last row at distance `far`."""
    rows: int
    far: int

    def __post_init__(self):
        if self.rows < 2 or self.far <= self.rows // 2:
            raise ValueError(f"bias by distance: {self.rows} rows up to distance {self.far}")

    def row(self, n: int) -> int:
        half = self.rows // 2
        if n < half:
            return n
        return min(self.rows - 1, half + math.floor(math.log(n / half) / math.log(self.far / half) * (self.rows - half)))

    def rows_by_distance(self) -> List[int]:
        """The rows of distances 0, 1, ..; the last entry holds for all longer ones."""
        out = []
        while not out or out[-1] != self.rows - 1:
            out.append(self.row(len(out)))
        return out


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
    qk_norm: bool = False         # RMSNorm of every query and key head (no rotation, no biases)
    q_temp: Optional["QueryTemperature"] = None   # with qk_norm: queries grow with the position
    rel: Optional["DistanceBias"] = None          # learned bias by distance and head, added to the scaled scores
    whole_norm: bool = False      # RMSNorm over all query heads together, and over all key heads, before the rotation
    chunked: bool = False         # the window is a chunk counted from position 0: a position sees its own chunk's keys
    sigmoid: bool = False         # weights are sigmoids of score + a learned number per head, not normalised
    kind = "attention"

    def __post_init__(self):
        if self.heads % self.kv_heads or self.rot_dims % 2 or self.rot_dims > self.dim:
            raise ValueError("attention mixer: heads must be a multiple of kv_heads, rotated dimensions even and within a head")
        if self.value_is_key and self.vdim != self.dim:
            raise ValueError("attention mixer: values that are keys have the keys' size")
        if self.qk_norm and (self.rot_dims or self.bias or self.value_is_key or self.kv_from is not None):
            raise ValueError("attention mixer: normed queries and keys come without rotation, biases or shared caches")
        if self.q_temp and not self.qk_norm:
            raise ValueError("attention mixer: a query temperature goes with normed queries")
        if self.whole_norm and (self.qk_norm or self.bias or self.value_is_key or self.kv_from is not None):
            raise ValueError("attention mixer: a norm over all heads comes without other norms, biases or shared caches")
        if self.chunked and (not self.window or self.keep_first):
            raise ValueError("attention mixer: chunks have a size and no kept tokens")
        if self.sigmoid and (self.rel or self.softcap or self.sink):
            raise ValueError("attention mixer: sigmoid weights do not go with a bias by distance, a cap or a sink")
        if self.rel and (self.window or self.softcap or self.sink):
            raise ValueError("attention mixer: a bias by distance does not go with a window, a cap or a sink")

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
        out = ([("sink", (self.heads,))] if self.sink else []) + ([(n + "_b", (w,)) for n, w in self._qkv()] if self.bias else [])
        if self.qk_norm:
            out += [("q_norm", (self.dim,)), ("k_norm", (self.dim,))]
        if self.whole_norm:
            out += [("q_norm", (self.heads * self.dim,)), ("k_norm", (self.kv_heads * self.dim,))]
        if self.sigmoid:
            out.append(("weight_b", (self.heads, 1)))
        if self.rel:
            out += [("rel", (self.rel.rows, self.heads)), ("rel_by_distance", (self.heads, len(self.rel.rows_by_distance())))]
        return out

    def derive_(self, t) -> None:
        if self.rel:      # the table spread out by distance: what the attention kernels read
            t("rel_by_distance").copy_(t("rel")[torch.tensor(self.rel.rows_by_distance(), device=t("rel").device)].t())


@dataclass(frozen=True)
class LatentAttentionMixer:
    """Attention whose keys and values come from one latent vector per token, which is cached together with a rotated key part
    that all heads share; queries come from a latent of their own.  Per head: `dim` unrotated and `rot_dim` rotated query and
    key dimensions, values of `vdim`."""
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot_base: float
    gate: bool = True             # as in AttentionMixer
    interleaved: bool = False     # rotation pairs, as in AttentionMixer
    window: int = 0               # likewise
    sink: bool = False            # likewise
    kind = "latent"
    kv_heads = 1                  # as the cache sees it: one key, its first kv_rank columns the value

    def __post_init__(self):
        if self.rot_dim % 2 or min(self.heads, self.dim, self.vdim, self.q_rank, self.kv_rank) < 1:
            raise ValueError("latent attention mixer: sizes must be positive and rotated dimensions even")

    @property
    def qdim(self) -> int:
        return self.dim + self.rot_dim

    @property
    def width(self) -> int:
        """Of a cached row."""
        return self.kv_rank + self.rot_dim

    @property
    def out_width(self) -> int:
        return self.heads * self.vdim

    def projections(self) -> List[Tuple[str, int]]:
        return [("dq", self.q_rank), ("dkv", self.width)] + ([("g", self.heads)] if self.gate else [])

    def tensors(self) -> List[Tuple[str, Tuple[int, ...]]]:
        # uk and uv: blocks of a head stacked along their inputs (absorbed into queries and outputs); k_up and v_up: the
        # same matrices as one product from cached rows to the keys and the values of all heads
        H = self.heads
        return [("dq_norm", (self.q_rank,)), ("dkv_norm", (self.kv_rank,)), ("uq", (self.q_rank, H * self.qdim)),
                ("uk", (H * self.dim, self.kv_rank)), ("uv", (H * self.kv_rank, self.vdim)),
                ("k_up", (self.width, H * self.qdim)), ("v_up", (self.kv_rank, H * self.vdim))] + ([("sink", (H,))] if self.sink else [])

    def derive_(self, t) -> None:
        H, R = self.heads, self.kv_rank
        k = t("k_up").zero_().view(self.width, H, self.qdim)
        k[:R, :, :self.dim].copy_(t("uk").view(H, self.dim, R).permute(2, 0, 1))
        k[R:, :, self.dim:].copy_(torch.eye(self.rot_dim, dtype=k.dtype, device=k.device)[:, None, :].expand(-1, H, -1))
        t("v_up").view(R, H, self.vdim).copy_(t("uv").view(H, R, self.vdim).permute(1, 0, 2))


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


@dataclass(frozen=True)
class WKVMixer:
    """Linear attention with a decay per key channel that depends on the token, a bonus for the current token and a token shift:
    each of its five projections reads a mix of the token's row and the one before it."""
    hidden: int
    heads: int
    dim: int
    rank: int                     # of the decay projection
    kind = "wkv"
    MIXES = ("r", "k", "v", "g", "w")

    @property
    def vdim(self) -> int:
        return self.dim

    @property
    def out_width(self) -> int:
        return self.heads * self.dim

    def projections(self) -> List[Tuple[str, int]]:
        return []                 # (each has an input of its own)

    def tensors(self) -> List[Tuple[str, Tuple[int, ...]]]:
        # rkvg: the four projections stacked along their inputs, as the blocks of a block-diagonal product
        H, n = self.hidden, self.out_width
        return [("mu", (len(self.MIXES), H)), ("rkvg", (4 * H, n)), ("w1", (H, pad8(self.rank))), ("w2", (self.rank, n)), ("w0", (n,)),
                ("bonus", (n,)), ("o_norm", (n,))]

    def state_floats(self) -> int:
        return self.heads * self.dim * self.dim

    def zero_padding_(self, t) -> None:
        t("w1")[:, self.rank:] = 0


@dataclass(frozen=True)
class SSDMixer:
    """State-space recurrence with a decay per head behind a short convolution, gated and normed in `norm_groups` parts."""
    heads: int
    vdim: int
    state: int
    groups: int                   # of heads that share their input and output vectors
    taps: int
    norm_groups: int
    kind = "ssd"

    def __post_init__(self):
        if self.heads % self.groups or self.out_width % self.norm_groups or self.taps < 1:
            raise ValueError(f"state-space mixer: {self.heads} heads in {self.groups} groups, {self.norm_groups} norm groups, {self.taps} taps")

    @property
    def out_width(self) -> int:
        return self.heads * self.vdim

    @property
    def channels(self) -> int:
        """Of the convolution: x, B and C."""
        return self.out_width + 2 * self.groups * self.state

    def projections(self) -> List[Tuple[str, int]]:
        return [("z", self.out_width), ("xbc", self.channels), ("dt", self.heads)]

    def tensors(self) -> List[Tuple[str, Tuple[int, ...]]]:
        h = (self.heads,)
        return [("conv", (self.taps, self.channels)), ("conv_b", (self.channels,)), ("dt_bias", h), ("A_log", h), ("D", h),
                ("o_norm", (self.out_width,))]

    def state_floats(self) -> int:
        return self.heads * self.state * self.vdim


@dataclass(frozen=True)
class ParallelMixer:
    """Two mixers side by side on one input; half the sum of their outputs, each RMS-normed over the model's width.  The names of
    the left one's projections and tensors start with l_, the right one's with r_ (``out`` is the left one's output projection)."""
    hidden: int
    left: AttentionMixer
    right: SSDMixer
    kind = "parallel"

    def parts(self):
        return (("l_", self.left), ("r_", self.right))

    @property
    def out_width(self) -> int:
        return self.left.out_width

    @property
    def right_rows(self) -> int:
        return pad8(self.right.out_width)

    def projections(self) -> List[Tuple[str, int]]:
        return [(p + n, w) for p, m in self.parts() for n, w in m.projections()]

    def tensors(self) -> List[Tuple[str, Tuple[int, ...]]]:
        return [(p + n, shape) for p, m in self.parts() for n, shape in m.tensors()] + [
            ("r_out", (self.right_rows, self.hidden)), ("l_out_norm", (self.hidden,)), ("r_out_norm", (self.hidden,))]

    def derive_(self, t) -> None:
        for p, m in self.parts():
            if hasattr(m, "derive_"):
                m.derive_(lambda n, p=p: t(p + n))

    def zero_padding_(self, t) -> None:
        t("r_out")[self.right.out_width:] = 0


Mixer = Union[AttentionMixer, LatentAttentionMixer, GLAMixer, RGLRUMixer, WKVMixer, SSDMixer, ParallelMixer]
PAGED = ("attention", "latent")   # mixers with a paged cache; the others keep a state per sequence


def mixer_parts(m: Mixer) -> Tuple[Mixer, ...]:
    return (m.left, m.right) if m.kind == "parallel" else (m,)


@dataclass(frozen=True)
class ExpertsSpec:
    """Mixture of experts without biases: W_down act(W_up h), act = the square of relu, or W_down (silu(W_gate h) * W_up h).  A
    token goes to the `top` experts with the largest router scores (sigmoid of the logits, or their softmax; optionally
    divided by the sum of the chosen ones); the score multiplies the expert's input or its output.  A shared expert runs for
    every token and is added, multiplied by the sigmoid of a projection.

    Choices may be made by scores with a learned correction (the weights use them without it), and among the experts of the
    best groups only: `groups` equal ones of neighbours, of which the `keep` with the largest choice scores stay.  The last
    `identity` of the router's outputs are experts that return their input."""
    experts: int
    top: int
    ff: int
    shared_ff: int = 0            # 0: no shared expert
    weight_on_input: bool = True
    renormalize: bool = False
    gated: bool = False           # silu(gate) * up instead of the square of relu
    softmax: bool = False
    correction: bool = False
    identity: int = 0
    groups: int = 0               # 0: any expert can be chosen
    keep: int = 0

    def __post_init__(self):
        if not 1 <= self.top <= self.outputs or self.ff < 1 or self.experts < 1 or self.identity < 0:
            raise ValueError(f"{self.top} of {self.experts} experts (and {self.identity} identity ones) of width {self.ff}")
        if (self.gated or self.identity) and self.shared_ff:
            raise ValueError("a shared expert comes with plain experts only")
        if self.identity and self.weight_on_input:
            raise ValueError("identity experts go with weights on the output")
        if self.groups and (self.outputs % self.groups or not 1 <= self.keep <= self.groups
                            or self.keep * (self.outputs // self.groups) < self.top):
            raise ValueError(f"{self.keep} of {self.groups} groups over {self.outputs} experts, {self.top} chosen")

    @property
    def outputs(self) -> int:
        """Of the router, the shared expert's gate not counted."""
        return self.experts + self.identity

    @property
    def ff_pad(self) -> int:
        return (self.ff + 31) // 32 * 32 if self.gated else pad8(self.ff)

    @property
    def up_cols(self) -> int:
        """Columns of an expert's first matrix (gated: 32 of the gate and 32 of up in turn)."""
        return 2 * self.ff_pad if self.gated else self.ff_pad

    @property
    def shared_pad(self) -> int:
        return pad8(self.shared_ff)

    def gate_and_up(self, up: torch.Tensor) -> torch.Tensor:
        """View [.., ff_pad / 32, (gate, up), 32] of a gated first matrix."""
        return up.view(*up.shape[:-1], self.ff_pad // 32, 2, 32)

    @property
    def per_token(self) -> int:
        """Expert rows of a token, the shared expert's included."""
        return self.top + bool(self.shared_ff)

    @property
    def router_cols(self) -> int:
        return pad8(self.outputs + bool(self.shared_ff))


@dataclass(frozen=True)
class ClampedUnit:
    """A feed-forward's gated unit with biases: g = min(gate, limit), u = up within +- limit, g sigmoid(beta g) (u + 1)."""
    limit: float
    beta: float = 1.702

    def __post_init__(self):
        if not self.limit > 0:
            raise ValueError(f"clamped unit: the limit must be positive, not {self.limit}")


@dataclass(frozen=True)
class LayerSpec:
    mixer: Mixer
    ff: int = 0                   # width of the gated feed-forward beside the mixer; 0: none
    moe: Optional[ExpertsSpec] = None   # experts behind the mixer, with a norm of their own
    ff_after: int = 0             # width of a gated feed-forward behind the mixer, with a norm of its own; 0: none
    unit: Optional[ClampedUnit] = None  # its unit (None: silu(gate) * up, no biases)

    def __post_init__(self):
        if bool(self.ff) + bool(self.moe) + bool(self.ff_after) > 1:
            raise ValueError("a layer has a feed-forward beside its mixer, one behind it, or experts behind it")
        if self.unit and not self.ff_after:
            raise ValueError("a clamped unit belongs to a feed-forward behind the mixer")

    @property
    def sublayers(self) -> Tuple[int, ...]:
        """Numbers of the parts with a norm of their own."""
        return (1, 2) if self.moe or self.ff_after else (1,)

    @property
    def ff_after_pad(self) -> int:
        return pad8(self.ff_after)

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
    norm: str = "rms"             # "tanh": the dynamic-tanh norm, tanh(alpha x) w + b
    norm_scalar: bool = False     # a norm's weight is one number
    mix_taps: int = 0             # mixers read their input plus a causal convolution of it with this many taps; 0: none
    streams: int = 0              # residual streams joined by learned coefficients; 0: one, with plain sums
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
        if self.norm not in ("rms", "tanh") or (self.norm == "tanh" and not self.streams):
            raise ValueError(f"{self.name}: the dynamic-tanh norm comes with several streams")
        plain = self.norm == "tanh" or not self.streams
        if plain and (self.norm_scalar or self.mix_taps or any(s.mixer.kind in ("wkv", "parallel") or s.unit for s in self.layer_specs)):
            raise ValueError(f"{self.name}: scalar norms, convolved inputs, token shifts, mixers side by side and clamped units go with "
                             "several streams and RMS norms")
        if not plain and any(s.moe for s in self.layer_specs):
            raise ValueError(f"{self.name}: experts do not go with several streams and RMS norms")
        if any(s.mixer.kind == "ssd" for s in self.layer_specs):
            raise ValueError(f"{self.name}: a state-space mixer comes beside another mixer")
        if not 0 <= self.mix_taps <= 16 or any(getattr(p, "taps", 1) > 16 for s in self.layer_specs for p in mixer_parts(s.mixer)):
            raise ValueError(f"{self.name}: convolutions have up to 16 taps")
        if any(getattr(p, "hidden", self.hidden) != self.hidden for s in self.layer_specs for p in (s.mixer,)):
            raise ValueError(f"{self.name}: a mixer is built for another width")
        if not 0 <= self.streams <= 8:
            raise ValueError(f"{self.name}: at most 8 streams")
        if self.streams and (lp is not None or any(s.ff or (s.moe and s.moe.shared_ff) for s in self.layer_specs)):
            raise ValueError(f"{self.name}: streams go with layers that run once, feed-forwards behind the mixer and no shared expert")
        if not self.streams and (any(s.ff_after for s in self.layer_specs) or any(s.moe and s.moe.identity for s in self.layer_specs)):
            raise ValueError(f"{self.name}: feed-forwards behind the mixer and identity experts go with streams")
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

    def run_parts(self) -> List[Mixer]:
        """The same with mixers side by side one by one."""
        return [p for m in self.run_mixers() for p in mixer_parts(m)]

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
        per = lambda m: m.width if m.kind == "latent" else m.kv_heads * (m.dim + m.vdim) if m.kv_from is None else 0
        return sum(per(m) * elem for m in self.run_parts() if m.kind in PAGED)

    def state_bytes_per_sequence(self, elem: int = 2) -> int:
        n = 4 * max(0, self.mix_taps - 1) * self.hidden * len(self.runs())
        for m in self.run_parts():
            if m.kind == "gla":
                n += 4 * m.state_floats()
            elif m.kind == "wkv":
                n += 4 * (m.state_floats() + m.hidden)
            elif m.kind == "ssd":
                n += 4 * m.state_floats() + elem * (m.taps - 1) * m.channels
            elif m.kind == "rglru":
                n += 4 * m.width + elem * (m.taps - 1) * m.width
        return n

    def attention_work(self, length: int) -> Tuple[int, int]:
        """(KV heads, positions) of the attention run with the fewest heads and of the one that looks furthest back, for a
        sequence of `length` tokens: what the number of key splits is chosen from.  (0, 0) without attention."""
        a = [m for m in self.run_parts() if m.kind in PAGED]
        if not a:
            return 0, 0
        span = max(min(length, m.window + getattr(m, "keep_first", 0)) if getattr(m, "window", 0) else length for m in a)
        return min(m.kv_heads for m in a), span

    @property
    def recurrent(self) -> bool:
        return self.mix_taps > 1 or any(m.kind not in PAGED for m in self.run_parts())

    @property
    def vocab_pad(self) -> int:
        return pad8(self.vocab)

    def init_(self, name: str, v: torch.Tensor, rand) -> None:
        """Random weights with activations of order one; `rand(shape)` gives normal numbers on v's device."""
        leaf = name.rsplit(".", 1)[-1]
        if leaf.startswith(("l_", "r_")):                    # one of two mixers side by side
            leaf = leaf[2:]
        if leaf.endswith("norm_alpha") or leaf in ("norm1_alpha", "norm2_alpha"):
            x = 0.7 + 0.1 * rand(v.shape)
        elif leaf in ("norm1_b", "norm2_b", "final_norm_b", "rel", "correction"):
            x = 0.1 * rand(v.shape)
        elif leaf in ("hc1_in", "hc2_in"):
            x = 1.0 / v.numel() + 0.2 * rand(v.shape)
        elif leaf in ("hc1_out", "hc2_out"):
            x = 1.0 + 0.2 * rand(v.shape)
        elif leaf in ("hc1_mix", "hc2_mix"):
            x = torch.eye(v.shape[0], device=v.device) + 0.1 * rand(v.shape)
        elif leaf == "mu":
            x = 0.5 + 0.2 * rand(v.shape)
        elif leaf == "rkvg":                                 # four matrices stacked along their inputs
            x = rand(v.shape) * (v.shape[0] // 4) ** -0.5
        elif leaf in ("w0", "dt_bias", "weight_b"):
            x = -2.0 + 0.5 * rand(v.shape)
        elif leaf in ("bonus", "A_log"):
            x = 0.5 * rand(v.shape)
        elif leaf in ("gate_up_b", "down_b"):
            x = 0.1 * rand(v.shape)
        elif leaf in ("q_norm", "k_norm", "dq_norm", "dkv_norm", "D", "out_norm"):
            x = 1.0 + 0.1 * rand(v.shape)
        elif leaf == "uk":                                   # stacked by head: [heads * dim, rank], the rank is the input
            x = rand(v.shape) * v.shape[1] ** -0.5
        elif leaf == "uv":
            x = rand(v.shape) * (v.shape[0] // self.layer_specs[int(name.split(".")[1])].mixer.heads) ** -0.5
        elif leaf in ("norm1", "norm2", "final_norm"):
            x = 1.0 - self.norm_offset + 0.1 * rand(v.shape)
        elif leaf == "o_norm":
            x = 1.0 + 0.1 * rand(v.shape)
        elif leaf == "a2_b":
            x = 2.0 + rand(v.shape)                          # slow decays with some fast channels
        elif leaf == "lam":
            x = -4.0 + rand(v.shape)                         # a between about 0.8 and 0.99
        elif leaf in ("x_b", "y_b", "conv_b", "gate_b", "sink", "loop_step", "q_b", "k_b", "v_b"):
            x = 0.2 * rand(v.shape)
        elif leaf in ("up", "down") and self.layer_specs[int(name.split(".")[1])].moe:   # experts stacked along their inputs
            moe = self.layer_specs[int(name.split(".")[1])].moe
            n = v.shape[0] // moe.experts
            for e in range(moe.experts):
                v[e * n:(e + 1) * n].copy_((rand((n, v.shape[1])) * n ** -0.5).to(v.dtype))
            return
        elif leaf in ("conv", "mix_conv"):
            x = rand(v.shape) * v.shape[0] ** -0.5
        elif leaf == "embed":
            x = rand(v.shape)
        elif leaf == "gates":
            x = rand(v.shape) * (v.shape[1] // 2) ** -0.5
        else:
            x = rand(v.shape) * v.shape[0] ** -0.5
        v.copy_(x.to(v.dtype))

    def derive_(self, tensors) -> None:
        """Fill the tensors that are other forms of stored ones (name -> tensor); every way of filling a segment ends here."""
        for l, s in enumerate(self.layer_specs):
            if hasattr(s.mixer, "derive_"):
                s.mixer.derive_(lambda n, l=l: tensors[f"layers.{l}.{n}"])

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
            if s.ff_after:
                tensors[p + "down"][s.ff_after:] = 0
            if s.unit:
                b = tensors[p + "gate_up_b"]
                b[s.ff_after:s.ff_after_pad] = 0
                b[s.ff_after_pad + s.ff_after:] = 0
            if hasattr(s.mixer, "zero_padding_"):
                s.mixer.zero_padding_(lambda n, p=p: tensors[p + n])
            n, pad = (s.ff, s.ff_pad) if s.ff else (s.ff_after, s.ff_after_pad)
            if n:
                g = tensors[p + "gate_up"]
                g[:, n:pad] = 0
                g[:, pad + n:] = 0
            if s.moe:
                e = s.moe
                tensors[p + "router"][:, e.outputs + bool(e.shared_ff):] = 0
                if not e.gated:
                    tensors[p + "up"][:, e.ff:] = 0
                elif e.ff % 32:
                    e.gate_and_up(tensors[p + "up"])[:, -1, :, e.ff % 32:] = 0
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

    def add_norm(name):
        add(name, (1,) if cfg.norm_scalar else (cfg.hidden,))
        if cfg.norm == "tanh":
            add(name + "_b", (cfg.hidden,))
            add(name + "_alpha", (1,))

    start = cur
    add("embed", (cfg.vocab, cfg.hidden))
    if cfg.loop is not None:
        add("loop_step", (cfg.loop.times, cfg.hidden))
    lay.units.append(("embed", start, cur - start))
    for l, s in enumerate(cfg.layer_specs):
        start, p = cur, f"layers.{l}."
        add_norm(p + "norm1")
        if cfg.mix_taps:
            add(p + "mix_conv", (cfg.mix_taps, cfg.hidden))
        add(p + "in", (cfg.hidden, s.in_columns()[1]))
        for n, shape in s.mixer.tensors():
            add(p + n, shape)
        add(p + "out", (s.out_rows, cfg.hidden))
        if s.ff:
            add(p + "gate_up", (cfg.hidden, 2 * s.ff_pad))
        if s.moe:
            e = s.moe
            add_norm(p + "norm2")
            add(p + "router", (cfg.hidden, e.router_cols))
            if e.correction:
                add(p + "correction", (e.outputs,))
            add(p + "up", (e.experts * cfg.hidden, e.up_cols))
            add(p + "down", (e.experts * e.ff_pad, cfg.hidden))
            if e.shared_ff:
                add(p + "shared_up", (cfg.hidden, e.shared_pad))
                add(p + "shared_down", (e.shared_pad, cfg.hidden))
        if s.ff_after:
            add_norm(p + "norm2")
            add(p + "gate_up", (cfg.hidden, 2 * s.ff_after_pad))
            add(p + "down", (s.ff_after_pad, cfg.hidden))
        if s.unit:
            add(p + "gate_up_b", (2 * s.ff_after_pad,))
            add(p + "down_b", (cfg.hidden,))
        if cfg.streams:
            for q in s.sublayers:
                for n, shape in (("in", (cfg.streams,)), ("out", (cfg.streams,)), ("mix", (cfg.streams, cfg.streams))):
                    add(f"{p}hc{q}_{n}", shape)
        lay.units.append((f"layer.{l}", start, cur - start))
    start = cur
    add_norm("final_norm")
    add("lm_head", (cfg.hidden, cfg.vocab_pad))
    lay.units.append(("head", start, cur - start))
    lay.total_bytes = cur
    return lay
