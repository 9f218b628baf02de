"""Model shape registry and the per-rank weight-segment layout.

The registry mirrors the shapes the reference serves (src/model/common_hyper.h:11-177:
OPT, Llama-2 7B/13B/70B, Llama-3 8B, Mistral 13B/24B, Qwen 72B) plus the tiny shapes used by
the CPU plumbing configuration and the GPU unit tests.  Only the Llama architecture (pre-RMSNorm,
RoPE, GQA, SwiGLU, no biases) is executed from these records, as in the reference, where every served
model goes through the Llama hyper-parameter constructor.  Models whose layers differ have records of
their own (hybrid_config.py); `get_config` finds both, and reads checkpoint folders.

Weight segment (one contiguous allocation per GPU = per TP rank, every matrix stored ``[in, out]``
row-major, cf. src/model/llama.h:139-218 and scripts/util/make_dangertensors.py:9-30)::

    embed_tokens [vocab/tp, hidden]
    L x { input_ln [hidden] | qkv^T [hidden, (qh + 2 kvh)/tp * hd] | o^T [qh/tp * hd, hidden]
          | post_ln [hidden] | gate_up^T [hidden, 2 inter/tp] | down^T [inter/tp, hidden] }
    final_norm [hidden] | lm_head^T [hidden, vocab/tp]

Transfer units are ``embed | layer 0..L-1 | head`` (src/model/llama.h:236-246).  Two deliberate
differences from the reference layout: q, k and v projections are stored as one fused matrix whose
rows are ``[q | k | v]`` (one GEMM instead of two), and every tensor starts on a 256-byte boundary
(TMA operands need 16-byte alignment; 256 keeps copies sector-aligned).
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Dict, List, Tuple

ALIGN_BYTES = 256


@dataclass(frozen=True)
class ModelConfig:
    name: str
    vocab: int
    hidden: int
    layers: int
    q_heads: int
    kv_heads: int
    head_dim: int
    inter: int
    rope_theta: float = 10000.0
    rms_eps: float = 1e-5
    max_positions: int = 16384
    param_gb: float = 0.0  # size used for flow accounting by the router
    eos_token: int = -1    # end-of-sequence id of the family's tokenizer (-1: none known); workers stop a request there
                           # unless it sets ignore_eos_token
    family = "llama"       # which runner executes it (hybrid_config.HybridConfig has "hybrid")
    recurrent = False      # no per-sequence state beside the KV cache

    def kv_bytes_per_token(self, tp: int = 1, elem: int = 2) -> int:
        return 2 * (self.kv_heads // tp) * self.head_dim * elem * self.layers


# end-of-sequence ids of the published tokenizers: </s> = 2 (Llama-2, Mistral, OPT), <|end_of_text|> = 128001 (Llama-3),
# <|endoftext|> = 151643 (Qwen-2.5); a chat-tuned checkpoint that ends turns with another id sets --eos-token-id
_EOS = {"llama2": 2, "llama3": 128001, "mistral": 2, "qwen": 151643, "opt": 2, "tiny": 2}


def _c(name, vocab, hidden, layers, qh, kvh, inter, theta=10000.0, hd=None, gb=0.0, eps=1e-5):
    return ModelConfig(name, vocab, hidden, layers, qh, kvh, hd or hidden // qh, inter, theta, eps, 16384, gb,
                       _EOS.get(name.split("_")[0], -1))


REGISTRY: Dict[str, ModelConfig] = {c.name: c for c in [
    # CPU plumbing shape of the first benchmark configuration (2 layers, hidden 256, 4/2 heads, FFN 688)
    _c("tiny", 32000, 256, 2, 4, 2, 688),
    # smallest shape the tcgen05 attention (head_dim 128) accepts; used by GPU tests and smoke()
    _c("tiny_gpu", 4096, 512, 2, 4, 2, 1408, theta=5e5),
    _c("tiny_gpu_deep", 4096, 512, 8, 4, 2, 1408, theta=5e5),
    _c("tiny_gpu_wide", 4096, 1024, 2, 8, 4, 2816, theta=5e5),
    _c("opt_125m", 50272, 768, 12, 12, 12, 3072),
    _c("opt_1.3b", 50272, 2048, 24, 32, 32, 8192),
    _c("opt_6.7b", 50272, 4096, 32, 32, 32, 16384),
    _c("opt_13b", 50272, 5120, 40, 40, 40, 20480),
    _c("opt_30b", 50272, 7168, 48, 56, 56, 28672),
    _c("llama2_7b", 32000, 4096, 32, 32, 32, 11008, gb=14),
    _c("llama2_13b", 32000, 5120, 40, 40, 40, 13824, gb=26),
    _c("llama2_70b", 32000, 8192, 80, 64, 8, 28672, gb=140),
    _c("llama3_8b", 128256, 4096, 32, 32, 8, 14336, theta=5e5, gb=16),
    _c("mistral_13b", 32000, 5120, 40, 40, 8, 14336, theta=1e6, gb=26),
    _c("mistral_24b", 131072, 5120, 40, 32, 8, 32768, theta=1e8, hd=128, gb=48),
    _c("qwen_72b", 152064, 8192, 80, 64, 8, 29568, theta=1e6, gb=145, eps=1e-6),
]}


def hybrid_registry():
    """Shapes of the models whose layers differ (a separate table: the native twin of the registry holds the uniform ones)."""
    from . import komulorn, norusun, vofidra
    from .fafudra import shape_config
    mixed = ("gla", "attention", "rglru", "gla")
    return {c.name: c for c in [
        # small shapes for tests: one with the sizes the tensor-core kernels take, one with sizes that none of them take
        shape_config("fafudra_tiny", 2048, 256, mixed, 512, heads=4, kv_heads=2, dim=64, window=96, gla_heads=4, gla_dim=32,
                     gla_vdim=64, width=256, blocks=4, loop=(1, 3, 2)),
        shape_config("fafudra_odd", 1003, 120, mixed, 100, heads=6, kv_heads=2, dim=20, window=50, gla_heads=3, gla_dim=12,
                     gla_vdim=20, rank=5, width=90, blocks=3, loop=(0, 2, 2)),
        # layer sizes of the 8 B Llama shape
        shape_config("fafudra_8b", 128256, 4096, mixed * 8, 14336, heads=32, kv_heads=8, dim=128, window=2048,
                     gla_heads=16, gla_dim=128, gla_vdim=256, width=4096, blocks=16, gb=16),
        # attention with shared key/value caches and experts: a test shape for the tensor-core kernels, one whose sizes none
        # of them takes, and one of 13 B parameters, a mixture of experts
        komulorn.shape_config("komulorn_tiny", 2048, 320, 4, heads=4, kv_heads=2, dim=64, vdim=32, rot_dims=32, experts=8, top=2,
                              ff=128, shared_ff=192),
        komulorn.shape_config("komulorn_odd", 1003, 122, 3, heads=9, kv_heads=3, dim=22, vdim=13, rot_dims=10, experts=5, top=3,
                              ff=51, shared_ff=30, share=3),
        komulorn.shape_config("komulorn_13b", 128256, 2048, 32, heads=32, kv_heads=4, dim=128, vdim=128, rot_dims=64, experts=64,
                              top=6, ff=1408, shared_ff=2816, gb=27),
        # several residual streams, attention with a bias by distance, latent attention, a mixture of experts with identity
        # experts: likewise, the last one of 13 B parameters
        vofidra.shape_config("vofidra_tiny", 2048, 320, 4, heads=8, kv_heads=2, dim=64, latent=dict(heads=4, dim=64, rot_dim=32, vdim=64,
                             q_rank=192, kv_rank=128), experts=10, identity=6, top=4, groups=4, keep=2, ff=96, dense_ff=512, streams=2),
        vofidra.shape_config("vofidra_odd", 1003, 122, 3, heads=6, kv_heads=3, dim=22, latent=dict(heads=3, dim=13, rot_dim=6, vdim=11,
                             q_rank=35, kv_rank=21), experts=5, identity=1, top=3, groups=3, keep=2, ff=51, dense_ff=77, streams=3),
        vofidra.shape_config("vofidra_13b", 128256, 2048, 28, heads=16, kv_heads=4, dim=128, latent=dict(heads=32, dim=64, rot_dim=32,
                             vdim=64, q_rank=768, kv_rank=256), experts=48, identity=16, top=6, groups=8, keep=4, ff=1536,
                             dense_ff=8192, streams=4, gb=26),
        # several residual streams with scalar norms and convolved mixer inputs; linear attention with a token shift, latent
        # attention in a window, attention without softmax beside a state space: likewise, the last one of 8 B parameters
        norusun.shape_config("norusun_tiny", 2048, 320, ("wkv", "latent_attention", "parallel", "wkv"), 512, wkv=(5, 64, 24),
                             latent=dict(heads=4, dim=64, rot_dim=32, vdim=64, q_rank=192, kv_rank=128, window=70), heads=8, kv_heads=2,
                             dim=64, chunk=96, ssd=dict(heads=6, vdim=64, state=64, groups=2, taps=4, norm_groups=3), streams=2, taps=4),
        norusun.shape_config("norusun_odd", 1003, 122, ("parallel", "wkv", "latent_attention"), 77, wkv=(3, 13, 5),
                             latent=dict(heads=3, dim=13, rot_dim=6, vdim=11, q_rank=35, kv_rank=21, window=19), heads=6, kv_heads=3,
                             dim=22, vdim=17, rot_dims=10, chunk=23, ssd=dict(heads=5, vdim=7, state=9, groups=1, taps=3, norm_groups=5),
                             streams=3, taps=2),
        norusun.shape_config("norusun_8b", 128256, 4096, ("wkv", "latent_attention", "parallel", "latent_attention") * 8, 14336, wkv=(32, 128, 64),
                             latent=dict(heads=32, dim=96, rot_dim=32, vdim=128, q_rank=1024, kv_rank=512, window=2048), heads=32,
                             kv_heads=8, dim=128, chunk=2048,
                             ssd=dict(heads=64, vdim=64, state=128, groups=8, taps=4, norm_groups=8), streams=2, taps=4, gb=16),
    ]}


# designs described by data: "architecture" of config.json -> module of this package with parse_config and to_segment
DESIGNS = {"Fafudra": "fafudra", "Komulorn": "komulorn", "Vofidra": "vofidra", "Norusun": "norusun"}


def design_module(name: str):
    import importlib
    return importlib.import_module("." + name, __package__)


def config_from_dir(path):
    """Configuration of a checkpoint folder whose config.json names an architecture this package describes by data."""
    import json
    from pathlib import Path
    from .convert import list_checkpoint
    d = Path(path)
    c = json.loads((d / "config.json").read_text())
    arch = c.get("architecture")
    if arch not in DESIGNS:
        raise KeyError(f"{d / 'config.json'}: unknown architecture {arch!r}; known: {sorted(DESIGNS)}")
    shapes = {n: shape for n, _, shape in list_checkpoint(d)}
    return design_module(DESIGNS[arch]).parse_config(c, shapes, name=d.resolve().name)


def get_config(name: str):
    """A model by registry name, or by the path of a checkpoint folder with a config.json."""
    import os
    if name in REGISTRY:
        return REGISTRY[name]
    hybrid = hybrid_registry()
    if name in hybrid:
        return hybrid[name]
    if os.path.isfile(os.path.join(str(name), "config.json")):
        return config_from_dir(name)
    raise KeyError(f"unknown model {name!r}; known: {sorted(REGISTRY) + sorted(hybrid)}, or a folder with config.json")


@dataclass
class TensorSpec:
    name: str
    shape: Tuple[int, ...]
    offset: int  # bytes from the start of the segment
    nbytes: int


@dataclass
class SegmentLayout:
    """Byte offsets of every tensor and of the transfer units of one TP rank's segment."""
    cfg: ModelConfig
    tp: int
    elem_bytes: int
    tensors: Dict[str, TensorSpec] = field(default_factory=dict)
    units: List[Tuple[str, int, int]] = field(default_factory=list)  # (name, offset, nbytes)
    total_bytes: int = 0

    def unit(self, name: str) -> Tuple[int, int]:
        for n, off, nb in self.units:
            if n == name:
                return off, nb
        raise KeyError(name)


def _align(x: int, a: int = ALIGN_BYTES) -> int:
    return (x + a - 1) // a * a


def layer_tensor_shapes(cfg: ModelConfig, tp: int) -> List[Tuple[str, Tuple[int, ...]]]:
    qh, kvh, hd = cfg.q_heads // tp, cfg.kv_heads // tp, cfg.head_dim
    return [
        ("input_ln", (cfg.hidden,)),
        ("qkv", (cfg.hidden, (qh + 2 * kvh) * hd)),
        ("o", (qh * hd, cfg.hidden)),
        ("post_ln", (cfg.hidden,)),
        ("gate_up", (cfg.hidden, 2 * (cfg.inter // tp))),
        ("down", (cfg.inter // tp, cfg.hidden)),
    ]


def build_layout(cfg: ModelConfig, tp: int = 1, elem_bytes: int = 2) -> SegmentLayout:
    if cfg.family == "hybrid":
        from .hybrid_config import build_hybrid_layout
        return build_hybrid_layout(cfg, tp, elem_bytes)
    if cfg.q_heads % tp or cfg.kv_heads % tp or cfg.inter % tp or cfg.vocab % tp:
        raise ValueError(f"{cfg.name}: heads/inter/vocab not divisible by tp={tp}")
    lay = SegmentLayout(cfg, tp, elem_bytes)
    cur = 0

    def add(name, shape):
        nonlocal cur
        n = 1
        for s in shape:
            n *= s
        nb = n * elem_bytes
        lay.tensors[name] = TensorSpec(name, tuple(shape), cur, nb)
        cur = _align(cur + nb)

    start = cur
    add("embed", (cfg.vocab // tp, cfg.hidden))
    lay.units.append(("embed", start, cur - start))
    for l in range(cfg.layers):
        start = cur
        for n, shp in layer_tensor_shapes(cfg, tp):
            add(f"layers.{l}.{n}", shp)
        lay.units.append((f"layer.{l}", start, cur - start))
    start = cur
    add("final_norm", (cfg.hidden,))
    add("lm_head", (cfg.hidden, cfg.vocab // tp))
    lay.units.append(("head", start, cur - start))
    lay.total_bytes = cur
    return lay
