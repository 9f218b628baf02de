"""Komulorn on the host: configuration, weight mapping, shared caches, and checks of the plain oracle itself (every planted
mistake shows in the inputs that the GPU tests use)."""
import functools
import json
import math

import pytest
import torch

import komulorn_cases as cases
from komulorn_plain import FLAWS, Plain, rotate_half, yarn_frequencies


@pytest.mark.parametrize("name", sorted(cases.CASES))
def test_checkpoint_round_trip_and_layout(tmp_path, name):
    from blitz_scale_b200.models.config import get_config
    from blitz_scale_b200.models.convert import CheckpointReader, checkpoint_to_segment, convert, verify
    from blitz_scale_b200.models.komulorn import from_segment
    c = cases.CASES[name]
    w = cases.weights(c)
    d = cases.write(tmp_path / "ckpt", c, w)
    cfg = get_config(d)
    assert cfg.family == "hybrid" and cfg.vocab == c["vocab"] and cfg.layers == len(c["layers"]) and not cfg.recurrent
    seg = checkpoint_to_segment(CheckpointReader(d), cfg)
    back = from_segment(seg)
    assert set(back) == set(w) and all(torch.equal(back[n], w[n]) for n in w)
    assert [n for n, _, _ in seg.layout.units] == ["embed"] + [f"layer.{i}" for i in range(cfg.layers)] + ["head"]
    at = 0
    for _, off, nb in seg.layout.units:
        assert off == at
        at += nb
    assert at == seg.layout.total_bytes
    before = seg.buffer.clone()
    cfg.zero_padding_({n: seg[n] for n in seg.names()})
    assert torch.equal(before, seg.buffer)
    convert(d, d, tmp_path / "seg")
    assert verify(d, d, tmp_path / "seg") == []


def test_shared_caches():
    from blitz_scale_b200.models.komulorn import parse_config
    from blitz_scale_b200.runtime.hybrid_cache import HybridCache
    cfg = parse_config(cases.CASES["regular"])
    assert cfg.kv_runs() == [0, 1, 0, 0, 1]
    assert cfg.kv_bytes_per_token() == 2 * 2 * (64 + 32) * 2
    cache = HybridCache(cfg, 5, 16, 1, torch.bfloat16, "cpu")
    k = [r.kv.k.data_ptr() for r in cache.runs]
    assert k[0] == k[2] == k[3] != k[1] == k[4] and cache.runs[0].kv.v.shape == (5, 16, 2, 32)
    assert cache.bytes() == 5 * 16 * cfg.kv_bytes_per_token()
    assert HybridCache(parse_config(cases.CASES["plain"]), 5, 16, 1, torch.bfloat16, "cpu").runs[1].kv.shape == (5, 2, 16, 2, 64)


def test_refusals(tmp_path):
    from blitz_scale_b200.models.convert import CheckpointReader, checkpoint_to_segment
    from blitz_scale_b200.models.config import get_config
    from blitz_scale_b200.models.hybrid_config import ExpertsSpec
    from blitz_scale_b200.models.komulorn import parse_config
    at, mo = cases.attention, cases.moe
    for mixers in ([at(kv_from=0)], [at(), at(kv_from=1)], [at(), at(kv_from=0), at(kv_from=1)], [at(), at(vdim=64, kv_from=0)],
                   [at(heads=4, kv_heads=4), at(heads=4, kv_heads=2, kv_from=0)]):
        with pytest.raises(ValueError):
            parse_config(cases.config(mixers, [None] * len(mixers)))
    c = cases.config([at()], [mo()])
    for path, value in ((("type",), "other"), (("mlp", "kind"), "other")):
        bad = json.loads(json.dumps(c))
        t = bad["layers"][0]
        for n in path[:-1]:
            t = t[n]
        t[path[-1]] = value
        with pytest.raises(ValueError):
            parse_config(bad)
    with pytest.raises(ValueError):
        ExpertsSpec(4, 5, 8)
    w = cases.weights(c)
    w["l0.mlp.e1.up"] = w["l0.mlp.e1.up"][:-1].clone()
    d = cases.write(tmp_path, c, w)
    with pytest.raises(ValueError, match="l0.mlp.e1.up"):
        checkpoint_to_segment(CheckpointReader(d), get_config(d))


def test_registry_shapes():
    from blitz_scale_b200.models.config import get_config
    from blitz_scale_b200.models.weights import WeightSegment
    for n in ("komulorn_tiny", "komulorn_odd"):
        cfg = get_config(n)
        seg = WeightSegment(cfg).random_init_(3)
        assert all(torch.isfinite(seg[t].float()).all() for t in seg.names())
        assert not torch.equal(seg["lm_head"][:, :cfg.vocab], seg["embed"].t()) and not seg["lm_head"][:, cfg.vocab:].any()
        e = cfg.layer_specs[0].moe
        assert not seg["layers.0.down"].view(e.experts, e.ff_pad, -1)[:, e.ff:].any()
    big = get_config("komulorn_13b")
    assert big.kv_runs()[:4] == [0, 0, 2, 2] and big.kv_bytes_per_token() == 16 * 2 * 4 * 128 * 2
    assert big.attention_work(10 ** 5) == (4, 10 ** 5)


def test_scaled_frequencies():
    """Product code against the oracle's own formula, where both ends of the ramp, neither, or only clipped ones lie inside."""
    from blitz_scale_b200.models.hybrid_config import YarnScaling
    seen = set()
    for dims, base, sc in ((64, 1e4, (4.0, 2048, 32.0, 1.0)), (16, 300.0, (2.0, 40, 8.0, 2.0)), (2, 5e4, (3.0, 128, 32.0, 1.0)),
                           (128, 1e6, (8.0, 300, 100.0, 0.5)), (32, 1e4, (1.0, 64, 1.0, 1.0)), (8, 10.0, (2.0, 1e6, 4.0, 2.0))):
        y = YarnScaling(*sc)
        want, gain = yarn_frequencies(dims, base, dict(zip(("factor", "original", "fast", "slow"), sc)))
        plain, _ = yarn_frequencies(dims, base, None)
        got = [p * s for p, s in zip(plain, y.stretch(dims, base))]
        assert all(math.isclose(a, b, rel_tol=1e-13) for a, b in zip(got, want)) and math.isclose(gain, y.gain, rel_tol=1e-15)
        seen.add((got[0] == plain[0], math.isclose(got[-1], plain[-1] / sc[0], rel_tol=1e-12)))
    assert seen == {(True, False), (True, True)}
    x = torch.randn(5, 2, 6, dtype=torch.float64)
    r = rotate_half(x, {"dims": 4, "base": 100.0})
    assert torch.equal(r[..., 4:], x[..., 4:]) and torch.equal(r[0], x[0])
    a = 3 * 100.0 ** (-2 / 4)
    assert abs(float(r[3, 0, 1] - (x[3, 0, 1] * math.cos(a) - x[3, 0, 3] * math.sin(a)))) < 1e-12


@functools.lru_cache(maxsize=None)
def _good(name):
    c = cases.CASES[name]
    toks = tuple(torch.randint(0, c["vocab"], (300,), generator=torch.Generator().manual_seed(2)).tolist())
    return toks, Plain(c, cases.weights(c, 1), torch.float32).run(list(toks))


@pytest.mark.parametrize("flaw", FLAWS)
def test_every_planted_mistake_shows(flaw):
    """The inputs the GPU tests use would reveal each mistake, far above the tolerance of the 16-bit comparison."""
    name = "values" if flaw == "yarn_unclipped" else "regular"
    toks, good = _good(name)
    c = cases.CASES[name]
    bad = Plain(c, cases.weights(c, 1), torch.float32, [flaw]).run(list(toks))
    err = ((good - bad).pow(2).mean(-1) / good.pow(2).mean()).sqrt()
    assert float(err.max()) > 0.1, (flaw, float(err.max()))
    if flaw == "far_key_lost":
        assert float(err[:128].max()) == 0.0
