"""Vofidra on the host: configuration, weight mapping, derived tensors, and checks of the plain oracle itself (every planted
mistake shows in the inputs that the GPU tests use)."""
import functools
import json
import math

import pytest
import torch

import vofidra_cases as cases
from vofidra_plain import FLAWS, Plain, bucket, dyt, route, streams_in, streams_out


@pytest.mark.parametrize("name", sorted(cases.CASES))
def test_checkpoint_round_trip_and_layout(tmp_path, name):
    from blitz_scale_b200.models.config import get_config
    from blitz_scale_b200.models.convert import CheckpointReader, checkpoint_to_segment, convert, verify
    from blitz_scale_b200.models.vofidra import from_segment
    c = cases.CASES[name]
    w = cases.weights(c)
    d = cases.write(tmp_path / "ckpt", c, w)
    cfg = get_config(d)
    assert cfg.family == "hybrid" and cfg.vocab == c["vocab"] and cfg.layers == len(c["layers"]) and not cfg.recurrent
    assert cfg.streams == c["streams"] and cfg.norm == "tanh"
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
    cfg.derive_(seg)
    assert torch.equal(before, seg.buffer)
    convert(d, d, tmp_path / "seg")
    assert verify(d, d, tmp_path / "seg") == []


def test_derived_tensors():
    """Keys and values of all heads from one cached row, and the bias of every distance."""
    from blitz_scale_b200.models.vofidra import parse_config, to_segment
    c = cases.CASES["regular"]
    w = cases.weights(c, dtype=torch.float32)

    class Reader:
        get = staticmethod(lambda n: w[n])
    cfg = parse_config(c, {n: tuple(t.shape) for n, t in w.items()})
    seg = to_segment(Reader, cfg, torch.float32)
    m = cfg.layer_specs[1].mixer
    row = torch.randn(m.width)
    k = (row @ seg["layers.1.k_up"]).view(m.heads, m.qdim)
    assert torch.allclose(k[:, :m.dim], (w["l1.mix.uk"] @ row[:m.kv_rank]).view(m.heads, -1), atol=1e-4)
    assert torch.equal(k[:, m.dim:], row[m.kv_rank:].expand(m.heads, -1))
    assert torch.allclose(row[:m.kv_rank] @ seg["layers.1.v_up"], w["l1.mix.uv"] @ row[:m.kv_rank], atol=1e-4)
    by = seg["layers.0.rel_by_distance"]
    for n in (0, 1, 9, 10, 11, 50, 98, 99, 100, 101, 5000):
        want = w["l0.mix.rel"][bucket(n, 20, 100)]
        assert torch.equal(by[:, min(n, by.shape[1] - 1)], want), n


def test_distance_rows():
    """Product code against the oracle's formula: odd and even tables, the last row reached early, late, and at once."""
    from blitz_scale_b200.models.hybrid_config import DistanceBias
    for rows, far in ((2, 2), (3, 2), (7, 12), (9, 33), (16, 128), (20, 100), (32, 4096), (64, 33), (33, 1000)):
        got = DistanceBias(rows, far).rows_by_distance()
        assert got[-1] == rows - 1 and rows - 1 not in got[:-1] and got == sorted(got)
        at = lambda n: got[min(n, len(got) - 1)]
        assert all(at(n) == bucket(n, rows, far) for n in list(range(2 * far)) + [10 ** 6])
    for rows, far in ((1, 10), (8, 4), (8, 3)):
        with pytest.raises(ValueError):
            DistanceBias(rows, far)


def test_cache_and_work():
    from blitz_scale_b200.models.vofidra import parse_config
    from blitz_scale_b200.ops import LatentKV
    from blitz_scale_b200.runtime.hybrid_cache import HybridCache
    c = cases.CASES["regular"]
    cfg = parse_config(c, {n: tuple(t.shape) for n, t in cases.weights(c).items()})
    assert cfg.kv_bytes_per_token() == 2 * (2 * 3 * 128 + 104 + 32 + 64 + 16) and cfg.kv_runs() == [0, 1, 2, 3]
    cache = HybridCache(cfg, 5, 16, 1, torch.bfloat16, "cpu")
    assert isinstance(cache.runs[1].kv, LatentKV) and cache.runs[1].kv.pool.shape == (5, 16, 1, 136) and cache.runs[0].kv.shape == (5, 2, 16, 3, 64)
    assert cache.bytes() == 5 * 16 * cfg.kv_bytes_per_token()
    assert cfg.attention_work(5000) == (1, 5000)


def test_refusals(tmp_path):
    from blitz_scale_b200.models.config import get_config
    from blitz_scale_b200.models.convert import CheckpointReader, checkpoint_to_segment
    from blitz_scale_b200.models.hybrid_config import AttentionMixer, DistanceBias, ExpertsSpec, HybridConfig, LayerSpec, QueryTemperature
    from blitz_scale_b200.models.vofidra import parse_config
    c = cases.config([cases.attention(), cases.latent()], [cases.moe(), cases.dense()])
    w = cases.weights(c)
    shapes = {n: tuple(t.shape) for n, t in w.items()}
    parse_config(c, shapes)
    for layer, path, value in ((0, ("type",), "other"), (0, ("mlp", "kind"), "other"), (0, ("mixer", "heads"), 4), (0, ("mixer", "bias_max"), 10),
                               (0, ("mixer", "q_temp", "every"), 2.5), (1, ("mixer", "rot", "dims"), 16), (1, ("mixer", "rot_dim"), 7),
                               (0, ("mlp", "router", "top"), 11), (0, ("mlp", "router", "groups", "count"), 3), (0, ("mlp", "router", "groups", "keep"), 1)):
        bad = json.loads(json.dumps(c))
        t = bad["layers"][layer]
        for n in path[:-1]:
            t = t[n]
        t[path[-1]] = value
        with pytest.raises(ValueError):
            parse_config(bad, shapes)
    with pytest.raises(ValueError):
        parse_config({**c, "streams": 9}, shapes)
    with pytest.raises(ValueError):
        ExpertsSpec(4, 2, 8, identity=1)                       # weights on the input
    with pytest.raises(ValueError):
        ExpertsSpec(4, 2, 8, shared_ff=8, gated=True)
    with pytest.raises(ValueError):
        AttentionMixer(2, 1, 8, 1.0, 0, 1.0, q_temp=QueryTemperature(0.1, 4))
    with pytest.raises(ValueError):
        AttentionMixer(2, 1, 8, 1.0, 0, 1.0, window=4, rel=DistanceBias(4, 8))
    with pytest.raises(ValueError):
        HybridConfig("x", 8, 8, (LayerSpec(AttentionMixer(2, 1, 8, 1.0, 0, 1.0)),), norm="tanh")
    w["l0.mlp.e1.up"] = w["l0.mlp.e1.up"][:-1].clone()
    d = cases.write(tmp_path, c, w)
    with pytest.raises(ValueError, match="l0.mlp.e1.up"):
        checkpoint_to_segment(CheckpointReader(d), get_config(d))


def test_registry_shapes():
    from blitz_scale_b200.models.config import get_config
    from blitz_scale_b200.models.weights import WeightSegment
    for n in ("vofidra_tiny", "vofidra_odd"):
        cfg = get_config(n)
        seg = WeightSegment(cfg).random_init_(3)
        assert all(torch.isfinite(seg[t].float()).all() for t in seg.names())
        assert not torch.equal(seg["lm_head"][:, :cfg.vocab], seg["embed"].t()) and not seg["lm_head"][:, cfg.vocab:].any()
        e, l = cfg.layer_specs[1].moe, "layers.1."
        assert not seg[l + "down"].view(e.experts, e.ff_pad, -1)[:, e.ff:].any()
        up = e.gate_and_up(seg[l + "up"]).permute(0, 2, 1, 3).reshape(-1, 2, e.ff_pad)
        assert not up[:, :, e.ff:].any() and up[:, :, :e.ff].any(0).all()
        m = cfg.layer_specs[1].mixer
        assert torch.equal(seg[l + "v_up"].view(m.kv_rank, m.heads, m.vdim)[:, -1], seg[l + "uv"].view(m.heads, m.kv_rank, m.vdim)[-1])
    big = get_config("vofidra_13b")
    assert big.kv_bytes_per_token() == 14 * 2 * (2 * 4 * 128 + 256 + 32) and big.attention_work(10 ** 5) == (1, 10 ** 5)


def test_plain_mechanisms():
    """The oracle's own functions on numbers worked out by hand."""
    one = torch.ones(1, dtype=torch.float64)
    assert abs(float(dyt(2 * one, 3 * one, 0.5 * one, 0.25 * one)) - (3 * math.tanh(0.5) + 0.5)) < 1e-12
    xs = torch.tensor([[[1.0]], [[10.0]]])
    assert float(streams_in(xs, torch.tensor([2.0, 3.0]))) == 32.0
    new = streams_out(xs, torch.tensor([[1.0, 2.0], [3.0, 4.0]]), torch.tensor([5.0, 6.0]), torch.tensor([[100.0]]))
    assert new.flatten().tolist() == [1 + 30 + 500, 2 + 40 + 600]
    z = torch.log(torch.tensor([0.4, 0.1, 0.3, 0.2]))
    r = {"top": 2, "groups": {"count": 2, "keep": 1}}
    pairs, margin = route(z, torch.zeros(4), r)
    assert [e for e, _ in pairs] == [0, 1] and abs(float(pairs[0][1]) - 0.8) < 1e-6 and abs(margin - 0.1) < 1e-6
    pairs, _ = route(z, torch.tensor([-0.5, -0.5, 0.0, -0.5]), r)        # a choice score below zero still beats a lost group
    assert [e for e, _ in pairs] == [2, 3] and abs(float(pairs[0][1]) - 0.6) < 1e-6
    assert [bucket(n, 8, 64) for n in (0, 3, 4, 7, 8, 15, 16, 31, 32, 63, 64, 999)] == [0, 3, 4, 4, 5, 5, 6, 6, 7, 7, 7, 7]


@functools.lru_cache(maxsize=None)
def _good(name):
    c = cases.CASES[name]
    toks = tuple(torch.randint(0, c["vocab"], (300,), generator=torch.Generator().manual_seed(2)).tolist())
    return toks, Plain(c, cases.weights(c, 1), torch.float32).run(list(toks))


@pytest.mark.parametrize("flaw", FLAWS)
def test_every_planted_mistake_shows(flaw):
    """The inputs the GPU tests use would reveal each mistake, far above the tolerance of the 16-bit comparison."""
    toks, good = _good("regular")
    c = cases.CASES["regular"]
    bad = Plain(c, cases.weights(c, 1), torch.float32, [flaw]).run(list(toks))
    err = ((good - bad).pow(2).mean(-1) / good.pow(2).mean()).sqrt()
    assert float(err.max()) > 0.25, (flaw, float(err.max()))
    if flaw == "far_key_lost":
        assert float(err[:128].max()) == 0.0
