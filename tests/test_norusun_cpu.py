"""Norusun on the host: configuration, weight mapping, caches, and checks of the plain oracle itself (every planted mistake shows in
the inputs that the GPU tests use)."""
import functools
import json
import math

import pytest
import torch

import norusun_cases as cases
import norusun_plain as plain
from norusun_plain import FLAWS, Plain


def _cfg(c, w=None):
    from blitz_scale_b200.models.norusun import parse_config
    return parse_config(c, {n: tuple(t.shape) for n, t in (w or cases.weights(c)).items()})


@pytest.mark.parametrize("name", sorted(cases.CASES))
def test_checkpoint_round_trip_and_layout(tmp_path, name):
    from blitz_scale_b200.models.config import get_config
    from blitz_scale_b200.models.convert import CheckpointReader, checkpoint_to_segment, convert, verify
    from blitz_scale_b200.models.norusun import from_segment
    c = cases.CASES[name]
    w = cases.weights(c)
    d = cases.write(tmp_path / "ckpt", c, w)
    cfg = get_config(d)
    assert cfg.family == "hybrid" and cfg.vocab == c["vocab"] and cfg.layers == len(c["layers"]) and cfg.recurrent
    assert cfg.streams == c["streams"] and cfg.norm == "rms" and cfg.norm_scalar and cfg.mix_taps == c["canon"]["taps"]
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


def test_caches_and_work():
    from blitz_scale_b200.ops import KVPair, LatentKV
    from blitz_scale_b200.runtime.hybrid_cache import HybridCache
    cfg = _cfg(cases.CASES["regular"])
    cache = HybridCache(cfg, 5, 16, 3, torch.bfloat16, "cpu")
    a, b, c, d, e = cache.runs
    assert a.kv is None and a.state.shape == (3, 5, 40, 40) and a.shift.shape == (3, 200) and a.state.dtype == torch.float32
    assert isinstance(b.kv, LatentKV) and b.kv.pool.shape == (5, 16, 1, 120) and b.state is None and b.shift is None
    assert c.kv.shape == (5, 2, 16, 3, 64) and c.state.shape == (3, 6, 56, 40) and c.hist.shape == (3, 2, 240 + 2 * 3 * 56)
    assert all(r.mix_hist.shape == (3, 3, 200) for r in cache.runs) and d.state.shape == (3, 2, 64, 64) and e.kv.shape[3] == 4
    assert cache.bytes() == 5 * 16 * cfg.kv_bytes_per_token() + 3 * cfg.state_bytes_per_sequence()
    assert cfg.attention_work(5000) == (1, 50) and cfg.attention_work(20) == (1, 20)
    other = HybridCache(_cfg(cases.CASES["values"]), 2, 16, 1, torch.float32, "cpu")
    assert isinstance(other.runs[0].kv, KVPair) and other.runs[0].mix_hist.shape == (1, 0, 136)


def test_recurrent_by_its_convolution_alone():
    """A model of attention layers whose only state is the convolution's history still needs slots; with one tap it does not."""
    for taps, want in ((2, True), (1, False)):
        assert _cfg(cases.config([cases.latent()], [None], taps=taps)).recurrent == want


def test_refusals(tmp_path):
    from blitz_scale_b200.models.config import get_config
    from blitz_scale_b200.models.convert import CheckpointReader, checkpoint_to_segment
    from blitz_scale_b200.models.hybrid_config import (AttentionMixer, ClampedUnit, ExpertsSpec, GLAMixer, HybridConfig, LayerSpec, SSDMixer,
                                                       WKVMixer)
    c = cases.config([cases.wkv(), cases.latent(), cases.parallel()], [None, cases.dense(), cases.dense()])
    w = cases.weights(c)
    _cfg(c, w)
    for layer, path, value in ((0, ("type",), "other"), (1, ("mlp", "kind"), "other"), (1, ("mlp", "limit"), 0.0), (1, ("mixer", "mask", "size"), 2.5),
                               (1, ("mixer", "rot", "dims"), 8), (1, ("mixer", "rot_dim"), 7), (2, ("mixer", "left", "heads"), 4),
                               (2, ("mixer", "left", "rot", "dims"), 66), (2, ("mixer", "left", "mask", "size"), 0), (2, ("mixer", "right", "groups"), 4),
                               (2, ("mixer", "right", "norm_groups"), 7), (2, ("mixer", "right", "conv"), 17)):
        bad = json.loads(json.dumps(c))
        t = bad["layers"][layer]
        for n in path[:-1]:
            t = t[n]
        t[path[-1]] = value
        with pytest.raises(ValueError):
            _cfg(bad, w)
    for key, value in (("streams", 9), ("canon", {"taps": 17})):
        with pytest.raises(ValueError):
            _cfg({**c, key: value}, w)
    plain_layer = LayerSpec(GLAMixer(1, 8, 8, 1.0, 4))
    for bad in (dict(layer_specs=(plain_layer,), norm_scalar=True), dict(layer_specs=(plain_layer,), mix_taps=2),
                dict(layer_specs=(LayerSpec(WKVMixer(8, 1, 8, 4)),)), dict(layer_specs=(LayerSpec(WKVMixer(16, 1, 8, 4)),), streams=2),
                dict(layer_specs=(LayerSpec(SSDMixer(1, 8, 8, 1, 2, 1)),), streams=2),
                dict(layer_specs=(LayerSpec(plain_layer.mixer, moe=ExpertsSpec(2, 1, 8)),), streams=2)):
        with pytest.raises(ValueError):
            HybridConfig("x", 8, 8, **bad)
    for bad in (dict(whole_norm=True, bias=True), dict(chunked=True), dict(chunked=True, window=4, keep_first=2), dict(sigmoid=True, sink=True)):
        with pytest.raises(ValueError):
            AttentionMixer(2, 1, 8, 1.0, 0, 1.0, **bad)
    with pytest.raises(ValueError):
        LayerSpec(plain_layer.mixer, unit=ClampedUnit(1.0))
    w["l2.mix.right.in"] = w["l2.mix.right.in"][:-1].clone()
    d = cases.write(tmp_path, c, w)
    with pytest.raises(ValueError, match="l2.mix.right.in"):
        checkpoint_to_segment(CheckpointReader(d), get_config(d))


def test_registry_shapes():
    from blitz_scale_b200.models.config import build_layout, get_config
    from blitz_scale_b200.models.weights import WeightSegment
    for n in ("norusun_tiny", "norusun_odd"):
        cfg = get_config(n)
        seg = WeightSegment(cfg).random_init_(3)
        assert all(torch.isfinite(seg[t].float()).all() for t in seg.names())
        assert not torch.equal(seg["lm_head"][:, :cfg.vocab], seg["embed"].t()) and not seg["lm_head"][:, cfg.vocab:].any()
        for l, s in enumerate(cfg.layer_specs):
            if s.mixer.kind == "wkv":
                assert not seg[f"layers.{l}.w1"][:, s.mixer.rank:].any()
            if s.unit:
                b = seg[f"layers.{l}.gate_up_b"].view(2, -1)
                assert not b[:, s.ff_after:].any() and b[:, :s.ff_after].any(1).all()
    big = get_config("norusun_8b")
    assert big.kv_bytes_per_token() == 8 * 2 * (2 * 544 + 2 * 8 * 128) and big.attention_work(10 ** 5) == (1, 2048)
    assert 14e9 < build_layout(big).total_bytes < 16e9


def test_plain_mechanisms():
    """The oracle's own functions on numbers worked out by hand."""
    f = lambda *v: torch.tensor(v, dtype=torch.float64)
    x = f(1, 2, 3, 4).view(4, 1)
    assert plain.causal_conv(x, f(10, 1).view(1, 2)).flatten().tolist() == [1, 12, 23, 34]
    xs = torch.tensor([[[1.0]], [[10.0]]])
    assert float(plain.streams_in(xs, torch.tensor([2.0, 3.0]))) == 32.0
    new = plain.streams_out(xs, torch.tensor([[1.0, 2.0], [3.0, 4.0]]), torch.tensor([5.0, 6.0]), torch.tensor([[100.0]]))
    assert new.flatten().tolist() == [1 + 30 + 500, 2 + 40 + 600]
    # a head of one channel: o_0 = u k v r, S = k v; o_1 = (S + u k v) r, S = w S + k v
    r, k, v, w = f(1, 2, 1).view(3, 1, 1), f(3, 1, 1).view(3, 1, 1), f(5, 7, 1).view(3, 1, 1), f(0.9, 0.5, 0.1).view(3, 1, 1)
    assert plain.wkv_recurrence(r, k, v, w, f(2).view(1, 1)).flatten().tolist() == [30, 2 * (15 + 14), 0.5 * 15 + 7 + 2]
    # a state of one row: S = e^(-rate dt) S + dt B x, y = C S + D x
    y = plain.ssd_recurrence(f(3, 4).view(2, 1, 1), f(1, 2).view(2, 1, 1), f(1, 10).view(2, 1, 1), f(0.5, 1).view(2, 1), f(math.log(2)), f(100))
    assert torch.allclose(y.flatten(), f(1.5 + 300, 10 * (0.75 + 8) + 400))
    one = torch.ones(6, 1, dtype=torch.float64)
    assert torch.allclose(plain.sigmoid_attention(one, 0 * one, one, 1.0, 4, 0.0).flatten(), f(0.5, 1, 1.5, 2, 0.5, 1))
    assert torch.allclose(plain.sink_attention(one, 0 * one, one, 1.0, 3, f(0)).flatten(), f(1 / 2, 2 / 3, 3 / 4, 3 / 4, 3 / 4, 3 / 4))
    assert torch.allclose(plain.rms(f(3, 4), 0.0), f(3, 4) / math.sqrt(12.5))


@functools.lru_cache(maxsize=None)
def _good():
    c = cases.CASES["regular"]
    toks = tuple(torch.randint(0, c["vocab"], (160,), generator=torch.Generator().manual_seed(2)).tolist())
    return toks, Plain(c, cases.weights(c), torch.float32).run(list(toks))


@pytest.mark.parametrize("flaw", FLAWS)
def test_every_planted_mistake_shows(flaw):
    """The inputs the GPU tests use would reveal each mistake, far above the tolerance of the 16-bit comparison."""
    toks, good = _good()
    c = cases.CASES["regular"]
    bad = Plain(c, cases.weights(c), torch.float32, [flaw]).run(list(toks))
    err = ((good - bad).pow(2).mean(-1) / good.pow(2).mean()).sqrt()
    assert float(err.max()) > 0.2, (flaw, float(err.max()))
    if flaw == "no_window":
        assert float(err[:37].max()) == 0.0
    if flaw == "no_chunks":
        assert float(err[:16].max()) == 0.0
