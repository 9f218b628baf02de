"""Hybrid models on the host: configuration, weight mapping, slots and ragged steps of the native batch, and checks of
the plain oracle itself (every planted mistake shows at the places it concerns)."""
import json

import numpy as np
import pytest
import torch

import fafudra_cases as cases
from fafudra_plain import FLAWS, Plain, rotate_pairs, visible
from blitz_scale_b200.runtime import core


@pytest.mark.parametrize("name", sorted(cases.CASES))
def test_checkpoint_round_trip_and_layout(tmp_path, name):
    from blitz_scale_b200.models.config import get_config
    from blitz_scale_b200.models.convert import CheckpointReader, checkpoint_to_segment, convert, verify
    from blitz_scale_b200.models.fafudra import from_segment
    c = cases.CASES[name]
    w = cases.weights(c)
    d = cases.write(tmp_path / "ckpt", c, w)
    cfg = get_config(d)
    assert cfg.family == "hybrid" and cfg.vocab == c["vocab"] and cfg.layers == len(c["layers"])
    seg = checkpoint_to_segment(CheckpointReader(d), cfg)
    back = from_segment(seg)
    assert set(back) == set(w) and all(torch.equal(back[n], w[n]) for n in w)
    names = [n for n, _, _ in seg.layout.units]
    assert names == ["embed"] + [f"layer.{i}" for i in range(cfg.layers)] + ["head"]
    # units tile the segment; padding of the fused projections is zero
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


def test_order_of_layer_runs():
    from blitz_scale_b200.models.fafudra import parse_config
    c = cases.config([cases.gla(), cases.rglru(), cases.attention(), cases.gla()], loop=(1, 3, 3))
    runs = parse_config(c).runs()
    assert [r.layer for r in runs] == [0, 1, 2, 1, 2, 1, 2, 3]
    assert [(r.step, r.add_embed) for r in runs] == [(-1, False), (0, False), (-1, False), (1, True), (-1, False), (2, True),
                                                     (-1, False), (-1, False)]
    assert [i for i, _ in Plain(c, {}).order()] == [r.layer for r in runs]
    assert [r.layer for r in parse_config(cases.config([cases.gla()] * 2)).runs()] == [0, 1]
    with pytest.raises(ValueError):
        parse_config(cases.config([cases.gla()] * 2, loop=(1, 3, 2)))


def test_refusals(tmp_path):
    from blitz_scale_b200.models.config import get_config
    from blitz_scale_b200.models.fafudra import parse_config
    from blitz_scale_b200.models.weights import WeightSegment
    c = cases.config([cases.attention()])
    bad = json.loads(json.dumps(c))
    bad["layers"][0]["mixer"]["vdim"] = 32
    with pytest.raises(ValueError):
        parse_config(bad)
    with pytest.raises(ValueError):
        WeightSegment(parse_config(c), tp=2)
    d = cases.write(tmp_path, c, cases.weights(c))
    (tmp_path / "config.json").write_text(json.dumps({**c, "architecture": "Other"}))
    with pytest.raises(KeyError):
        get_config(d)
    with pytest.raises(KeyError):
        get_config(str(tmp_path / "nothing"))


def test_registry_shapes_and_sizes():
    from blitz_scale_b200.models.config import get_config
    from blitz_scale_b200.models.weights import WeightSegment
    for n in ("fafudra_tiny", "fafudra_odd"):
        cfg = get_config(n)
        seg = WeightSegment(cfg).random_init_(3)
        assert torch.isfinite(seg["embed"].float()).all()
        assert torch.equal(seg["lm_head"][:, :cfg.vocab], seg["embed"].t())
        assert not seg["lm_head"][:, cfg.vocab:].any()
    big = get_config("fafudra_8b")
    att = sum(m.kind == "attention" for m in big.run_mixers())
    assert big.kv_bytes_per_token() == att * 2 * 8 * 128 * 2 and big.recurrent
    assert big.attention_work(100) == (8, 100) and big.attention_work(10 ** 6) == (8, 2052)


def test_state_slots_follow_the_requests():
    pool, slots = core.PagePool(32, 16), core.SlotPool(3)
    a, b = core.Batch(1, pool, slots), core.Batch(2, pool, slots)
    assert a.add_prompts([core.SeqSpec(0, [1, 2], 4), core.SeqSpec(1, [3], 4)])
    assert not b.add_prompts([core.SeqSpec(2, [1], 4), core.SeqSpec(3, [1], 4)])      # all or nothing
    assert b.size == 0 and pool.used_pages == 2 and slots.free_slots == 1
    assert b.add_prompts([core.SeqSpec(2, [1], 4)])
    held = [s.slot for s in a.seqs]
    assert len(set(held + [s.slot for s in b.seqs])) == 3
    a.extend(b)
    a.filter([0, 2])
    assert slots.free_slots == 1 and slots.allocate() == held[1]
    slots.release(held[1])
    with pytest.raises(Exception):
        slots.release(held[1])
    with pytest.raises(Exception):
        a.extend(core.Batch(3, pool))                       # a batch without slots
    a.clear()
    assert slots.free_slots == 3 and pool.used_pages == 0


def test_ragged_step_staging():
    ps = 4
    pool, slots = core.PagePool(16, ps), core.SlotPool(4)
    b = core.Batch(1, pool, slots)
    assert b.add_prompts([core.SeqSpec(0, [10, 11, 12], 1), core.SeqSpec(1, [20], 1), core.SeqSpec(2, [30, 31, 32, 33, 34, 35], 1)], False)
    assert [len(s.pages) for s in b.seqs] == [1, 1, 2]      # no page for a token that may never come
    L = core.MetaLayout.make(16, 4, 16)
    h = np.full(L.total, -7, dtype=np.int32)
    T, P, rows, singles, order, q, kv = b.fill_step(h, L, [2, 1, 5], 8)
    assert (T, rows, singles, order, q, kv) == (8, 3, 1, [1, 0, 2], [1, 2, 5], [1, 2, 5])
    assert list(h[L.ids:L.ids + 8]) == [20, 10, 11, 30, 31, 32, 33, 34] and list(h[L.pos:L.pos + 8]) == [0, 0, 1, 0, 1, 2, 3, 4]
    assert list(h[L.tok_indptr:L.tok_indptr + 4]) == [0, 1, 3, 8] and list(h[L.page_indptr:L.page_indptr + 4]) == [0, 1, 2, 4]
    assert list(h[L.seq_slot:L.seq_slot + 3]) == [b.seqs[1].slot, b.seqs[0].slot, b.seqs[2].slot]
    b.advance([2, 1, 5])
    assert b.cached_lens() == [2, 1, 5]
    # next step: one request sits out, another gets more tokens, across a page border
    assert b.extend_prompt(0, [13, 14, 15])
    T, P, rows, singles, order, q, kv = b.fill_step(h, L, [4, 0, 1], 8)
    assert (T, rows, singles, order, q, kv) == (5, 2, 1, [2, 0], [1, 4], [6, 6])
    pages = list(b.seqs[0].pages)
    assert list(h[L.ids:L.ids + 5]) == [35, 12, 13, 14, 15] and list(h[L.pos:L.pos + 5]) == [5, 2, 3, 4, 5]
    assert list(h[L.slot + 1:L.slot + 5]) == [pages[0] * ps + 2, pages[0] * ps + 3, pages[1] * ps, pages[1] * ps + 1]
    assert list(h[L.last_page_len:L.last_page_len + 2]) == [2, 2]
    b.advance([4, 0, 1])
    with pytest.raises(Exception):
        b.fill_step(h, L, [1, 0, 0], 8)                     # nothing left of request 0
    # single tokens only: padded to the graph's batch size
    assert b.extend_prompt(1, [21]) and b.extend_prompt(0, [16])
    T, P, rows, singles, order, q, kv = b.fill_step(h, L, [1, 1, 0], 4)
    assert (T, rows, singles, order, kv) == (2, 2, 2, [0, 1], [7, 2])
    assert list(h[L.seq_slot + 2:L.seq_slot + 4]) == [-1, -1] and list(h[L.slot + 2:L.slot + 4]) == [-1, -1]
    # a pool that is too small leaves the request as it was
    assert not b.extend_prompt(0, list(range(100))) and len(b.seqs[0].spec.prompt) == 7
    b.clear()
    assert pool.used_pages == 0


def test_oracle_pieces():
    see = visible(8, 3, 2)
    assert see[6].tolist() == [True, True, False, False, True, True, True, False]
    x = torch.randn(5, 2, 6, dtype=torch.float64)
    r = rotate_pairs(x, torch.arange(5), 4, 100.0)
    assert torch.equal(r[..., 4:], x[..., 4:]) and torch.equal(r[0], x[0])
    n = lambda t, i: t[..., i] ** 2 + t[..., i + 1] ** 2
    assert torch.allclose(n(r, 0), n(x, 0)) and torch.allclose(n(r, 2), n(x, 2))
    # angle of pair 1 at position 3
    a = 3 * 100.0 ** (-2 / 4)
    assert abs(float(r[3, 0, 2] - (x[3, 0, 2] * np.cos(a) - x[3, 0, 3] * np.sin(a)))) < 1e-12


@pytest.mark.parametrize("flaw", FLAWS)
def test_every_planted_mistake_shows(flaw):
    """The inputs the GPU tests use would reveal each mistake: far above the tolerance of the fp32 comparison, and (but for
    a rounded state) above that of the 16-bit one."""
    c = cases.CASES["regular"]
    w = cases.weights(c, 1)
    toks = torch.randint(0, c["vocab"], (90,), generator=torch.Generator().manual_seed(2)).tolist()
    good, bad = Plain(c, w, torch.float32).run(toks), Plain(c, w, torch.float32, [flaw]).run(toks)
    err = ((good - bad).pow(2).mean(-1) / good.pow(2).mean(-1)).sqrt()
    assert float(err.max()) > (1e-3 if flaw == "state_16bit" else 5e-2), (flaw, float(err.max()))
    if flaw in ("window_long", "window_short", "no_first", "first_short"):
        assert float(err[:20].max()) == 0.0        # not before the window has moved off the start
