"""Norusun on the GPU against the plain oracle: whole prompts, portions, decoding, mixed batches, reuse of pages and slots,
greedy generation through the engine and through the worker, trace replay."""
import functools
import json
import os
import subprocess
import sys

import pytest
import torch

import norusun_cases as cases
from hybrid_feed import DTYPES, TOL, Feed, check
from norusun_plain import Plain

pytestmark = pytest.mark.gpu

PAGE = 16


@functools.lru_cache(maxsize=None)
def _weights(name):
    return cases.weights(cases.CASES[name])


def _tokens(name, n, seed):
    return tuple(torch.randint(0, cases.CASES[name]["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist())


@functools.lru_cache(maxsize=None)
def _want(name, n, seed):
    return Plain(cases.CASES[name], _weights(name), torch.float32).run(list(_tokens(name, n, seed)))


@functools.lru_cache(maxsize=None)
def _rounding(name, n, seed):
    """How much rounding to 16 bits between the sublayers changes the logits of every position (relative rms)."""
    want = _want(name, n, seed)
    got = Plain(cases.CASES[name], _weights(name), torch.float32, rounded=torch.bfloat16).run(list(_tokens(name, n, seed)))
    return (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean().sqrt()


def _check(got, name, n, seed, dtype, what=""):
    """In 16 bits a position where rounding alone changes much has room for more."""
    want = _want(name, n, seed)
    if dtype == torch.bfloat16:
        room = (4 * _rounding(name, n, seed) / TOL[dtype]).clamp(min=1.0)[:, None]
        got = want + (got - want) / room
    check(got, want, dtype, (name, n, what))


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    root = tmp_path_factory.mktemp("ckpt")
    return {n: cases.write(root / n, c, _weights(n)) for n, c in cases.CASES.items()}


def _engine(folder, dtype=torch.bfloat16, **kw):
    from blitz_scale_b200.runtime.engine import Engine
    torch.cuda.set_device(0)
    args = dict(num_pages=96, page_size=PAGE, max_batch=8, max_batch_tokens=1024)
    eng = Engine(folder, dtype=dtype, ready=False, **{**args, **kw})
    eng.load_checkpoint(folder)
    return eng


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(cases.CASES))
def test_whole_prompt(folders, name, dtype):
    f = Feed(_engine(folders[name], dtype))
    for r, n in enumerate((1, 2, 7, 150, 400)):
        f.step({r: _tokens(name, n, r)})
        _check(f.logits(r), name, n, r, dtype)
        f.end(r)
    assert f.eng.pool.used_pages == 0 and (f.eng.slots is None or f.eng.slots.free_slots == f.eng.slots.total_slots)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(cases.CASES))
def test_portions_and_single_tokens(folders, name, dtype):
    """The same prompt in portions of many sizes, cut inside pages and key blocks, and its tail token by token."""
    n = 150
    toks = _tokens(name, n, 3)
    f = Feed(_engine(folders[name], dtype))
    for r, sizes in enumerate(([2] * 75, [1, 2, 3, 64, 5, 2, 33, 40], [100] + [1] * 50, [65, 63, 2, 1, 17, 1, 1])):
        at = 0
        for s in sizes:
            f.step({r: toks[at:at + s]})
            at += s
        assert at == n
        _check(f.logits(r), name, n, 3, dtype, sizes[:4])
        f.end(r)


@pytest.mark.parametrize("dtype", DTYPES)
def test_token_by_token_from_the_first(folders, dtype):
    for name, n in (("regular", 130), ("odd", 60), ("wide", 70)):
        f = Feed(_engine(folders[name], dtype))
        for t in _tokens(name, n, 4):
            f.step({0: (t,)})
        _check(f.logits(0), name, n, 4, dtype)


@pytest.mark.parametrize("graphs", [True, False])
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["regular", "odd", "values", "wide", "ones"])
def test_mixed_batch_with_reused_pages_and_slots(folders, name, dtype, graphs):
    """Unequal requests side by side: portions of some beside single tokens of others, one sitting out, and later ones on
    the pages and slots of those that have ended; pools that hold no more than the live ones need."""
    f = Feed(_engine(folders[name], dtype, num_pages=20, state_slots=4, use_graphs=graphs))
    plan = {0: 130, 1: 9, 2: 70, 3: 33, 4: 150, 5: 1, 6: 40}
    at = {r: 0 for r in plan}

    def step(**parts):
        todo = {}
        for k, n in parts.items():
            r = int(k[1:])
            todo[r] = _tokens(name, plan[r], 10 + r)[at[r]:at[r] + n]
            assert len(todo[r]) == n
            at[r] += n
        f.step(todo)
        for r in todo:
            if at[r] == plan[r]:
                _check(f.logits(r), name, plan[r], 10 + r, dtype, r)
                f.end(r)
    step(r0=60, r1=1)
    step(r0=1, r1=1, r2=45)
    step(r1=1, r2=1, r0=2)
    step(r0=1, r1=1, r2=1, r3=2)
    step(r3=30, r1=5, r2=3)             # request 1 ends; 0 sits out
    step(r0=66, r2=20, r3=1)            # 0, 2 and 3 end
    step(r4=31, r5=1)                   # fresh requests on their pages
    step(r4=1, r6=1)
    step(r4=100, r6=38)
    for _ in range(18):
        step(r4=1)
    step(r6=1)
    assert f.eng.pool.used_pages == 0 and (f.eng.slots is None or f.eng.slots.free_slots == f.eng.slots.total_slots) and all(at[r] == plan[r] for r in plan)


def test_expanded_keys_some_heads_at_a_time(folders):
    """Prompts whose expanded keys and values would be large: a few heads per pass over them, the last one with fewer."""
    f = Feed(_engine(folders["regular"], torch.bfloat16))
    f.eng.runner.EXPANDED_BYTES = 2 * 160 * 160 * 2
    toks, other = _tokens("regular", 150, 3), _tokens("regular", 7, 2)
    f.step({0: toks[:70], 1: other[:6]})
    f.step({0: toks[70:], 1: other[6:]})
    _check(f.logits(0), "regular", 150, 3, torch.bfloat16)
    _check(f.logits(1), "regular", 7, 2, torch.bfloat16)


def test_steps_beyond_the_token_budget_are_cut(folders):
    f = Feed(_engine(folders["regular"], torch.float32, max_batch_tokens=64))
    f.step({0: _tokens("regular", 150, 3), 1: _tokens("regular", 90, 5)})
    _check(f.logits(0), "regular", 150, 3, torch.float32)
    _check(f.logits(1), "regular", 90, 5, torch.float32)


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(folders, dtype):
    """Many pages of decoded tokens, over the lengths at which keys are split among blocks."""
    name, n = "regular", 620
    f = Feed(_engine(folders[name], dtype))
    toks = _tokens(name, n, 6)
    f.step({0: toks[:20]})
    for t in toks[20:]:
        f.step({0: (t,)})
    _check(f.logits(0), name, n, 6, dtype)


@pytest.mark.parametrize("budget", [1024, 48])
@pytest.mark.parametrize("name", ["regular", "odd", "ones", "wide"])
def test_greedy_generation(folders, name, budget):
    """Engine.prefill (one pass or several) and Engine.decode of a batch, in fp32: the oracle's tokens."""
    from blitz_scale_b200 import ops
    from blitz_scale_b200.runtime import core
    plain = Plain(cases.CASES[name], _weights(name), torch.float32)
    eng = _engine(folders[name], torch.float32, max_batch_tokens=budget)
    lens, new = (50, 3, 17), 8
    for round_ in range(2):             # the second round runs on freed pages
        prompts = [list(_tokens(name, n, 20 + 5 * round_ + i)) for i, n in enumerate(lens)]
        b = eng.new_batch(round_, [core.SeqSpec(i, p, new) for i, p in enumerate(prompts)])
        out = [[t] for t in eng.prefill(b)]
        for _ in range(new - 1):
            for o, t in zip(out, eng.decode(b)):
                o.append(t)
        ops.check_status()
        assert out == [plain.greedy(p, new) for p in prompts]
        b.clear()
    assert eng.pool.used_pages == 0


def test_worker_serves_a_checkpoint_folder(folders):
    from blitz_scale_b200 import ops
    from blitz_scale_b200.pb.schema import pb
    from blitz_scale_b200.runtime import core
    from blitz_scale_b200.worker.gpu_backend import GpuBackend
    torch.cuda.set_device(0)
    w = GpuBackend(0, 1, folders["regular"], num_pages=64, page_size=PAGE, max_batch=4, max_batch_tokens=256)
    batch = pb.Batch(id=1, size=2, max_tokens=128)
    for i in range(2):
        r = batch.requests.add()
        r.id = i
        r.input_tokens.extend(_tokens("regular", 12 + 9 * i, 60 + i))
        r.stopping_parameters.max_new_tokens = 5
        r.stopping_parameters.ignore_eos_token = True
    gens, cb, _ = w.prefill(batch, 0, None, [])
    got = list(zip(*core.parse_generations(gens)))
    while cb is not None:
        gens, cb = w.decode([cb], [pb.Tokens()])
        got += list(zip(*core.parse_generations(gens)))
    ops.check_status()
    per = [[t[1] for t in got if t[0] == i] for i in range(2)]
    assert [len(p) for p in per] == [5, 5] and w.engine.pool.used_pages == 0
    # the same engine, directly, with a sampled row beside the greedy one
    b = w.engine.new_batch(9, [core.SeqSpec(i, list(_tokens("regular", 12 + 9 * i, 60 + i)), 5) for i in range(2)])
    direct = [[t] for t in w.engine.prefill(b)]
    for _ in range(4):
        for o, t in zip(direct, w.engine.decode(b)):
            o.append(t)
    assert per == direct
    b.clear()
    specs = [core.SeqSpec(i, list(_tokens("regular", 12 + 9 * i, 60 + i)), 5) for i in range(2)]
    specs[1].do_sample, specs[1].temperature, specs[1].seed = True, 3.0, 7
    drawn = []
    for k in range(2):
        b = w.engine.new_batch(10 + k, specs)
        drawn.append([[t] for t in w.engine.prefill(b)])
        for _ in range(4):
            for o, t in zip(drawn[-1], w.engine.decode(b)):
                o.append(t)
        b.clear()
    assert drawn[0] == drawn[1] and drawn[0][0] == direct[0] and drawn[0][1] != direct[1]
    w.close()


def test_trace_replay_program(folders, tmp_path):
    import numpy as np
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    a, b = list(_tokens("regular", 70, 70)), list(_tokens("regular", 5, 71))
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:66], "want": [65, 0]}, {"id": "b", "tokens": b[:2], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": b[2:], "want": [2]}, {"id": "a", "tokens": a[66:67], "want": [0]}], "end": ["b"]},
             {"step": 3, "entries": [{"id": "c", "tokens": b, "want": [4]}, {"id": "a", "tokens": a[67:], "want": [2]}], "end": ["a", "c"]}]
    p = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", folders["regular"], "--dtype", "float32",
                        "--out", str(tmp_path), "--max-tokens", "192"], input="\n".join(map(json.dumps, steps)) + "\n",
                       capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [x for x in p.stdout.split("\n") if x.startswith("done")] == ["done 0", "done 2", "done 3"]
    ea, eb = _want("regular", 70, 70), _want("regular", 5, 71)
    for n, want in ((0, [ea[65], ea[0]]), (2, [eb[4], ea[66]]), (3, [eb[4], ea[69]])):
        got = torch.from_numpy(np.fromfile(tmp_path / f"{n}.f32", dtype="<f4")).view(len(want), -1)
        check(got, torch.stack(want), torch.float32, n)
