"""Saninex through the engine against the plain implementation: whole prompts, portions, decoding, batches, pages and slots
used again, greedy generation through the scheduler, sampling, the command line."""
import json
import os
import subprocess
import sys
from pathlib import Path

import pytest
import torch

import saninex_cases as sc
import saninex_oracle as oracle

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parents[1]
LIMIT = {"float32": 5e-5, "bfloat16": 6e-2}


@pytest.fixture(scope="module")
def folder(tmp_path_factory):
    d = tmp_path_factory.mktemp("saninex")
    paths = {}

    def get(name):
        if name not in paths:
            paths[name] = sc.write_checkpoint(d / name, sc.CASES[name], sc.tensors(name))
        return paths[name]

    return get


_want: dict = {}


def _expected(name, ids):
    key = (name, tuple(ids))
    if key not in _want:
        _want[key] = oracle.forward(sc.CASES[name], sc.tensors(name), ids)
    return _want[key]


def _engine(path, dtype, **kw):
    from crosspool_b200.deployment import build_loopback
    from crosspool_b200.engine.atn_engine import EngineConfig

    kw = {**dict(max_batch=4, prefill_chunk=512, max_seq_len=512, page_size=64, max_prefill_seqs=4), **kw}
    return build_loopback([("m", path, 0)], EngineConfig(dtype=dtype, **kw)).instances[0].engine


def _feed(eng, s, ids, sizes):
    """Logits at every token of ``ids`` fed in portions of ``sizes`` (the last size repeats)."""
    out, at, i = [], 0, 0
    while at < len(ids):
        n = min(sizes[min(i, len(sizes) - 1)], len(ids) - at)
        out.append(eng.run_given([(s, ids[at:at + n])], [list(range(n))]))
        at, i = at + n, i + 1
    return torch.cat(out)


@pytest.mark.parametrize("page", [16, 64])
@pytest.mark.parametrize("dtype", list(LIMIT))
@pytest.mark.parametrize("name", list(sc.CASES))
def test_prompt_portions_and_token_by_token(folder, name, dtype, page):
    """The same 150 tokens whole, in portions of several sizes and one by one through captured decode graphs; pages and the
    state slot are used again each time and hold another sequence's leftovers."""
    eng = _engine(folder(name), dtype, num_pages=192 // page, page_size=page)
    eng.warmup()
    c = sc.CASES[name]
    ids, other = sc.prompt(c, 150, 1), sc.prompt(c, 180, 2)
    want = _expected(name, ids)
    for sizes in ([150], [64, 1], [2], [17, 3, 40, 2, 16], [1], [100, 33, 1], [63, 65, 1], [1, 2, 3, 4, 5, 6]):
        s = eng.open_sequence()
        _feed(eng, s, other, [180])
        eng.close_sequence(s)
        s = eng.open_sequence()
        e = sc.error(_feed(eng, s, ids, sizes), want)
        eng.close_sequence(s)
        assert e.max().item() < LIMIT[dtype], (sizes, e.argmax().item(), e.max().item())
    assert eng.kv.allocator.free_pages == 192 // page and eng.kv.slots.free_slots == 4


@pytest.mark.parametrize("dtype", list(LIMIT))
@pytest.mark.parametrize("name", ["mixed", "odd", "wide"])
def test_batches_of_unequal_requests_equal_each_alone(folder, name, dtype):
    """Portions of some requests beside single tokens of others, requests that pause, end, and hand pages and slots on."""
    c = sc.CASES[name]
    req = {k: sc.prompt(c, n, 10 + i) for i, (k, n) in enumerate({"a": 1, "b": 120, "c": 37, "d": 64, "e": 90, "f": 2}.items())}
    eng = _engine(folder(name), dtype, num_pages=6)
    eng.warmup()
    plan = [{"a": 1, "b": 40}, {"b": 1, "c": 20, "d": 63}, {"b": 2, "d": 1}, {"b": 1, "c": 1}, {"c": 16, "e": 30, "b": 17},
            {"b": 1, "e": 1}, {"f": 2, "e": 2}, {"b": 58, "e": 57}]
    at, live, got = {k: 0 for k in req}, {}, {k: [] for k in req}
    for step in plan:
        portions, ids = [], list(step)
        for k in ids:
            if k not in live:
                live[k] = eng.open_sequence()
            portions.append((live[k], req[k][at[k]:at[k] + step[k]]))
            at[k] += step[k]
        out = eng.run_given(portions, [list(range(step[k])) for k in ids])
        for k, o in zip(ids, out.split([step[k] for k in ids])):
            got[k].append(o)
        for k in ids:
            if at[k] == len(req[k]):
                eng.close_sequence(live.pop(k))
    assert not live
    for k in req:
        e = sc.error(torch.cat(got[k]), _expected(name, req[k]))
        assert e.max().item() < LIMIT[dtype], (k, e.argmax().item(), e.max().item())


@pytest.mark.parametrize("dtype", list(LIMIT))
def test_a_far_key_is_found_from_every_schedule(tmp_path, dtype):
    """Every query of the first layer looks for a marked token among hundreds: losing it, or its page, changes the logits."""
    c, t = sc.far_key_model()
    path = sc.write_checkpoint(tmp_path / "far", c, t)
    ids = [i for i in sc.prompt(c, 420, 6) if i != 7][:400]
    eng = _engine(path, dtype)
    for place in (33, 0, 63, 64):                        # somewhere, the first token, both sides of a page's border
        ids_p = ids[:place] + [7] + ids[place + 1:]
        want = oracle.forward(c, t, ids_p)
        without = oracle.forward(c, t, [i if j != place else 8 for j, i in enumerate(ids_p)])
        assert sc.error(without[380:], want[380:]).min().item() > 2 * LIMIT["bfloat16"]
        for sizes in ([400], [34, 200, 1], [16, 33, 2, 64], [370, 1]) if place == 33 else ([64, 300, 1],):
            s = eng.open_sequence()
            e = sc.error(_feed(eng, s, ids_p, sizes), want)
            eng.close_sequence(s)
            assert e.max().item() < LIMIT[dtype], (place, sizes, e.argmax().item(), e.max().item())


def test_long_decoding_in_32_bit(folder):
    c = sc.CASES["recurrent"]
    ids = sc.prompt(c, 500, 4)
    eng = _engine(folder("recurrent"), "float32")
    eng.warmup()
    s = eng.open_sequence()
    assert sc.error(_feed(eng, s, ids, [3, 1]), _expected("recurrent", ids)).max().item() < LIMIT["float32"]


def _greedy(name, prompt, n):
    c, t, ids = sc.CASES[name], sc.tensors(name), list(prompt)
    for _ in range(n):
        ids.append(int(oracle.forward(c, t, ids)[-1].argmax()))
    return ids[len(prompt):]


@pytest.mark.parametrize("mixed", [False, True])
@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_greedy_generation_through_the_scheduler(folder, name, mixed):
    """Chunked prefill, more requests than decode rows, requests that arrive while others decode."""
    c = sc.CASES[name]
    prompts = [sc.prompt(c, n, 20 + n) for n in (1, 40, 23, 70, 2, 33)]
    eng = _engine(folder(name), "float32", prefill_chunk=32, max_batch=3, mixed_batches=mixed)
    eng.warmup()
    seqs = [eng.add_request(p, 7) for p in prompts[:3]]
    for _ in range(4):
        eng.step()
    seqs += [eng.add_request(p, 7) for p in prompts[3:]]
    while eng.has_work:
        eng.step()
    for s, p in zip(seqs, prompts):
        assert s.generated == _greedy(name, p, 7)
    assert not eng.kv.tables and eng.kv.slots.free_slots == 3


def test_a_retracted_sequence_is_recomputed_with_its_states(folder):
    """Too few pages for everyone: the engine takes one sequence's pages and slot away and rebuilds both later."""
    c = sc.CASES["mixed"]
    prompts = [sc.prompt(c, n, 40 + n) for n in (30, 29, 31)]
    eng = _engine(folder("mixed"), "float32", num_pages=8, page_size=16)
    out = eng.generate(prompts, 24)
    assert out == [_greedy("mixed", p, 24) for p in prompts]
    assert eng.kv.allocator.free_pages == 8 and eng.kv.slots.free_slots == 4


def test_sampling_is_seeded_and_greedy_at_temperature_zero(folder):
    eng = _engine(folder("mixed"), "bfloat16", sampling=True)
    p = sc.prompt(sc.CASES["mixed"], 12, 3)

    def run(**kw):
        s = eng.add_request(p, 12, **kw)
        while eng.has_work:
            eng.step()
        return s.generated

    assert run(temperature=60.0, seed=1) == run(temperature=60.0, seed=1) != run(temperature=60.0, seed=2)
    assert run() == run(temperature=0.0, seed=9)


def test_command_lines(folder):
    """``bin/trace_run`` and ``xpool generate`` as processes of their own."""
    import numpy as np

    path, c = folder("mixed"), sc.CASES["mixed"]
    ids = sc.prompt(c, 70, 8)
    out = Path(path).parent / "logits"
    out.mkdir()
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": ids[:60], "want": [0, 59]}], "end": []}] + \
        [{"step": 1 + i, "entries": [{"id": "x", "tokens": [t], "want": [0]}], "end": ["x"] if i == 9 else []} for i, t in enumerate(ids[60:])]
    r = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", path, "--dtype", "float32", "--out", str(out), "--max-tokens", "128"],
                       input="\n".join(json.dumps(s) for s in steps), capture_output=True, text=True, timeout=120)
    assert r.returncode == 0, r.stderr[-2000:]
    got = torch.cat([torch.from_numpy(np.fromfile(out / f"{i}.f32", "<f4")).view(-1, c["vocab"]) for i in range(11)])
    assert sc.error(got, _expected("mixed", ids)[[0] + list(range(59, 70))]).max().item() < LIMIT["float32"]
    r = subprocess.run([sys.executable, "-m", "crosspool_b200.cli.main", "generate", "--model", path, "--dtype", "float32", "--max-batch", "4",
                        "--max-seq-len", "256", "--max-new-tokens", "5", "--ids", ",".join(map(str, ids[:9])), "--ids", "3"],
                       capture_output=True, text=True, timeout=120, cwd=str(ROOT), env={**os.environ, "PYTHONPATH": str(ROOT)})
    assert r.returncode == 0, r.stderr[-2000:]
    lines = [json.loads(l)["output_ids"] for l in r.stdout.splitlines() if l.startswith("{")]
    assert lines == [_greedy("mixed", ids[:9], 5), _greedy("mixed", [3], 5)]
