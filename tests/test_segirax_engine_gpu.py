"""Segirax through the engine against the plain implementation: whole prompts, portions, decoding, batches, pages and slots
used again, greedy generation through the scheduler, sampling, the command line."""
import json
import os
import subprocess
import sys
from pathlib import Path

import pytest
import torch

import segirax_cases as sc
import segirax_oracle as oracle

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parents[1]
LIMIT = {"float32": 5e-5, "bfloat16": 6e-2}


@pytest.fixture(scope="module")
def folder(tmp_path_factory):
    d = tmp_path_factory.mktemp("segirax")
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

    kw = {**dict(max_batch=4, prefill_chunk=512, max_seq_len=512, page_size=16, max_prefill_seqs=4), **kw}
    return build_loopback([("m", path, 0)], EngineConfig(dtype=dtype, **kw)).instances[0].engine


def _feed(eng, s, ids, sizes):
    """Logits at every token of ``ids`` fed in portions of ``sizes`` (the last size repeats)."""
    out, at, i = [], 0, 0
    while at < len(ids):
        n = min(sizes[min(i, len(sizes) - 1)], len(ids) - at)
        out.append(eng.run_given([(s, ids[at:at + n])], [list(range(n))]))
        at, i = at + n, i + 1
    return torch.cat(out)


@pytest.mark.parametrize("dtype", list(LIMIT))
@pytest.mark.parametrize("name", list(sc.CASES))
def test_prompt_portions_and_token_by_token(folder, name, dtype):
    """The same 150 tokens whole, in portions of several sizes and one by one through captured decode graphs; pages and the
    state slot are used again each time and hold another sequence's leftovers."""
    eng = _engine(folder(name), dtype, num_pages=12)
    eng.warmup()
    c = sc.CASES[name]
    ids, other = sc.prompt(c, 150, 1), sc.prompt(c, 180, 2)
    want = _expected(name, ids)
    for sizes in ([150], [64, 1], [2], [17, 3, 40, 2, 16], [1], [100, 33, 1], [63, 65, 1]):
        s = eng.open_sequence()
        _feed(eng, s, other, [180])
        eng.close_sequence(s)
        s = eng.open_sequence()
        e = sc.error(_feed(eng, s, ids, sizes), want)
        eng.close_sequence(s)
        assert e.max().item() < LIMIT[dtype], (sizes, e.argmax().item(), e.max().item())
    assert eng.kv.allocator.free_pages == 12 and (eng.kv.slots is None or eng.kv.slots.free_slots == 4)


@pytest.mark.parametrize("dtype", list(LIMIT))
@pytest.mark.parametrize("name", ["mixed", "odd", "heads"])
def test_batches_of_unequal_requests_equal_each_alone(folder, name, dtype):
    """Portions of some requests beside single tokens of others, requests that pause, end, and hand pages and slots on."""
    c = sc.CASES[name]
    req = {k: sc.prompt(c, n, 10 + i) for i, (k, n) in enumerate({"a": 1, "b": 120, "c": 37, "d": 64, "e": 90, "f": 2}.items())}
    eng = _engine(folder(name), dtype, num_pages=24)
    eng.warmup()
    plan = [{"a": 1, "b": 40}, {"b": 1, "c": 20, "d": 63}, {"b": 2, "d": 1}, {"b": 1, "c": 1}, {"c": 16, "e": 30, "b": 17},
            {"b": 1, "e": 1}, {"f": 2, "e": 2}, {"b": 58, "e": 57}]
    at, live, got = {k: 0 for k in req}, {}, {k: [] for k in req}
    for step in plan:
        portions, ids = [], list(step)
        for k in ids:
            live.setdefault(k, None)
            if live[k] is None:
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
def test_a_far_key_is_found_from_every_schedule(folder, tmp_path, dtype):
    """Queries and keys of the first layer are made so that a marked token stands out among hundreds: losing it, or its
    page, changes the logits."""
    c = sc.model(64, 90, [(sc.latent(2, 16, 8, 32, 48, base=1e8), 64), (sc.lightning(2, 16, 16, [0.9, 0.99]), 64)])
    t = oracle.random_tensors(c, 7)
    # rotary dimensions almost stand still; both query heads look for the latent direction of token 7
    x = oracle.dynamic_tanh(t["embed"].double(), *(t["l0.norm1" + s].double() for s in (".alpha", "", ".b")))
    lat = oracle.rms(x @ t["l0.mix.dkv"].double()[:48].T, 1e-5) * t["l0.mix.dkv.norm"].double()
    key = (lat[7] @ t["l0.mix.uk"].double().T).view(2, 16)
    u = x.mean(0) / x.mean(0).norm()
    t["l0.mix.q"].view(2, 24, 64)[:, :16] = (key[:, :, None] * u * 6.0).bfloat16()
    t["l0.mix.o"] *= 4
    t["l0.rg1.b"] += 2
    path = sc.write_checkpoint(tmp_path / "far", c, t)
    ids = [i for i in sc.prompt(c, 420, 6) if i != 7][:400]
    ids[33] = 7
    want = oracle.forward(c, t, ids)
    without = oracle.forward(c, t, [i if j != 33 else 8 for j, i in enumerate(ids)])
    assert sc.error(without[380:], want[380:]).min().item() > 2 * LIMIT["bfloat16"]
    eng = _engine(path, dtype)
    for sizes in ([400], [34, 200, 1], [16, 33, 2, 64], [370, 1]):
        s = eng.open_sequence()
        e = sc.error(_feed(eng, s, ids, sizes), want)
        eng.close_sequence(s)
        assert e.max().item() < LIMIT[dtype], (sizes, e.argmax().item(), e.max().item())


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
    assert not eng.kv.tables and (eng.kv.slots is None or eng.kv.slots.free_slots == 3)


def test_a_retracted_sequence_is_recomputed_with_its_state(folder):
    """Too few pages for everyone: the engine takes one sequence's pages and slot away and rebuilds both later."""
    c = sc.CASES["mixed"]
    prompts = [sc.prompt(c, n, 40 + n) for n in (30, 29, 31)]
    eng = _engine(folder("mixed"), "float32", num_pages=8)
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

    assert run(temperature=5.0, seed=1) == run(temperature=5.0, seed=1) != run(temperature=5.0, seed=2)
    assert run() == run(temperature=0.0, seed=9)


def test_limits_are_checked_before_anything_runs(folder):
    eng = _engine(folder("mixed"), "bfloat16", num_pages=4)
    s = eng.open_sequence()
    for toks in ([], [-1], [211], list(range(0)), [1] * 513):
        with pytest.raises(ValueError):
            eng.run_given([(s, toks)], [[]])
    from crosspool_b200.engine.atn_engine import AttentionEngine, EngineConfig
    from crosspool_b200.engine.ffn_local import LocalFfnPort

    with pytest.raises(ValueError, match="prefix"):
        AttentionEngine(eng.cfg, eng.w, LocalFfnPort(eng.cfg, eng.port.weights), EngineConfig(prefix_cache=True))


def test_classic_models_take_running_sequences_along_too():
    from crosspool_b200.deployment import build_loopback
    from crosspool_b200.engine.atn_engine import EngineConfig
    from crosspool_b200.models import config as mc

    outs = []
    for mixed in (False, True):
        dep = build_loopback([("m", mc.preset("Qwen/Qwen3-0.6B").with_layers(2), 1)],
                             EngineConfig(max_batch=4, prefill_chunk=64, max_seq_len=256, mixed_batches=mixed))
        eng = dep.instances[0].engine
        g = torch.Generator().manual_seed(0)
        seqs = [eng.add_request(torch.randint(0, 1000, (n,), generator=g).tolist(), 6) for n in (20, 90)]
        eng.step(), eng.step()
        seqs.append(eng.add_request(torch.randint(0, 1000, (100,), generator=g).tolist(), 6))
        while eng.has_work:
            eng.step()
        outs.append([s.generated for s in seqs])
        assert not eng.kv.tables
    same = sum(a == b for x, y in zip(*outs) for a, b in zip(x, y))
    assert same >= 14        # 18 tokens; a near tie may fall the other way in bf16


def test_command_lines(folder):
    """``bin/trace_run`` and ``xpool generate`` as processes of their own."""
    path, c = folder("odd"), sc.CASES["odd"]
    ids = sc.prompt(c, 70, 8)
    out = Path(path).parent / "logits"
    out.mkdir()
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": ids[:60], "want": [0, 59]}], "end": []}] + \
        [{"step": 1 + i, "entries": [{"id": "x", "tokens": [t], "want": [0]}], "end": ["x"] if i == 9 else []} for i, t in enumerate(ids[60:])]
    r = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", path, "--dtype", "float32", "--out", str(out), "--max-tokens", "128"],
                       input="\n".join(json.dumps(s) for s in steps), capture_output=True, text=True, timeout=120)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(11)]
    import numpy as np

    got = torch.cat([torch.from_numpy(np.fromfile(out / f"{i}.f32", "<f4")).view(-1, c["vocab"]) for i in range(11)])
    want = _expected("odd", ids)
    assert sc.error(got, want[[0] + list(range(59, 70))]).max().item() < LIMIT["float32"]
    r = subprocess.run([sys.executable, "-m", "crosspool_b200.cli.main", "generate", "--model", path, "--dtype", "float32", "--max-batch", "4",
                        "--max-seq-len", "256", "--max-new-tokens", "5", "--ids", ",".join(map(str, ids[:9])), "--ids", "3"],
                       capture_output=True, text=True, timeout=120, cwd=str(ROOT), env={**os.environ, "PYTHONPATH": str(ROOT)})
    assert r.returncode == 0, r.stderr[-2000:]
    lines = [json.loads(l)["output_ids"] for l in r.stdout.splitlines() if l.startswith("{")]
    assert lines == [_greedy("odd", ids[:9], 5), _greedy("odd", [3], 5)]
