"""Dofevik through the engine against the plain implementation: whole prompts, portions, decoding, batches, pages used again, window
and block edges, greedy generation through the scheduler, shared prefixes, sampling, the command line."""
import json
import os
import subprocess
import sys
from pathlib import Path

import pytest
import torch

import dofevik_cases as dc
import dofevik_oracle as oracle

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parents[1]
LIMIT = {"float32": 5e-5, "bfloat16": 8e-2}


@pytest.fixture(scope="module")
def folder(tmp_path_factory):
    d = tmp_path_factory.mktemp("dofevik")
    paths = {}

    def get(name):
        if name not in paths:
            paths[name] = dc.write_checkpoint(d / name, dc.CASES[name], dc.tensors(name))
        return paths[name]

    return get


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
@pytest.mark.parametrize("name", list(dc.CASES))
def test_prompt_portions_and_token_by_token(folder, name, dtype, page):
    """The same 150 tokens whole, in portions of several sizes and one by one through captured decode graphs; pages (and the block
    means beside them) are used again each time and hold another sequence's leftovers."""
    eng = _engine(folder(name), dtype, num_pages=192 // page, page_size=page)
    eng.warmup()
    ids, want = dc.clear_prompt(name, 150, 1)
    other = dc.prompt(dc.CASES[name], 180, 2)
    for sizes in ([150], [64, 1], [2], [17, 3, 40, 2, 16], [1], [100, 33, 1], [63, 65, 1], [1, 2, 3, 4, 5, 6]):
        s = eng.open_sequence()
        _feed(eng, s, other, [180])
        eng.close_sequence(s)
        s = eng.open_sequence()
        e = dc.error(_feed(eng, s, ids, sizes), want)
        eng.close_sequence(s)
        assert e.max().item() < LIMIT[dtype], (sizes, e.argmax().item(), e.max().item())
    assert eng.kv.allocator.free_pages == 192 // page


@pytest.mark.parametrize("dtype", list(LIMIT))
@pytest.mark.parametrize("name", ["mixed", "odd", "wide", "edges"])
def test_batches_of_unequal_requests_equal_each_alone(folder, name, dtype):
    """Portions of some requests beside single tokens of others, requests that pause, end, and hand pages on."""
    req = {k: dc.clear_prompt(name, n, 10 + i) for i, (k, n) in enumerate({"a": 1, "b": 120, "c": 37, "d": 64, "e": 90, "f": 2}.items())}
    eng = _engine(folder(name), dtype, num_pages=6)
    eng.warmup()
    plan = [{"a": 1, "b": 40}, {"b": 1, "c": 20, "d": 63}, {"b": 2, "d": 1}, {"b": 1, "c": 1}, {"c": 16, "e": 30, "b": 17},
            {"b": 1, "e": 1}, {"f": 2, "e": 2}, {"b": 58, "e": 57}]
    at, live, got = {k: 0 for k in req}, {}, {k: [] for k in req}
    for step in plan:
        portions, names = [], list(step)
        for k in names:
            if k not in live:
                live[k] = eng.open_sequence()
            portions.append((live[k], req[k][0][at[k]:at[k] + step[k]]))
            at[k] += step[k]
        out = eng.run_given(portions, [list(range(step[k])) for k in names])
        for k, o in zip(names, out.split([step[k] for k in names])):
            got[k].append(o)
        for k in names:
            if at[k] == len(req[k][0]):
                eng.close_sequence(live.pop(k))
    assert not live
    for k, (_, want) in req.items():
        e = dc.error(torch.cat(got[k]), want)
        assert e.max().item() < LIMIT[dtype], (k, e.argmax().item(), e.max().item())


@pytest.mark.parametrize("dtype", list(LIMIT))
@pytest.mark.parametrize("kind,size,pool", [("attention", 40, 0), ("attention", 64, 0), ("attention", 130, 0), ("pooled", 40, 5), ("pooled", 33, 12), ("pooled", 64, 64),
                                            ("pooled", 70, 9), ("latent", 40, 0), ("latent", 64, 0), ("latent", 130, 0)])
def test_a_marked_token_is_seen_exactly_as_long_as_it_should(tmp_path, kind, size, pool, dtype):
    """Every query looks for a marked token. It is the first one, lies at both sides of a page's and a block's border, and leaves
    windows (and comes back with its block) in the middle of prompts, of portions and of decoding."""
    c, t = dc.marked_model(kind, size, pool)
    path = dc.write_checkpoint(tmp_path / "m", c, t)
    ids = [i for i in dc.prompt(c, 420, 6) if i != dc.MARK][:300]
    eng = _engine(path, dtype)
    eng.warmup()
    for place in (0, 5, 63, 64, 100):
        ids_p = ids[:place] + [dc.MARK] + ids[place + 1:]
        want = oracle.forward(c, t, ids_p)
        edge = place + size                                  # the first token that no longer sees it
        back = place // pool * pool + pool - 1 + size if pool else edge
        for sizes in ([300], [edge - 2, 1, 1, 1, 1, 40, 2], [edge - 1, 3, 30], [place + 1, 1], [34, 16, 200, 1], [back - 1, 1, 1, 1, 2, 60]):
            s = eng.open_sequence()
            e = dc.error(_feed(eng, s, ids_p, sizes), want)
            eng.close_sequence(s)
            assert e.max().item() < LIMIT[dtype], (place, sizes, e.argmax().item(), e.max().item())


@pytest.mark.parametrize("name", ["mixed", "edges"])
def test_long_decoding_in_32_bit(folder, name):
    ids, want = dc.clear_prompt(name, 500, 4, margin=1e-4)
    eng = _engine(folder(name), "float32")
    eng.warmup()
    s = eng.open_sequence()
    assert dc.error(_feed(eng, s, ids, [3, 1]), want).max().item() < LIMIT["float32"]


def test_every_layer_in_32_bit(folder):
    """The residual stream behind every layer."""
    name = "mixed"
    ids, _ = dc.clear_prompt(name, 90, 3)
    layers: list = []
    oracle.forward(dc.CASES[name], dc.tensors(name), ids, layer_outputs=layers)
    eng = _engine(folder(name), "float32")
    seen = []

    def tap(layer, rows, pending):
        from crosspool_b200.ops import mixers as M

        r = eng.body.resid[:rows].clone()
        M.resid_norm(r, None, None, **pending)
        seen.append(r)

    eng.body.tap = tap
    s = eng.open_sequence()
    eng.run_given([(s, ids)], [[0]])
    assert len(seen) == len(layers)
    for got, want in zip(seen, layers):
        assert torch.allclose(got.double().cpu(), want, rtol=1e-4, atol=1e-4)


def _greedy(name, prompt, n):
    c, t, ids = dc.CASES[name], dc.tensors(name), list(prompt)
    for _ in range(n):
        ids.append(int(oracle.forward(c, t, ids)[-1].argmax()))
    return ids[len(prompt):]


@pytest.mark.parametrize("mixed", [False, True])
@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_greedy_generation_through_the_scheduler(folder, name, mixed):
    """Chunked prefill, more requests than decode rows, requests that arrive while others decode."""
    prompts = [dc.prompt(dc.CASES[name], n, 20 + n) for n in (1, 40, 23, 70, 2, 33)]
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
    assert not eng.kv.tables


def test_a_retracted_sequence_is_recomputed_with_its_blocks(folder):
    """Too few pages for everyone: the engine takes one sequence's pages away and rebuilds them later."""
    prompts = [dc.prompt(dc.CASES["mixed"], n, 40 + n) for n in (30, 29, 31)]
    eng = _engine(folder("mixed"), "float32", num_pages=8, page_size=16)
    out = eng.generate(prompts, 24)
    assert out == [_greedy("mixed", p, 24) for p in prompts]
    assert eng.kv.allocator.free_pages == 8


def test_shared_prefixes(folder, tmp_path):
    """Whole pages of a prompt serve a second request, with windows and block means that reach into them. Where blocks and pages
    do not fit, sharing is refused."""
    name = "shared"
    dc.CASES[name] = dc.model(64, 90, [(dc.pooled(2, 2, 32, 20, 2), dc.moe(4, 2, 16)), (dc.attention(4, 2, 64, 64, 50), None),
                                       (dc.latent(4, 32, 16, 32, 48, 64, 40), dc.moe(4, 2, 32, 24))])
    path = dc.write_checkpoint(tmp_path / name, dc.CASES[name], dc.tensors(name))
    with pytest.raises(ValueError, match="prefix sharing"):
        _engine(folder("mixed"), "float32", prefix_cache=True)
    p = dc.prompt(dc.CASES[name], 120, 5)
    eng = _engine(path, "float32", page_size=16, prefix_cache=True)
    a = eng.generate([p + [3]], 12)[0]
    b = eng.generate([p + [4]], 12)[0]
    c = eng.generate([p[:70] + [5]], 12)[0]
    assert a == _greedy(name, p + [3], 12) and b == _greedy(name, p + [4], 12) and c == _greedy(name, p[:70] + [5], 12) and len(eng.prefix) > 0


def test_sampling_is_seeded_and_greedy_at_temperature_zero(folder):
    eng = _engine(folder("mixed"), "bfloat16", sampling=True)
    p = dc.prompt(dc.CASES["mixed"], 12, 3)

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

    path, c = folder("mixed"), dc.CASES["mixed"]
    ids, want = dc.clear_prompt("mixed", 70, 8)
    out = Path(path).parent / "logits"
    out.mkdir()
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": ids[:60], "want": [0, 59]}], "end": []}] + \
        [{"step": 1 + i, "entries": [{"id": "x", "tokens": [t], "want": [0]}], "end": ["x"] if i == 9 else []} for i, t in enumerate(ids[60:])]
    r = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", path, "--dtype", "float32", "--out", str(out), "--max-tokens", "128"],
                       input="\n".join(json.dumps(s) for s in steps), capture_output=True, text=True, timeout=120)
    assert r.returncode == 0, r.stderr[-2000:]
    got = torch.cat([torch.from_numpy(np.fromfile(out / f"{i}.f32", "<f4")).view(-1, c["vocab"]) for i in range(11)])
    assert dc.error(got, want[[0] + list(range(59, 70))]).max().item() < LIMIT["float32"]
    r = subprocess.run([sys.executable, "-m", "crosspool_b200.cli.main", "generate", "--model", path, "--dtype", "float32", "--max-batch", "4",
                        "--max-seq-len", "256", "--max-new-tokens", "5", "--ids", ",".join(map(str, ids[:9])), "--ids", "3"],
                       capture_output=True, text=True, timeout=120, cwd=str(ROOT), env={**os.environ, "PYTHONPATH": str(ROOT)})
    assert r.returncode == 0, r.stderr[-2000:]
    lines = [json.loads(l)["output_ids"] for l in r.stdout.splitlines() if l.startswith("{")]
    assert lines == [_greedy("mixed", ids[:9], 5), _greedy("mixed", [3], 5)]
