"""Trace replay: feeds given token ids through a model step by step and writes logits.

Drives :meth:`AttentionEngine.run_given`, i.e. the engine's own forward passes, paged cache, state slots and captured decode
graphs; nothing is sampled. One JSON object per line of standard input::

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

``entries`` bring the next tokens of live requests (all of them run as one batch), ``want`` names the places among those
tokens whose logits are written to ``<out>/<step>.f32`` (little-endian fp32 ``[wanted, vocab]``, in order), ``end`` lists
the requests that are finished after the step. ``done <step>`` is printed after every step.
"""

from __future__ import annotations

import argparse
import json
import os
import sys

PAGE = 64          # tokens per cache page
LIVE = 4           # requests alive at once: state slots, decode rows


def parse_args(argv=None):
    ap = argparse.ArgumentParser(prog="trace_run", description="replay given tokens through the engine, write logits")
    ap.add_argument("--model", required=True, help="folder with config.json and safetensors files")
    ap.add_argument("--dtype", choices=("bfloat16", "float32"), default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True,
                    help="tokens that live requests hold at most, each request rounded up to whole 64-token pages")
    return ap.parse_args(argv)


def build_engine(model: str, dtype: str, max_tokens: int):
    from ..deployment import build_loopback
    from ..engine.atn_engine import EngineConfig

    pages = (max_tokens + PAGE - 1) // PAGE
    ecfg = EngineConfig(max_batch=LIVE, prefill_chunk=pages * PAGE, max_seq_len=pages * PAGE, page_size=PAGE, num_pages=pages,
                        max_prefill_seqs=LIVE, dtype=dtype)
    return build_loopback([("trace", model, 0)], ecfg).instances[0].engine


class Replay:
    def __init__(self, engine, out_dir: str):
        self.engine, self.out_dir = engine, out_dir
        self.live: dict[str, object] = {}

    def step(self, record: dict) -> None:
        portions, want = [], []
        for e in record["entries"]:
            if e["id"] not in self.live:
                self.live[e["id"]] = self.engine.open_sequence()
            portions.append((self.live[e["id"]], [int(t) for t in e["tokens"]]))
            want.append([int(w) for w in e["want"]])
        if portions:
            logits = self.engine.run_given(portions, want)
            if logits.shape[0]:
                path = os.path.join(self.out_dir, f"{record['step']}.f32")
                logits.cpu().numpy().astype("<f4").tofile(path)
        for rid in record.get("end", ()):
            s = self.live.pop(rid, None)
            if s is not None:
                self.engine.close_sequence(s)


def main(argv=None) -> int:
    args = parse_args(argv)
    from ..native import build

    build.build_kernels()
    engine = build_engine(args.model, args.dtype, args.max_tokens)
    engine.warmup()
    replay = Replay(engine, args.out)
    for line in sys.stdin:
        if not line.strip():
            continue
        record = json.loads(line)
        replay.step(record)
        print(f"done {record['step']}", flush=True)
    return 0
