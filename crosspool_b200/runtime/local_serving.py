"""One GPU serves one model whole (``xpool serve`` / ``xpool generate``): the attention engine with its FFNs in-stream, no
daemon and no FFN tier. The serving endpoint is the one of a deployed Instance (``runtime/serving.py``)."""

from __future__ import annotations

import json


def build(model: str, *, dtype: str = "bfloat16", gpu: int = 0, max_batch: int = 64, max_seq_len: int = 8192, kv_tokens: int = 0,
          page_size: int = 64, sampling: bool = True):
    """A warmed-up single-Instance :class:`Deployment` of a checkpoint directory or preset."""
    import torch

    from ..deployment import build_loopback
    from ..engine.atn_engine import EngineConfig

    torch.cuda.set_device(gpu)
    ecfg = EngineConfig(max_batch=max_batch, max_seq_len=max_seq_len, page_size=page_size, dtype=dtype, sampling=sampling,
                        num_pages=(kv_tokens + page_size - 1) // page_size)
    dep = build_loopback([(model, model, 0)], ecfg, device=f"cuda:{gpu}")
    dep.warmup()
    return dep


def _from_args(ns, sampling: bool):
    return build(ns.model, dtype=ns.dtype, gpu=ns.gpu, max_batch=ns.max_batch, max_seq_len=ns.max_seq_len, kv_tokens=ns.kv_tokens,
                 sampling=sampling)


def serve(ns) -> int:
    import os

    import uvicorn

    from .serving import EngineLoop, create_serving_app, load_tokenizers

    loop = EngineLoop(_from_args(ns, sampling=True))
    loop.start()
    app = create_serving_app(loop, [ns.model], tokenizer=load_tokenizers({ns.model: ns.model if os.path.isdir(ns.model) else None}))
    uvicorn.run(app, host=ns.host, port=ns.port, log_level="warning")
    loop.stop()
    return 0 if loop.error is None else 1


def generate(ns) -> int:
    prompts = [[int(t) for t in p.split(",")] for p in ns.ids]
    dep = _from_args(ns, sampling=ns.temperature > 0)
    seqs = [dep.add_request(ns.model, p, ns.max_new_tokens, temperature=ns.temperature, seed=ns.seed) for p in prompts]
    dep.run_until_idle()
    for s in seqs:
        print(json.dumps({"prompt_tokens": len(s.prompt), "output_ids": s.generated}), flush=True)
    return 0
