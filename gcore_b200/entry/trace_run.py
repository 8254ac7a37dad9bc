"""Replays given token ids through a served model, step by step, and writes logits; nothing is sampled.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Steps come on standard input, one JSON object a line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

``entries`` brings the next tokens of each request and the places among them whose logits are wanted; all entries of a
step run as one batch.  A request is admitted at its first entry; those under ``end`` are finished after the step and give
back what they hold.  Logits go to ``DIR/<step>.f32`` (little-endian 32-bit floats, [wanted, vocab], in entry order), and
``done <step>`` is printed after every step.  The engine is the one that generates: its scheduler, paged cache, state
slots and kernels, with a cache pool for ``N`` tokens and slots for four requests."""
from __future__ import annotations

import argparse
import json
import os
import sys

PAGE = 64
REQUESTS = 4


def build_engine(model_dir: str, dtype: str, max_tokens: int, device, requests: int = REQUESTS):
    from ..checkpoint.hf import load_serving_model
    from ..rollout.engine import InferEngine, RolloutWeights
    cfg, model = load_serving_model(model_dir, device, dtype)
    blocks = (max_tokens + PAGE - 1) // PAGE
    eng = InferEngine(cfg, RolloutWeights.from_model(model), max_running_requests=requests,
                      max_model_len=min(cfg.max_position_embeddings, blocks * PAGE), kv_block_size=PAGE,
                      num_kv_blocks=blocks, device=device)
    eng.wake_up()
    return eng


def replay(engine, lines, out_dir: str, emit):
    """Runs the steps of ``lines``; ``emit`` receives the text to print after each."""
    live = {}
    for line in lines:
        if not line.strip():
            continue
        s = json.loads(line)
        for e in s["entries"]:
            if e["id"] not in live:
                live[e["id"]] = engine.open_request()
        logits = engine.step([(live[e["id"]], e["tokens"]) for e in s["entries"]], [e["want"] for e in s["entries"]])
        if logits is not None:
            part = os.path.join(out_dir, f".{s['step']}.part")
            with open(part, "wb") as f:
                f.write(logits.float().cpu().contiguous().numpy().astype("<f4").tobytes())
            os.replace(part, os.path.join(out_dir, f"{s['step']}.f32"))
        for rid in s.get("end", []):
            engine.close_request(live.pop(rid))
        emit(f"done {s['step']}")


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replays a trace of token ids and writes logits")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", required=True, choices=("bfloat16", "float32"))
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, required=True, help="tokens the cache pool holds")
    a = ap.parse_args(argv)
    import torch
    from .. import build_native
    from ..checkpoint.hf import read_model_config
    from ..ops import _lib
    if not torch.cuda.is_available():
        raise RuntimeError("trace_run needs a GPU")
    cfg = read_model_config(a.model)
    if cfg is None or cfg.layer_plan is None:
        raise ValueError(f"{a.model} does not hold a model whose steps can be replayed")
    _lib.use_library(build_native.ensure_kernels(cfg.arch))
    engine = build_engine(a.model, a.dtype, a.max_tokens, torch.device("cuda", 0))

    def emit(text):
        _lib.check_device_errors()
        print(text, flush=True)

    replay(engine, sys.stdin, a.out, emit)
    return 0
