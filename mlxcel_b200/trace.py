"""Trace replay: given token ids through a model, step by step, on the serving engine; nothing is sampled.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N   < steps.jsonl

Every input line is one step, ``{"step": 7, "entries": [{"id": "r1", "tokens": [11, 4, 9, 2], "want": [3]}], "end": ["r0"]}``:
the next tokens of each live request and the places among them whose logits are wanted, all run as one
batch (:meth:`Engine.feed`). The logits go to ``DIR/<step>.f32`` (little-endian fp32, ``[wanted, vocab]``, in the
order of the entries and places) and ``done <step>`` is printed after every step. ``end`` gives a request's
cache blocks and state slot back. The block pool holds N tokens and there are four state slots.

Exit code 3: ``--dtype float32`` for a model that has no fp32 kernels.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

LIVE_REQUESTS = 4


def build_engine(model_dir: str, dtype: str, max_tokens: int, device: str):
    import torch

    from . import _build
    from .config import ModelConfig
    from .engine import EngineConfig
    from .llm import LLM
    from .models.designs import DESIGNS
    from .ops import _lib

    cfg = ModelConfig.from_path(model_dir)
    if dtype == "float32" and cfg.model_type not in DESIGNS:
        raise SystemExit(3)
    _lib.prefer_units(_build.MODEL_UNITS.get(cfg.model_type))
    torch.backends.cuda.matmul.allow_tf32 = False
    torch.backends.cudnn.allow_tf32 = False
    block = 16
    blocks = max(1, -(-max_tokens // block))
    ecfg = EngineConfig(max_batch=LIVE_REQUESTS, max_prefill_seqs=LIVE_REQUESTS, state_slots=LIVE_REQUESTS, block_size=block,
                        num_blocks=blocks, max_num_batched_tokens=blocks * block, max_model_len=blocks * block,
                        prefix_cache=False, watermark=0.0)
    return LLM.from_pretrained(model_dir, device=device, engine_config=ecfg, dtype=getattr(torch, dtype)).engine


def replay(engine, lines, out_dir: str, emit) -> None:
    """Runs the steps of ``lines`` and calls ``emit(text)`` after each."""
    from .ops import _lib

    live: dict[str, int] = {}
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        entries = []
        for e in step["entries"]:
            if e["id"] not in live:
                live[e["id"]] = engine.open_sequence()
            entries.append((live[e["id"]], e["tokens"], e.get("want") or []))
        logits = engine.feed(entries) if entries else None
        if logits is not None:
            data = logits.float().cpu().contiguous().numpy().astype("<f4", copy=False)
        if engine.is_cuda:
            code = _lib.read_status(engine.device)
            if code:
                raise RuntimeError(f"a kernel reported failure code {code}")
        if logits is not None:
            with open(os.path.join(out_dir, f"{step['step']}.f32"), "wb") as f:
                f.write(data.tobytes())
        for rid in step.get("end") or []:
            if rid in live:
                engine.close_sequence(live.pop(rid))
        emit(f"done {step['step']}")


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.split("\n", 1)[0])
    add_arguments(ap)
    return run(ap.parse_args(argv))


def add_arguments(ap) -> None:
    ap.add_argument("--model", required=True, help="folder with config.json and safetensors")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True, help="folder the logits are written to")
    ap.add_argument("--max-tokens", type=int, required=True, help="tokens the cache pool holds")
    ap.add_argument("--device", default="cuda")


def run(a) -> int:
    engine = build_engine(a.model, a.dtype, a.max_tokens, a.device)
    os.makedirs(a.out, exist_ok=True)

    def emit(text):
        sys.stdout.write(text + "\n")
        sys.stdout.flush()

    replay(engine, iter(sys.stdin.readline, ""), a.out, emit)
    return 0
