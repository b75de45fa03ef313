"""Shared parts of the design benchmarks (``bench.py --design NAME``): measured peaks, engine throughput of a model, kernel
timing with CUDA events, the table of kernels beside their counterparts."""
from __future__ import annotations

import json
import time
from pathlib import Path

import torch

DEV = "cuda"
VOCAB = 32768


def peaks():
    p = Path(__file__).resolve().parent.parent / "MEASURED_PEAKS.json"
    if p.exists():
        d = json.loads(p.read_text())
        return float(d["hbm_gbs"]), float(d["bf16_tflops"]), "measured"
    return 6650.0, 1590.0, "fallback"


def engine_rates(make, s, decode_rows=64, decode_new=128, prompt=1024, prompts=8):
    """Output tok/s of a decoding batch and prompt tok/s of a prefill, through the engine."""
    from mlxcel_b200.engine import EngineConfig, SamplingParams
    ml = prompt + decode_new + 64
    ecfg = EngineConfig(max_batch=decode_rows, max_num_batched_tokens=8192, prefill_chunk_alone=prompt, prefill_chunk_contended=prompt,
                        max_prefill_seqs=8, block_size=16, num_blocks=(ml // 16 + 2) * decode_rows, max_model_len=ml, prefix_cache=False)
    llm = make(s, ecfg)
    g = torch.Generator().manual_seed(0)
    draw = lambda n, ln: torch.randint(0, VOCAB, (n, ln), generator=g).tolist()            # noqa: E731
    sp = lambda n: SamplingParams(max_tokens=n, temperature=0.0, ignore_eos=True)          # noqa: E731

    def timed(n, ln, new):
        p = draw(n, ln)
        torch.cuda.synchronize()
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        t0 = time.perf_counter()
        e0.record()
        outs = llm.generate(prompt_token_ids=p, sampling_params=sp(new))
        e1.record()
        torch.cuda.synchronize()
        return e0.elapsed_time(e1) / 1e3, time.perf_counter() - t0, outs
    for _ in range(2):                                     # kernels' first launches, decode graphs
        timed(prompts, 64, 1), timed(decode_rows, 8, 8)
    pre = min(timed(prompts, prompt, 1)[0] for _ in range(2))
    # decode: the difference between two generation lengths from the same short prompts
    short, long = min(timed(decode_rows, 8, 8)[0] for _ in range(2)), min(timed(decode_rows, 8, 8 + decode_new)[0] for _ in range(2))
    st = llm.engine.stats
    out = dict(prefill_tok_s=round(prompts * prompt / pre), decode_tok_s=round(decode_rows * decode_new / (long - short)),
               decode_step_us=round((long - short) / decode_new * 1e6, 1), graph_replays=st["graph_replays"])
    del llm
    torch.cuda.empty_cache()
    return out


class Timer:
    def __init__(self):
        self.flush = torch.empty(256 << 20, dtype=torch.uint8, device=DEV)

    def __call__(self, fn, iters=9, warm=3):
        for _ in range(warm):
            fn()
        ts = []
        for _ in range(iters):
            self.flush.zero_()
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record()
            fn()
            e1.record()
            torch.cuda.synchronize()
            ts.append(e0.elapsed_time(e1))
        return sorted(ts)[len(ts) // 2] * 1e3              # us


class Table:
    """Rows (new kernel, share of its roofline, its counterpart, share): ``add`` times both."""

    def __init__(self):
        self.hbm, self.tf, _ = peaks()
        self.timer, self.rows = Timer(), []

    def add(self, role, bound, new, new_work, old=None, old_work=None):
        """bound "hbm": work in bytes; "tensor": in flops. new / old: (name, callable)."""
        share = (lambda w, us: round(w / us / 1e3 / self.hbm, 3)) if bound == "hbm" else (lambda w, us: round(w / us / 1e6 / self.tf, 3))
        a, b = self.timer(new[1]), self.timer(old[1]) if old else None
        self.rows.append(dict(role=role, bound=bound, kernel=new[0], us=round(a, 1), frac=share(new_work, a),
                              counterpart=old[0] if old else None, counterpart_us=round(b, 1) if old else None,
                              counterpart_frac=share(new_work if old_work is None else old_work, b) if old else None))
