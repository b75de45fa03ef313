"""Pamasun on the CPU path: configuration and checkpoint reading, every mechanism's statement against the plain
model, the engine's portions / batches / slots, generation through the scheduler, the trace program."""
import json
import subprocess
import sys
from pathlib import Path

import pytest
import torch

import oracle_pamasun as O
from mlxcel_b200.config import ModelConfig, preset
from mlxcel_b200.engine import SamplingParams
from mlxcel_b200.ops import stream
from design_runs import cut, interleave, llm_for, oracle_greedy, run_alone, run_mixed, tokens_for, worst

TOL = 2e-5
ROOT = Path(__file__).resolve().parent.parent


def test_config_reader_orders_runs_and_geometry():
    c = ModelConfig.from_dict(O.CONFIGS["odd"])
    assert c.model_type == "pamasun" and (c.vocab_size, c.hidden_size) == (101, 75) and c.rms_norm_eps == 1e-4
    assert c.extra["layer_runs"] == [0, 1, 2, 1, 2, 1, 2] == O.layer_order(O.CONFIGS["odd"])
    assert c.kv_geometry() == [(1, 20, 13)] + [(4, 12, 36)] * 3
    assert c.kv_bytes_per_token(16) == 2 * (33 + 3 * 4 * 48)
    assert ModelConfig.from_dict(O.CONFIGS["attention_only"]).extra["layer_runs"] == [0, 1]
    bad = dict(O.CONFIGS["mixed"], loop=dict(start=1, stop=5, times=2))
    with pytest.raises(ValueError):
        ModelConfig.from_dict(bad)
    with pytest.raises(ValueError):
        ModelConfig.from_dict(dict(O.CONFIGS["mixed"], layers=[dict(type="convolution", mixer={}, mlp=None)], loop=None))
    with pytest.raises(ValueError):
        ModelConfig.from_dict(O.model_config(64, 32, [O.attn_spec(3, 2, 16, 16, 0.2, None)], None))


def test_memory_estimate_counts_shared_weights_once_and_state_per_run():
    from mlxcel_b200.utils.memory import estimate_memory
    raw = O.CONFIGS["mixed"]
    est = estimate_memory(ModelConfig.from_dict(raw), ctx=256, parallel=2)
    assert est["recurrent_state_bytes_per_seq"] == 4 * (2 * 3 * 24 * 24 + 2 * 32 * 32)
    once = estimate_memory(ModelConfig.from_dict(dict(raw, loop=None)), ctx=256, parallel=2)
    assert abs(est["parameters"] - once["parameters"]) <= 4 and est["kv_bytes_per_token"] == 2 * once["kv_bytes_per_token"]


def test_polynorm_and_stream_norm_match_the_plain_statement():
    g = torch.Generator().manual_seed(0)
    z, coef = torch.randn(5, 37, generator=g), torch.tensor([0.9, -0.4, 0.3, 0.25])
    assert torch.allclose(stream.polynorm(z, coef, 1e-5), O.polynorm(z.double(), coef.double(), 1e-5).float(), atol=1e-6)
    h, y, w, w2 = torch.randn(5, 37, generator=g), torch.randn(5, 37, generator=g), torch.randn(37, generator=g), torch.randn(37, generator=g)
    ls = torch.rand(37, generator=g)
    want_h = h.double() + O.around_zero_norm(y.double(), w.double(), 1e-5) * ls.double()
    x = stream.stream_norm(h, y, w, ls, w2, 1e-5, 1.0)
    assert torch.allclose(h.double(), want_h, atol=1e-6)
    assert torch.allclose(x.double(), O.around_zero_norm(want_h, w2.double(), 1e-5), atol=1e-5)


def test_delta_recurrence_statement_matches_the_matrix_form():
    """One step written with matrices: S <- (diag(w) - (a u) u^T) S + k v^T."""
    g = torch.Generator().manual_seed(1)
    r, k, v = (torch.randn(6, 2, 7, generator=g, dtype=torch.float64) for _ in range(3))
    w, a = torch.rand(6, 2, 7, generator=g, dtype=torch.float64), torch.rand(6, 2, 7, generator=g, dtype=torch.float64)
    out, last = O.delta_recurrence(r, k, v, w, a)
    S = torch.zeros(2, 7, 7, dtype=torch.float64)
    for t in range(6):
        for h in range(2):
            u = k[t, h] / (k[t, h].dot(k[t, h]) + 1e-6).sqrt()
            S[h] = (torch.diag(w[t, h]) - torch.outer(a[t, h] * u, u)) @ S[h] + torch.outer(k[t, h], v[t, h])
            assert torch.allclose(out[t, h], S[h].T @ r[t, h])
    assert torch.allclose(last, S)


@pytest.mark.parametrize("name", sorted(O.CONFIGS))
def test_prompt_portions_and_decoding_agree_with_the_plain_model(name):
    raw = O.CONFIGS[name]
    t = O.random_tensors(raw, seed=3)
    toks = tokens_for(raw, 45, 7)
    want, layers = O.forward(raw, t, toks, want_layers=True)
    llm = llm_for(raw, t, "cpu", torch.float32)
    llm.model.capture_layers = tuple(range(len(layers)))
    for sizes in ([45], [1], [2], [17, 3, 1, 8]):
        assert worst(run_alone(llm.engine, toks, sizes), want) < TOL, sizes
    run_alone(llm.engine, toks, [45])
    assert len(llm.model.captured) == len(layers)
    for got, ref in zip(llm.model.captured, layers):
        assert torch.allclose(got.double(), ref, atol=2e-4)


def test_mixed_batches_on_reused_pages_and_slots_equal_each_request_alone():
    raw = O.CONFIGS["mixed"]
    t = O.random_tensors(raw, seed=5)
    lengths = [50, 7, 33, 1, 20, 18, 2, 41]
    seqs = [tokens_for(raw, n, 20 + i) for i, n in enumerate(lengths)]
    sched = interleave(lengths, [[16, 2, 1], [1], [5, 1, 1, 9], [3, 2]])
    llm = llm_for(raw, t, "cpu", torch.float32, num_blocks=10, max_model_len=160)
    for got, s in zip(run_mixed(llm.engine, seqs, sched), seqs):
        assert worst(got, O.forward(raw, t, s)) < TOL
    assert llm.engine.bm.num_free == 10 and len(llm.model.ssm.free) == 4 and not llm.engine.seqs


def test_feed_refuses_what_does_not_fit_and_a_fifth_live_request():
    raw = O.CONFIGS["mixed"]
    eng = llm_for(raw, O.random_tensors(raw, 1), "cpu", torch.float32, num_blocks=4, max_model_len=64, max_num_batched_tokens=64).engine
    ids = [eng.open_sequence() for _ in range(5)]
    for s in ids[:4]:
        eng.feed([(s, [1, 2], [])])
    with pytest.raises(RuntimeError):
        eng.feed([(ids[4], [3], [0])])
    with pytest.raises(RuntimeError):
        eng.feed([(ids[0], [1] * 20, [])])


def test_a_fault_in_any_mechanism_would_show():
    """The comparison's resolution: mistakes planted in the plain model move its logits far beyond the
    tolerance the engine is held to."""
    raw = O.CONFIGS["mixed"]
    t = O.random_tensors(raw, seed=3)
    toks = tokens_for(raw, 45, 7)
    want = O.forward(raw, t, toks)

    def off_by(**edit):
        saved = {k: getattr(O, k) for k in edit}
        try:
            for k, v in edit.items():
                setattr(O, k, v)
            return worst(O.forward(raw, t, toks).float(), want)
        finally:
            for k, v in saved.items():
                setattr(O, k, v)
    bias, recur = O.distance_bias, O.delta_recurrence

    def shifted(r1, r2, n):
        return bias(r1, r2, n + 1)[:, 1:, :-1]                       # every distance one too far

    def forgetful(r, k, v, w, a, state=None):                       # state lost in the middle
        o1, _ = recur(r[:20], k[:20], v[:20], w[:20], a[:20])
        o2, s = recur(r[20:], k[20:], v[20:], w[20:], a[20:])
        return torch.cat([o1, o2]), s

    def new_state_read(r, k, v, w, a, state=None):                  # removal reads the decayed state
        n, h, d = r.shape
        s, out = torch.zeros(h, d, d, dtype=r.dtype), []
        for i in range(n):
            u = k[i] / (k[i].pow(2).sum(-1, keepdim=True) + 1e-6).sqrt()
            s = w[i][:, :, None] * s
            s = s - (a[i] * u)[:, :, None] * (u[:, :, None] * s).sum(1)[:, None] + k[i][:, :, None] * v[i][:, None]
            out.append((s * r[i][:, :, None]).sum(1))
        return torch.stack(out), s
    assert off_by(distance_bias=shifted) > 20 * TOL
    assert off_by(delta_recurrence=forgetful) > 20 * TOL
    assert off_by(delta_recurrence=new_state_read) > 20 * TOL
    assert off_by(sink_softmax=lambda s, sink: torch.softmax(s, -1)) > 20 * TOL
    assert off_by(layer_order=lambda cfg: range(len(cfg["layers"]))) > 20 * TOL


def test_greedy_generation_through_the_scheduler():
    raw = O.CONFIGS["mixed"]
    t = O.random_tensors(raw, seed=9)
    prompts = [tokens_for(raw, n, 40 + n) for n in (23, 1, 9, 30, 4)]
    want = [oracle_greedy(O, raw, t, p, 6) for p in prompts]
    sp = SamplingParams(max_tokens=6, temperature=0.0, ignore_eos=True)
    for kw in (dict(), dict(max_batch=2, max_num_batched_tokens=8, num_blocks=6)):       # roomy; queueing, portions, preemption
        llm = llm_for(raw, t, "cpu", torch.float32, **kw)
        outs = llm.generate(prompt_token_ids=prompts, sampling_params=sp)
        assert [s.output for s in outs] == want, kw
        assert not llm.model.ssm.slot_of and llm.engine.bm.num_free == llm.engine.ecfg.num_blocks


def test_prefix_cache_serves_stacks_without_state():
    raw = O.CONFIGS["attention_only"]
    t = O.random_tensors(raw, seed=2)
    p = tokens_for(raw, 40, 3)
    llm = llm_for(raw, t, "cpu", torch.float32, prefix_cache=True)
    sp = SamplingParams(max_tokens=4, temperature=0.0, ignore_eos=True)
    first = llm.generate(prompt_token_ids=[p], sampling_params=sp)[0].output
    again = llm.generate(prompt_token_ids=[p], sampling_params=sp)[0].output
    assert first == again == oracle_greedy(O, raw, t, p, 4) and llm.engine.stats["prefix_hit_tokens"] == 32


def test_loglikelihoods_and_checkpoint_round_trip(tmp_path):
    import argparse

    from safetensors.torch import load_file

    from mlxcel_b200 import cli
    from mlxcel_b200.engine import EngineConfig
    from mlxcel_b200.llm import LLM
    cli.cmd_random_init(argparse.Namespace(preset="tiny-pamasun", out=str(tmp_path), seed=3, quantize=None))
    raw, t = json.loads((tmp_path / "config.json").read_text()), load_file(str(tmp_path / "model.safetensors"))
    assert ModelConfig.from_path(tmp_path).extra == preset("tiny-pamasun").extra
    llm = LLM.from_pretrained(tmp_path, device="cpu", dtype=torch.float32,
                              engine_config=EngineConfig(num_blocks=32, block_size=16, max_batch=4, max_model_len=128))
    toks = tokens_for(raw, 30, 1)
    want = torch.log_softmax(O.forward(raw, t, toks), -1)[:-1].gather(1, torch.tensor(toks[1:])[:, None])[:, 0]
    assert torch.allclose(llm.loglikelihoods(toks).double(), want, atol=1e-4)
    with pytest.raises(ValueError):
        LLM.from_pretrained(tmp_path, device="cpu", engine_config=EngineConfig(num_blocks=32, kv_bits=8))


def _trace(args, lines):
    return subprocess.run([sys.executable, str(ROOT / "bin" / "trace_run"), *args], input="\n".join(lines) + "\n", text=True,
                          capture_output=True, timeout=240)


def test_trace_program_writes_the_wanted_logits(tmp_path):
    import numpy as np
    from safetensors.torch import save_file
    raw = O.CONFIGS["mixed"]
    t = O.random_tensors(raw, seed=4)
    model, out = tmp_path / "m", tmp_path / "out"
    model.mkdir()
    (model / "config.json").write_text(json.dumps(raw))
    save_file({k: v.to(torch.bfloat16).contiguous() for k, v in t.items()}, str(model / "model.safetensors"))
    a, b = tokens_for(raw, 21, 1), tokens_for(raw, 40, 2)
    lines = [json.dumps(x) for x in (
        dict(step=0, entries=[dict(id="a", tokens=a[:18], want=[])], end=[]),
        dict(step=1, entries=[dict(id="b", tokens=b[:30], want=[29, 3]), dict(id="a", tokens=a[18:19], want=[0])], end=[]),
        dict(step=2, entries=[dict(id="a", tokens=a[19:], want=[1])], end=["a"]),
        dict(step=3, entries=[dict(id="a", tokens=a, want=[20]), dict(id="b", tokens=b[30:], want=[9])], end=["a", "b"]))]
    r = _trace(["--model", str(model), "--dtype", "float32", "--out", str(out), "--max-tokens", "128", "--device", "cpu"], lines)
    assert r.returncode == 0, r.stderr
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
    la, lb = O.forward(raw, t, a), O.forward(raw, t, b)
    want = {1: torch.stack([lb[29], lb[3], la[18]]), 2: la[20][None], 3: torch.stack([la[20], lb[39]])}
    for n, w in want.items():
        got = torch.from_numpy(np.fromfile(out / f"{n}.f32", dtype="<f4")).view(len(w), -1)
        assert worst(got, w) < TOL
    assert not (out / "0.f32").exists()


def test_trace_program_refuses_fp32_for_other_families(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps(dict(model_type="llama", hidden_size=64)))
    r = _trace(["--model", str(tmp_path), "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "64", "--device", "cpu"], [])
    assert r.returncode == 3


def test_schedules_cover_every_token_once():
    sched = interleave([5, 9, 1], [[2], [1, 4]], width=2)
    assert [sum(s.get(i, 0) for s in sched) for i in range(3)] == [5, 9, 1] and cut(10, [4, 3]) == [4, 3, 3]
