"""Govopel on the CPU path: configuration and checkpoint reading, every mechanism's statement against the plain model, the
engine's portions / batches / pages, generation through the scheduler, the trace program."""
import contextlib
import json
import math
import subprocess
import sys
from pathlib import Path

import pytest
import torch

import oracle_govopel as O
from design_runs import interleave, llm_for, oracle_greedy, run_alone, run_mixed, tokens_for, worst
from mlxcel_b200 import ops
from mlxcel_b200.config import ModelConfig, preset
from mlxcel_b200.engine import SamplingParams
from mlxcel_b200.models.govopel import govopel_shapes, rotation_table
from mlxcel_b200.ops import KVLayer, latent, stream

TOL = 2e-5
ROOT = Path(__file__).resolve().parent.parent


def _gen(seed):
    return torch.Generator().manual_seed(seed)


# ----------------------------------------------------------------------------- configuration
def test_config_reader_keeps_every_constant_and_gives_each_layer_its_pool():
    raw = O.CONFIGS["mixed"]
    c = ModelConfig.from_dict(raw)
    assert c.model_type == "govopel" and (c.vocab_size, c.hidden_size, c.rms_norm_eps, c.final_logit_softcap) == (160, 96, 1e-5, 9.0)
    assert c.extra["layer_specs"] == raw["layers"] and c.extra["layer_runs"] == [0, 1, 2, 3]
    assert c.kv_geometry() == [(1, 72, 0), (2, 48, 48), (1, 56, 0), (1, 32, 32)]
    assert c.kv_bytes_per_token(16) == 2 * (72 + 192 + 56 + 64)
    assert set(govopel_shapes(c)) == set(O.random_tensors(raw, 0))
    assert all(tuple(v.shape) == govopel_shapes(c)[k] for k, v in O.random_tensors(raw, 0).items())
    att, lat = raw["layers"][1], raw["layers"][0]

    def edited(spec, **kw):
        return dict(raw, layers=[dict(spec, mixer=dict(spec["mixer"], **kw))])
    for bad in (edited(att, kv_heads=4), edited(att, vdim=24), edited(att, rot=dict(dims=64, base=1e4)), edited(att, mask=dict(size=0)),
                edited(lat, rot=dict(dims=8, base=1e4)), dict(raw, layers=[dict(att, type="convolution")]),
                dict(raw, layers=[dict(att, mlp=dict(kind="sparse", ff=8, limit=1.0))])):
        with pytest.raises(ValueError):
            ModelConfig.from_dict(bad)


def test_memory_estimate_counts_the_parameters():
    from mlxcel_b200.utils.memory import estimate_memory
    raw = O.CONFIGS["mixed"]
    c = ModelConfig.from_dict(raw)
    est = estimate_memory(c, ctx=256, parallel=2)
    have = sum(math.prod(s) for s in govopel_shapes(c).values())
    assert abs(est["parameters"] - have) <= 2 * c.hidden_size and est["kv_bytes_per_token"] == c.kv_bytes_per_token(16)


# ----------------------------------------------------------------------------- mechanisms
@pytest.mark.parametrize("scaling", [None, (2.0, 1000, 32.0, 1.0), (40.0, 50, 32.0, 1.0), (1.0, 64, 1.0, 1.0), (8.0, 4096, 4.0, 3.0)])
@pytest.mark.parametrize("dims,base", [(2, 10.0), (16, 3000.0), (64, 5e5)])
def test_frequency_table(dims, base, scaling):
    rot = O.attn_spec(1, 1, dims, dims, 8, 1.0, 1.0, None, base=base, scaling=scaling)["mixer"]["rot"]
    want, m = O.frequencies(rot)
    got, gm = rotation_table(rot, "cpu")
    assert torch.allclose(got.double(), want, rtol=1e-6) and abs(gm - m) < 1e-12


def test_stream_steps_without_inner_norm():
    g = _gen(0)
    table, w, ids = torch.randn(9, 37, generator=g), torch.randn(37, generator=g), torch.tensor([3, 0, 8, 3])
    h, x = stream.embed_stream(ids, table, 1.0, None, 1e-5, 0.0, w)
    assert torch.allclose(h.double(), O.embed(ids, table.double(), w.double(), 1e-5), atol=1e-6) and torch.equal(x, h)
    y, pw = torch.randn(4, 37, generator=g), torch.randn(37, generator=g)
    want = h.double() + O.norm(y.double(), pw.double(), 1e-5)
    x = stream.stream_norm(h, y, pw, None, None, 1e-5, 0.0, plain=True)
    assert torch.allclose(h.double(), want, atol=1e-6) and torch.equal(x, h)
    assert stream.stream_norm(h, y, pw, None, None, 1e-5, 0.0) is None


def test_glu_and_soft_cap():
    g = _gen(1)
    x, w = torch.randn(5, 24, generator=g) * 2, torch.randn(2 * 17, 24, generator=g)
    want = O.clipped_glu(x.double() @ w[:17].double().T, x.double() @ w[17:].double().T, 1.25)
    got = ops.glu_linear(x, w, 17, "clipped_swiglu", limit=1.25)
    assert torch.allclose(got.double(), want, atol=1e-5)
    z = torch.randn(5, 24, generator=g) * 10
    assert torch.allclose(stream.softcap_(z.clone(), 3.0).double(), O.soft_cap(z.double(), 3.0), atol=1e-6)


def _pool(blocks, h, bs, dk, dv, dtype=torch.float32):
    return KVLayer(torch.zeros(blocks, h, bs, dk, dtype=dtype), torch.zeros(blocks, h, bs, dv, dtype=dtype), None, None, bs)


def test_rotation_before_the_norm_and_values_from_raw_keys():
    g, T, Hq, Hkv, D = _gen(2), 11, 4, 2, 20
    rot = O.attn_spec(4, 2, D, 12, 8, 1.0, 1.0, None)["mixer"]["rot"]
    row = torch.randn(T, (Hq + Hkv) * D + 3, generator=g)
    kv, inv = _pool(4, Hkv, 4, D, D), rotation_table(rot, "cpu")
    src = row.clone()
    slots = torch.arange(T, dtype=torch.int32) + 2
    slots[5] = -1
    stream.rope_norm_append(row, torch.arange(T, dtype=torch.int32) + 7, slots, kv, Hq=Hq, Hkv=Hkv, Dk=D, Dv=D, inv_freq=inv[0],
                            mscale=inv[1], values_are_keys=True, eps=1e-5)
    turned = lambda z: O.unit_rms(O.rotate(z.double(), rot, 7), 1e-5)      # noqa: E731
    q, k = src[:, :Hq * D].view(T, Hq, D), src[:, Hq * D:(Hq + Hkv) * D].view(T, Hkv, D)
    assert torch.allclose(row[:, :Hq * D].view(T, Hq, D).double(), turned(q), atol=1e-5) and torch.equal(row[:, Hq * D:], src[:, Hq * D:])
    kr = turned(k)
    for t in range(T):
        s = int(slots[t])
        if s >= 0:
            assert torch.allclose(kv.k[s // 4, :, s % 4].double(), kr[t], atol=1e-5) and torch.equal(kv.v[s // 4, :, s % 4], k[t])
    assert not kv.k[7 // 4, :, 7 % 4].any()


def test_a_planted_key_is_seen_just_inside_its_chunk_only():
    """One key that outscores all others, at every place around chunk borders."""
    H, D, n, chunk = 2, 8, 41, 13
    for place in (0, 12, 13, 25, 26, 38):
        kv = _pool(3, 1, 16, D, D)
        k, v = torch.zeros(n, 1, D), torch.zeros(n, 1, D)
        k[place, 0, 0], v[place, 0, 1] = 60.0, 1.0
        kv.k.view(3, 16, D).view(-1, D)[:n], kv.v.view(-1, D)[:n] = k[:, 0], v[:, 0]
        q = torch.zeros(n, H * D)
        q[:, ::D] = 1.0
        out = torch.empty(n, H * D)
        stream.paged_attention(q, kv, torch.tensor([[0, 1, 2]]), torch.tensor([n]), torch.tensor([0, n]), out, Hq=H, Hkv=1, Dk=D, Dv=D,
                               scale=1.0, max_q_len=n, softcap=50.0, chunk=chunk)
        seen = out[:, 1] > 0.5
        assert seen.tolist() == [t >= place and t // chunk == place // chunk for t in range(n)]


def test_absorbed_latent_attention_equals_the_expanded_statement():
    raw = O.CONFIGS["mixed"]
    m, eps, n = raw["layers"][2]["mixer"], 1e-5, 23
    t = {k[7:]: v.double() for k, v in O.random_tensors(raw, 6).items() if k.startswith("l2.mix.")}
    h = torch.randn(n, 96, generator=_gen(3), dtype=torch.float64)
    llm = llm_for(raw, O.random_tensors(raw, 6), "cpu", torch.float32)
    w = llm.model.w.runs[2][0].attn
    a = h.float() @ w.w_in.T
    kv, C, R, D, H = _pool(4, 1, 16, 56, 0), 32, 24, m["dim"], m["heads"]
    pos = torch.arange(n, dtype=torch.int32)
    latent.latent_append(a, pos, pos, kv, Q=24, C=C, R=R, inv_freq=w.inv_freq, mscale=1.0, q_norm=w.q_norm, c_norm=w.c_norm, eps=eps)
    q = a[:, :24] @ w.w_uq.T
    qa = torch.empty(n, H * (C + R))
    ops.batched_linear(q, w.w_uk_t, qa, D + R, C + R)
    latent.latent_q_rope(q, qa, pos, H=H, q_at=D, q_head=D + R, d_at=C, d_head=C + R, inv_freq=w.inv_freq, mscale=1.0)
    o, out = torch.empty(n, H * C), torch.empty(n, H * m["vdim"])
    latent.latent_attention(qa, kv, torch.tensor([[0, 1, 2, 3]]), torch.tensor([n]), torch.tensor([0, n]), o, H=H, C=C, scale=m["scale"])
    ops.batched_linear(o, w.w_uv.view(H, m["vdim"], C), out, C, m["vdim"])
    assert torch.allclose((out @ w.out_proj.T).double(), O.latent_attention(h, t, m, eps), atol=1e-4)


# ----------------------------------------------------------------------------- whole models
@pytest.mark.parametrize("name", sorted(O.CONFIGS))
def test_prompt_portions_and_decoding_agree_with_the_plain_model(name):
    raw = O.CONFIGS[name]
    t = O.random_tensors(raw, seed=3)
    toks = tokens_for(raw, 53, 7)
    want, layers = O.forward(raw, t, toks, want_layers=True)
    llm = llm_for(raw, t, "cpu", torch.float32)
    llm.model.capture_layers = tuple(range(len(layers)))
    for sizes in ([53], [1], [2], [17, 3, 1, 8]):
        assert worst(run_alone(llm.engine, toks, sizes), want) < TOL, sizes
    run_alone(llm.engine, toks, [53])
    assert len(llm.model.captured) == len(layers)
    for got, ref in zip(llm.model.captured, layers):
        assert torch.allclose(got.double(), ref, atol=2e-4)


def test_mixed_batches_on_reused_pages_equal_each_request_alone():
    raw = O.CONFIGS["mixed"]
    t = O.random_tensors(raw, seed=5)
    lengths = [50, 7, 33, 1, 20, 18, 2, 41]
    seqs = [tokens_for(raw, n, 20 + i) for i, n in enumerate(lengths)]
    llm = llm_for(raw, t, "cpu", torch.float32, num_blocks=10, max_model_len=160)
    for got, s in zip(run_mixed(llm.engine, seqs, interleave(lengths, [[16, 2, 1], [1], [5, 1, 1, 9], [3, 2]])), seqs):
        assert worst(got, O.forward(raw, t, s)) < TOL
    assert llm.engine.bm.num_free == 10 and not llm.engine.seqs


def _planted(name, value):
    @contextlib.contextmanager
    def cm():
        saved = getattr(O, name)
        setattr(O, name, value(saved))
        try:
            yield
        finally:
            setattr(O, name, saved)
    return cm()


def _late_chunks(f):
    def chunk_mask(n, size):
        p = torch.arange(n)
        return (p[None, :] <= p[:, None]) & ((p[None, :] + 1) // size == (p[:, None] + 1) // size)
    return chunk_mask


def _edit(key, value):
    def wrap(f):
        def mixer(h, w, m, eps):
            return f(h, w, dict(m, **{key: value(m[key])}), eps)
        return mixer
    return wrap


def _unit_before_rotation(f):
    def attention(h, w, m, eps):
        plain, turn = O.unit_rms, O.rotate
        O.unit_rms, O.rotate = (lambda x, e: x), (lambda x, rot, start=0: turn(plain(x, eps), rot, start))
        try:
            return f(h, w, m, eps)
        finally:
            O.unit_rms, O.rotate = plain, turn
    return attention


FAULTS = {
    "chunks one off": ("chunk_mask", _late_chunks),
    "no chunks": ("chunk_mask", lambda f: lambda n, size: O.causal_mask(n)),
    "no soft cap": ("soft_cap", lambda f: lambda s, cap: s),
    "norm before the rotation": ("attention", _unit_before_rotation),
    "no scaling of the frequencies": ("attention", _edit("rot", lambda r: dict(r, scaling=None))),
    "rotation on too few dimensions": ("attention", _edit("rot", lambda r: dict(r, dims=r["dims"] - 2))),
    "latent scale": ("latent_attention", _edit("scale", lambda s: s * 1.01)),
    "latent rotation base": ("latent_attention", _edit("rot", lambda r: dict(r, base=r["base"] * 1.1))),
    "glu without the one": ("clipped_glu", lambda f: lambda g, u, limit: f(g, u - 1, limit)),
    "glu clip": ("clipped_glu", lambda f: lambda g, u, limit: f(g, u, limit * 1.05)),
    "embedding not normalised": ("embed", lambda f: lambda t, table, w, eps: table[torch.as_tensor(t)] * w),
}


@pytest.mark.parametrize("what", sorted(FAULTS))
def test_a_fault_in_any_mechanism_would_show(what):
    """The comparison's resolution: mistakes planted in the plain model move its logits far beyond the tolerance the engine is
    held to."""
    raw = O.CONFIGS["mixed"]
    t, toks = O.random_tensors(raw, seed=3), tokens_for(raw, 53, 7)
    want = O.forward(raw, t, toks)
    with _planted(*FAULTS[what]):
        assert worst(O.forward(raw, t, toks).float(), want) > 20 * TOL


# ----------------------------------------------------------------------------- entry points
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
        assert llm.engine.bm.num_free == llm.engine.ecfg.num_blocks


def test_prefix_cache():
    raw = O.CONFIGS["mixed"]
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
    cli.cmd_random_init(argparse.Namespace(preset="tiny-govopel", out=str(tmp_path), seed=3, quantize=None))
    raw, t = json.loads((tmp_path / "config.json").read_text()), load_file(str(tmp_path / "model.safetensors"))
    assert ModelConfig.from_path(tmp_path).extra == preset("tiny-govopel").extra
    llm = LLM.from_pretrained(tmp_path, device="cpu", dtype=torch.float32,
                              engine_config=EngineConfig(num_blocks=32, block_size=16, max_batch=4, max_model_len=128))
    toks = tokens_for(raw, 60, 1)
    want = torch.log_softmax(O.forward(raw, t, toks), -1)[:-1].gather(1, torch.tensor(toks[1:])[:, None])[:, 0]
    assert torch.allclose(llm.loglikelihoods(toks).double(), want, atol=1e-4)
    with pytest.raises(ValueError):
        LLM.from_pretrained(tmp_path, device="cpu", engine_config=EngineConfig(num_blocks=32, kv_bits=8))
    assert [f["executor"] for f in cli.arch_catalog()["families"] if f["name"] == "govopel"] == \
        [f["executor"] for f in cli.arch_catalog()["families"] if f["name"] == "pamasun"]


def test_trace_program_writes_the_wanted_logits(tmp_path):
    import numpy as np
    from safetensors.torch import save_file
    raw = O.CONFIGS["odd"]
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
    r = subprocess.run([sys.executable, str(ROOT / "bin" / "trace_run"), "--model", str(model), "--dtype", "float32", "--out", str(out),
                        "--max-tokens", "128", "--device", "cpu"], input="\n".join(lines) + "\n", text=True, capture_output=True, timeout=240)
    assert r.returncode == 0, r.stderr
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
    la, lb = O.forward(raw, t, a), O.forward(raw, t, b)
    for n, w in {1: torch.stack([lb[29], lb[3], la[18]]), 2: la[20][None], 3: torch.stack([la[20], lb[39]])}.items():
        got = torch.from_numpy(np.fromfile(out / f"{n}.f32", dtype="<f4")).view(len(w), -1)
        assert worst(got, w) < TOL
