"""Vavadra on the CPU path: configuration and checkpoint reading, every mechanism's statement against the plain model, the
engine's portions / batches / pages / slots, generation through the scheduler, the trace program."""
import contextlib
import json
import math
import subprocess
import sys
from pathlib import Path

import pytest
import torch

import oracle_vavadra as O
from design_runs import interleave, llm_for, oracle_greedy, run_alone, run_mixed, tokens_for, worst
from mlxcel_b200.config import ModelConfig, preset
from mlxcel_b200.engine import SamplingParams
from mlxcel_b200.models.vavadra import second_map_factor, vavadra_shapes
from mlxcel_b200.ops import KVLayer, moe, stream
from mlxcel_b200.ops.reference import rope_inv_freq

TOL = 2e-5
ROOT = Path(__file__).resolve().parent.parent


def _gen(seed):
    return torch.Generator().manual_seed(seed)


# ----------------------------------------------------------------------------- configuration
def test_config_reader_keeps_every_constant_and_gives_each_run_its_pool_or_slab():
    raw = O.CONFIGS["mixed"]
    c = ModelConfig.from_dict(raw)
    assert c.model_type == "vavadra" and (c.vocab_size, c.hidden_size, c.rms_norm_eps, c.embed_scale) == (160, 96, 1e-5, 3.0)
    assert c.extra["layer_specs"] == raw["layers"] and c.extra["loop"] == raw["loop"] and c.extra["logit_scale"] == 0.8
    assert c.extra["layer_runs"] == [0, 1, 2, 1, 2, 1, 2, 3]
    assert c.kv_geometry() == [(1, 64, 0), (2, 32, 40)] * 3 + [(1, 48, 0)]
    assert set(vavadra_shapes(c)) == set(O.random_tensors(raw, 0))
    for name, r in O.CONFIGS.items():
        assert all(tuple(v.shape) == vavadra_shapes(ModelConfig.from_dict(r))[k] for k, v in O.random_tensors(r, 0).items()), name
    delta, lat, att = raw["layers"][:3]
    edited = lambda spec, **kw: dict(raw, loop=None, layers=[dict(spec, mixer=dict(spec["mixer"], **kw))])      # noqa: E731
    router = lambda **kw: dict(raw, loop=None, layers=[dict(delta, mlp=dict(delta["mlp"], router=dict(delta["mlp"]["router"], **kw)))])   # noqa: E731
    for bad in (edited(att, kv_heads=4), edited(att, mask=dict(size=0)), edited(lat, rot=dict(dims=8, base=1e4)), edited(delta, conv=0),
                edited(delta, kv_heads=3), router(top=8), router(experts=0), dict(raw, layers=[dict(att, type="convolution")] * 3),
                dict(raw, layers=[dict(att, mlp=dict(delta["mlp"], kind="dense"))] * 3), dict(raw, loop=dict(start=2, stop=5, times=2))):
        with pytest.raises(ValueError):
            ModelConfig.from_dict(bad)


@pytest.mark.parametrize("name", sorted(O.CONFIGS))
def test_memory_estimate_counts_parameters_and_state(name):
    from mlxcel_b200.utils.memory import estimate_memory
    raw = O.CONFIGS[name]
    c = ModelConfig.from_dict(raw)
    est = estimate_memory(c, ctx=256, parallel=2)
    have = sum(math.prod(s) for s in vavadra_shapes(c).values())
    assert abs(est["parameters"] - have) <= (2 + (raw["loop"] or {"times": 0})["times"]) * c.hidden_size + len(c.extra["layer_runs"])
    assert est["kv_bytes_per_token"] == c.kv_bytes_per_token(16)


# ----------------------------------------------------------------------------- mechanisms
def test_stream_steps():
    g = _gen(0)
    table, vec, w, ids = torch.randn(9, 37, generator=g), torch.randn(37, generator=g), torch.randn(37, generator=g), torch.tensor([3, 0, 8, 3])
    h, x = stream.embed_stream(ids, table, 2.0, w, 1e-5, 0.0, vec=vec)
    first = table.double()[ids] * 2.0
    assert torch.allclose(h.double(), O.before_pass(first, first, vec[None].double(), 0), atol=1e-6)
    assert torch.allclose(x.double(), O.norm(h.double(), w.double(), 1e-5), atol=1e-6)
    y = torch.randn(4, 37, generator=g)
    want = O.before_pass(h.double() + y.double(), first, vec[None].double().repeat(2, 1), 1)
    stream.stream_norm(h, y, None, None, w, 1e-5, 0.0, entry=stream.Entry(vec, ids, table, 2.0))
    assert torch.allclose(h.double(), want, atol=1e-6)


def test_rotation_pairs_neighbours():
    x = torch.randn(5, 3, 11, generator=_gen(1))
    inv = rope_inv_freq(6, 50.0, None)[0]
    got = stream.rotate_half(x, torch.arange(5) + 9, inv, 1.0, adjacent=True)
    assert torch.allclose(got.double(), O.rotate(x.double(), dict(dims=6, base=50.0), 9), atol=1e-5)


def test_factor_of_the_second_map():
    t = {n: torch.randn(7, generator=_gen(i)) * 0.5 for i, n in enumerate(("lq1", "lk1", "lq2", "lk2"))}
    assert abs(second_map_factor(t.__getitem__, "", 0.3) - float(O.map_weight({k: v.double() for k, v in t.items()}, 0.3))) < 1e-9


def test_a_planted_key_is_seen_by_its_map_inside_its_chunk_only():
    """One key that outscores all others in one map, at every place around chunk borders."""
    H, D, n, chunk = 2, 4, 41, 13
    for place in (0, 12, 13, 25, 26, 38):
        for which in (0, 1):
            k, v, q = torch.zeros(n, 1, 2, D), torch.zeros(n, 1, 3), torch.zeros(n, H, 2, D)
            k[place, 0, which, 0], v[place, 0, 1] = 60.0, 1.0
            q[..., 0] = 1.0
            kv = KVLayer(torch.zeros(3, 1, 16, 2 * D), torch.zeros(3, 1, 16, 3), None, None, 16)
            kv.k.view(-1, 2 * D)[:n], kv.v.view(-1, 3)[:n] = k.view(n, -1), v.view(n, -1)
            out = torch.empty(n, H * 3)
            stream.paged_attention(q.view(n, -1), kv, torch.tensor([[0, 1, 2]]), torch.tensor([n]), torch.tensor([0, n]), out, Hq=H, Hkv=1, Dk=2 * D,
                                   Dv=3, scale=1.0, max_q_len=n, chunk=chunk, diff=(0.5, 1.0, 1e-4))
            m = O.chunk_mask(n, chunk)
            a = [O.attend(q[:, 0, i].double() @ k[:, 0, i].double().T, m, v[:, 0].double()) for i in (0, 1)]
            assert torch.allclose(out[:, :3].double(), O.combine_maps(*a, 0.5, 0.0, 1e-4), atol=1e-5)
            inside = torch.tensor([t > place + 1 and t // chunk == place // chunk for t in range(n)])
            blind = torch.tensor([t < place or t // chunk != place // chunk for t in range(n)])
            assert not out[blind].any() and (out[inside, 1] * (1 if which == 0 else -1) > 0.5).all()


def test_choice_by_corrected_score_weight_by_plain_score():
    z, c = torch.randn(30, 9, generator=_gen(2)) * 2, torch.randn(9, generator=_gen(3)) * 0.3
    ids, wts = moe.route_choice(z, c, 4, 2.5)
    want, ww = O.choose(z.double(), c.double(), 4, 2.5)
    assert torch.equal(ids.long(), want) and torch.allclose(wts.double(), ww, atol=1e-6)


# ----------------------------------------------------------------------------- whole models
@pytest.mark.parametrize("name", sorted(O.CONFIGS))
def test_prompt_portions_and_decoding_agree_with_the_plain_model(name):
    raw = O.CONFIGS[name]
    t = O.random_tensors(raw, seed=3)
    toks = tokens_for(raw, 53, 7)
    want, layers = O.forward(raw, t, toks, want_layers=True)
    llm = llm_for(raw, t, "cpu", torch.float32)
    for sizes in ([53], [1], [2], [17, 3, 1, 8]):
        assert worst(run_alone(llm.engine, toks, sizes), want) < TOL, sizes
    llm.model.capture_layers = tuple(range(len(layers)))
    assert worst(run_alone(llm.engine, toks, [53]), want) < TOL
    assert len(llm.model.captured) == len(layers)
    for got, ref in zip(llm.model.captured, layers):
        assert torch.allclose(got.double(), ref, atol=2e-4)


def test_mixed_batches_on_reused_pages_and_slots_equal_each_request_alone():
    raw = O.CONFIGS["mixed"]
    t = O.random_tensors(raw, seed=5)
    lengths = [50, 7, 33, 1, 20, 18, 2, 41]
    seqs = [tokens_for(raw, n, 20 + i) for i, n in enumerate(lengths)]
    llm = llm_for(raw, t, "cpu", torch.float32, num_blocks=10, max_model_len=160)
    for got, s in zip(run_mixed(llm.engine, seqs, interleave(lengths, [[16, 2, 1], [1], [5, 1, 1, 9], [3, 2]])), seqs):
        assert worst(got, O.forward(raw, t, s)) < TOL
    assert llm.engine.bm.num_free == 10 and not llm.engine.seqs and len(llm.model.ssm.free) == 4


@contextlib.contextmanager
def _planted(name, wrap):
    saved = getattr(O, name)
    setattr(O, name, wrap(saved))
    try:
        yield
    finally:
        setattr(O, name, saved)


def _edit(**changes):
    """A mixer whose record is changed."""
    return lambda f: lambda h, w, m, eps: f(h, w, dict(m, **{k: v(m[k]) for k, v in changes.items()}), eps)


def _spec(change):
    return lambda f: lambda h, w, spec: f(h, w, change(spec))


def _late_chunks(f):
    def chunk_mask(n, size):
        p = torch.arange(n) + 1
        return (p[None, :] <= p[:, None]) & (p[None, :] // size == p[:, None] // size)
    return chunk_mask


def _rotate_halves(f):
    def rotate(x, rot, start=0):
        n = rot["dims"]
        order = torch.arange(x.shape[-1])
        order[:n] = torch.cat([torch.arange(0, n, 2), torch.arange(1, n, 2)])
        return f(x[..., torch.argsort(order)], rot, start)[..., order]
    return rotate


def _decay_behind_the_write(f):
    def memory(q, k, v, beta, g):
        S, out = q.new_zeros(q.shape[1], q.shape[2], v.shape[2]), []
        for t in range(q.shape[0]):
            u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
            S = g[t][:, None, None] * (S + k[t][:, :, None] * u[:, None, :])
            out.append(torch.einsum("hdv,hd->hv", S, q[t]))
        return torch.stack(out)
    return memory


def _read_before_write(f):
    def memory(q, k, v, beta, g):
        return torch.cat([torch.zeros_like(v[:1]), f(q, k, v, beta, g)[:-1]])
    return memory


def _renormalised(f):
    def choose(z, c, top, scale):
        ids, w = f(z, c, top, scale)
        return ids, w / w.sum(-1, keepdim=True) * scale
    return choose


def _weights_from_choice(f):
    def choose(z, c, top, scale):
        ids, w = f(z, c, top, scale)
        return ids, w + c[ids] * scale
    return choose


FAULTS = {
    "chunks one off": ("chunk_mask", _late_chunks),
    "no chunks": ("chunk_mask", lambda f: lambda n, size: f(n, n)),
    "window one longer": ("window_mask", lambda f: lambda n, size: f(n, size + 1)),
    "window one shorter": ("window_mask", lambda f: lambda n, size: f(n, size - 1)),
    "no sink": ("attend", lambda f: lambda s, m, v, sink=None: f(s, m, v)),
    "sink scaled": ("attend", lambda f: lambda s, m, v, sink=None: f(s, m, v, sink if sink is None else sink * 0.9)),
    "halves rotated": ("rotate", _rotate_halves),
    "rotation base": ("latent_attention", _edit(rot=lambda r: dict(r, base=r["base"] * 1.1))),
    "latent scale": ("latent_attention", _edit(scale=lambda s: s * 1.01)),
    "attention scale": ("attention", _edit(scale=lambda s: s * 1.01)),
    "second map's factor": ("map_weight", lambda f: lambda w, diff: f(w, diff) * 1.01),
    "no gain behind the maps": ("combine_maps", lambda f: lambda a, b, lam, diff, eps: f(a, b, lam, 0.0, eps)),
    "taps reversed": ("short_conv", lambda f: lambda x, taps: f(x, taps.flip(1))),
    "decay behind the write": ("delta_memory", _decay_behind_the_write),
    "read-out before the write": ("delta_memory", _read_before_write),
    "write rate": ("delta_memory", lambda f: lambda q, k, v, beta, g: f(q, k, v, beta * 0.99, g)),
    "decay": ("delta_memory", lambda f: lambda q, k, v, beta, g: f(q, k, v, beta, g ** 1.02)),
    "no unit vectors": ("unit", lambda f: lambda x: x),
    "heads grouped the other way": ("delta_memory", lambda f: lambda q, k, v, beta, g: f(q.flip(1), k.flip(1), v, beta, g)),
    "no correction": ("choose", lambda f: lambda z, c, top, scale: f(z, c * 0, top, scale)),
    "weights from the corrected scores": ("choose", _weights_from_choice),
    "weights renormalised": ("choose", _renormalised),
    "router scale": ("experts", _spec(lambda s: dict(s, router=dict(s["router"], scale=s["router"]["scale"] * 1.02)))),
    "expert limit": ("experts", _spec(lambda s: dict(s, expert=dict(s["expert"], limit=s["expert"]["limit"] * 1.05)))),
    "shared expert's limit": ("experts", _spec(lambda s: dict(s, shared=dict(s["shared"], limit=s["expert"]["limit"])))),
    "no shared expert": ("experts", _spec(lambda s: dict(s, shared=None))),
    "glu without the one": ("clipped_glu", lambda f: lambda g, u, limit: f(g, u - 1, limit)),
    "embedding added in the first pass too": ("before_pass", lambda f: lambda x, first, step, t: x + first + step[t]),
    "embedding not added": ("before_pass", lambda f: lambda x, first, step, t: x + step[t]),
    "the first step in every pass": ("before_pass", lambda f: lambda x, first, step, t: f(x, first, step[:1].expand_as(step), t)),
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


def test_prefix_cache_of_a_model_without_recurrent_layers():
    raw = O.CONFIGS["latent_only"]
    t, p = O.random_tensors(raw, seed=2), tokens_for(raw, 40, 3)
    llm = llm_for(raw, t, "cpu", torch.float32, prefix_cache=True)
    sp = SamplingParams(max_tokens=4, temperature=0.0, ignore_eos=True)
    first, again = (llm.generate(prompt_token_ids=[p], sampling_params=sp)[0].output for _ in range(2))
    assert first == again == oracle_greedy(O, raw, t, p, 4) and llm.engine.stats["prefix_hit_tokens"] == 32


def test_loglikelihoods_and_checkpoint_round_trip(tmp_path):
    import argparse

    from safetensors.torch import load_file

    from mlxcel_b200 import cli
    from mlxcel_b200.engine import EngineConfig
    from mlxcel_b200.llm import LLM
    cli.cmd_random_init(argparse.Namespace(preset="tiny-vavadra", out=str(tmp_path), seed=3, quantize=None))
    raw, t = json.loads((tmp_path / "config.json").read_text()), load_file(str(tmp_path / "model.safetensors"))
    assert ModelConfig.from_path(tmp_path).extra == preset("tiny-vavadra").extra
    llm = LLM.from_pretrained(tmp_path, device="cpu", dtype=torch.float32,
                              engine_config=EngineConfig(num_blocks=32, block_size=16, max_batch=4, max_model_len=128))
    toks = tokens_for(raw, 60, 1)
    want = torch.log_softmax(O.forward(raw, t, toks), -1)[:-1].gather(1, torch.tensor(toks[1:])[:, None])[:, 0]
    assert torch.allclose(llm.loglikelihoods(toks).double(), want, atol=1e-4)
    with pytest.raises(ValueError):
        LLM.from_pretrained(tmp_path, device="cpu", engine_config=EngineConfig(num_blocks=32, kv_bits=8))
    fams = {f["name"]: f for f in cli.arch_catalog()["families"]}
    assert fams["vavadra"]["executor"] == fams["pamasun"]["executor"] and fams["vavadra"]["checked_against"] == fams["pamasun"]["checked_against"]


def test_a_missing_tensor_is_named(tmp_path):
    from safetensors.torch import save_file

    from mlxcel_b200.llm import LLM
    raw = O.CONFIGS["odd"]
    t = {k: v.to(torch.bfloat16).contiguous() for k, v in O.random_tensors(raw, 0).items() if k != "loop.step"}
    (tmp_path / "config.json").write_text(json.dumps(raw))
    save_file(t, str(tmp_path / "model.safetensors"))
    with pytest.raises(KeyError, match="loop.step"):
        LLM.from_pretrained(tmp_path, device="cpu")


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
