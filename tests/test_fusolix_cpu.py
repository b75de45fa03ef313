"""Fusolix on the CPU path: configuration and checkpoint reading, every mechanism's statement against the plain model, the
engine's portions / batches / pages / slots, generation through the scheduler, the trace program."""
import contextlib
import json
import math
import subprocess
import sys
from pathlib import Path

import pytest
import torch

import oracle_fusolix as O
from design_runs import bounds, interleave, llm_for, oracle_greedy, paged_tables, run_alone, run_mixed, tokens_for, worst
from mlxcel_b200.config import ModelConfig, preset
from mlxcel_b200.engine import SamplingParams
from mlxcel_b200.models.fusolix import fusolix_shapes
from mlxcel_b200.ops import KVLayer, block_means, moe, retention, stream, streams
from mlxcel_b200.ops.reference import rope_inv_freq

TOL = 2e-5
ROOT = Path(__file__).resolve().parent.parent


def _gen(seed):
    return torch.Generator().manual_seed(seed)


# ----------------------------------------------------------------------------- configuration
def test_config_reader_keeps_every_constant_and_gives_each_layer_its_pool():
    raw = O.CONFIGS["mixed"]
    c = ModelConfig.from_dict(raw)
    assert c.model_type == "fusolix" and (c.vocab_size, c.hidden_size, c.rms_norm_eps, c.embed_scale) == (160, 96, 1e-5, 2.0)
    assert c.extra["layer_specs"] == raw["layers"] and (c.extra["streams"], c.extra["taps"]) == (3, 4)
    assert c.kv_geometry() == [(2, 32, 40), (3, 16, 24), (1, 24, 16)] and c.kv_means() == [4, 6, 16]
    assert set(fusolix_shapes(c)) == set(O.random_tensors(raw, 0))
    for name, r in O.CONFIGS.items():
        assert all(tuple(v.shape) == fusolix_shapes(ModelConfig.from_dict(r))[k] for k, v in O.random_tensors(r, 0).items()), name
    first = raw["layers"][0]
    side = lambda which, **kw: dict(raw, layers=[dict(first, mixer=dict(first["mixer"], **{which: dict(first["mixer"][which], **kw)}))])   # noqa: E731
    router = lambda **kw: dict(raw, layers=[dict(first, mlp=dict(first["mlp"], router=dict(first["mlp"]["router"], **kw)))])   # noqa: E731
    for bad in (side("left", kv_heads=3), side("left", mask=dict(size=0, pool=4)), side("left", mask=dict(size=4, pool=0)),
                side("right", decay=[0.5]), side("right", decay=[0.5, 1.5]), side("right", rot=dict(dims=26, base=1e4)),
                side("right", rot=dict(dims=3, base=1e4)), router(top=7), router(experts=10), router(groups=dict(count=3, keep=4)),
                dict(raw, streams=0), dict(raw, canon=dict(taps=0)), dict(raw, layers=[dict(first, type="attention")]),
                dict(raw, layers=[dict(first, mlp=dict(first["mlp"], kind="ensemble"))])):
        with pytest.raises(ValueError):
            ModelConfig.from_dict(bad)


@pytest.mark.parametrize("name", sorted(O.CONFIGS))
def test_memory_estimate_counts_parameters_pool_and_state(name):
    from mlxcel_b200.cache.kv_pool import KVPool
    from mlxcel_b200.utils.memory import estimate_memory
    raw = O.CONFIGS[name]
    c = ModelConfig.from_dict(raw)
    est = estimate_memory(c, ctx=256, parallel=2)
    assert abs(est["parameters"] - sum(math.prod(s) for s in fusolix_shapes(c).values())) <= c.hidden_size
    llm = llm_for(raw, O.random_tensors(raw, 0), "cpu", torch.float32)
    assert est["recurrent_state_bytes_per_seq"] == sum(t[0].numel() * 4 for t in llm.model.ssm.state)
    slabs = sum(t[0].numel() for layer in llm.engine.kv_layers for t in (layer.k, layer.v, layer.k_mean, layer.v_mean))
    assert KVPool.bytes_per_block(c, 16) == 2 * slabs and est["kv_bytes_per_token"] == c.kv_bytes_per_token() == 2 * slabs // 16


# ----------------------------------------------------------------------------- mechanisms
def _around(S, H, K, g):
    n = lambda *s: torch.randn(*s, generator=g)      # noqa: E731
    return streams.Sublayer(w_in=n(S), w_out=n(S), mix=n(S, S), norm_w=n(H), norm_b=n(H), taps=n(K, H), bias=n(H))


def test_streams_step_and_its_convolution():
    g, S, H, K, T = _gen(0), 3, 11, 4, 9
    a, b = _around(S, H, K, g), _around(S, H, K, g)
    xs, y = torch.randn(T, S, H, generator=g), torch.randn(T, H, generator=g)
    want = O.spread(xs.double(), y.double() + a.bias.double(), a.mix.double(), a.w_out.double())
    n = O.layer_norm(O.gather_streams(want, b.w_in.double()), b.norm_w.double(), b.norm_b.double(), 1e-5)
    want_x = O.short_conv(n, b.taps.t().double())
    total = streams.sum_streams(xs, a, y, None, torch.float32)
    assert torch.allclose(total.double(), want.sum(1), atol=1e-5)
    tail, got = torch.full((2, K - 1, H), 7.0), []
    for i, (lo, hi) in enumerate(((0, 4), (4, 5), (5, 6), (6, 9))):       # portions of one sequence in slot 1
        part = xs[lo:hi].clone()
        pieces = (torch.tensor([1]), torch.tensor([0, hi - lo]), torch.tensor([int(i == 0)]), 0, hi - lo)
        got.append(streams.mix_streams(part, a, y[lo:hi], None, b, 1e-5, torch.float32, tail, pieces))
        assert torch.allclose(part.double(), want[lo:hi], atol=1e-5)
    assert torch.allclose(torch.cat(got).double(), want_x, atol=1e-5)
    assert (tail[0] == 7).all() and torch.allclose(tail[1].double(), n[-(K - 1):], atol=1e-5)


def test_embedding_fills_every_stream():
    g = _gen(1)
    b, table, ids = _around(2, 5, 1, g), torch.randn(9, 5, generator=g), torch.tensor([3, 0, 8])
    xs, x = streams.embed_streams(ids, table, 1.5, 2, b, 1e-5, torch.zeros(1, 0, 5), (torch.tensor([0]), torch.tensor([0, 3]), torch.tensor([1]), 0, 3))
    e = O.embedding(table.double(), ids, 1.5)
    assert torch.allclose(xs.double(), e[:, None].repeat(1, 2, 1))
    n = O.layer_norm(e * b.w_in.sum().double(), b.norm_w.double(), b.norm_b.double(), 1e-5)
    assert torch.allclose(x.double(), O.short_conv(n, b.taps.t().double()), atol=1e-5)


@pytest.mark.parametrize("bs,size,pool", [(16, 18, 4), (16, 11, 6), (16, 5, 16), (16, 7, 23), (16, 1, 1), (8, 20, 3), (16, 40, 32)])
def test_a_planted_block_is_seen_from_its_window_exit_on(bs, size, pool):
    """A key that outscores all others, at every place around block, window and page borders: seen itself inside the window, not
    at all between, and by its block's mean behind it."""
    n, Dk, Dv, lens = 75, 4, 3, [75]
    tab, nb = paged_tables(lens, bs)
    for place in (0, pool - 1, pool, 2 * pool - 1, 30, 47, 48, n - 1):
        if place >= n:
            continue
        row = torch.zeros(n, Dk + Dk + Dv)
        row[:, 0], row[place, Dk], row[place, 2 * Dk + 1] = 1.0, 60.0 * pool, 1.0
        per = -(-bs // pool)
        kv = KVLayer(torch.zeros(nb, 1, bs, Dk), torch.zeros(nb, 1, bs, Dv), None, None, bs, 16, torch.full((nb, 1, per, Dk), 9.0),
                     torch.full((nb, 1, per, Dv), 9.0), pool)
        got, at = [], 0
        for count in (13, 1, 1, 34, 2, 24):
            pos = torch.arange(at, at + count)
            slots = tab[0, pos // bs] * bs + pos % bs
            b = type("B", (), dict(pf_cu_q_host=[0, count], pf_starts=[at], pf_context_lens=torch.tensor([at + count])))()
            args = (tab, torch.tensor([at + count]), torch.tensor([0, count]))
            block_means.append(row[at:at + count], pos, slots.to(torch.int32), kv, args[0], args[2], Hq=1, Hkv=1, Dk=Dk, Dv=Dv)
            out = torch.empty(count, Dv)
            stream.paged_attention(row[at:at + count, :Dk], kv, *args, out, Hq=1, Hkv=1, Dk=Dk, Dv=Dv, scale=1.0, max_q_len=count, window=size,
                                   means=block_means.portion_means(b, size, pool))
            got.append(out)
            at += count
        got = torch.cat(got)
        k, v = row[:, None, Dk:2 * Dk].double(), row[:, None, 2 * Dk:].double()
        keys, vals = torch.cat([k, O.block_means(k, pool)])[:, 0], torch.cat([v, O.block_means(v, pool)])[:, 0]
        seen = torch.cat([O.tokens_seen(n, size), O.blocks_seen(n, size, pool)], 1)
        assert torch.allclose(got.double(), O.attend(row[:, :Dk].double() @ keys.T, seen, vals), atol=1e-5)
        t, last = torch.arange(n), place // pool * pool + pool - 1
        inside, behind = (t >= place) & (t < place + size), t >= last + size
        assert (got[inside, 1] > 0.5).all() and (got[behind, 1] * pool > 0.5).all() and not got[~inside & ~behind].any()


def test_portion_means_cover_what_the_last_row_sees():
    assert [block_means.seen(n, 10, 4) for n in (1, 13, 14, 17, 18, 50)] == [0, 0, 1, 1, 2, 10]


def test_retention_over_portions_and_a_reused_slot():
    H, D, V, T, rot = 2, 6, 5, 23, dict(dims=4, base=30.0)
    g = _gen(3)
    proj = torch.randn(T, 2 * H * (D + V), generator=g)
    decay = torch.tensor([0.5, 1.0])
    q, k = (O.rotate(proj[:, i * H * D:(i + 1) * H * D].double().view(T, H, D), rot) for i in (0, 1))
    v, gate = proj[:, 2 * H * D:2 * H * D + H * V].double().view(T, H, V), proj[:, 2 * H * D + H * V:].double()
    want = O.unit_rms(O.retain(q, k * D ** -0.5, v, decay.double()), 1e-4).reshape(T, -1) * O.silu(gate) * 0.7
    memory, out = torch.full((3, H, D, V), 5.0), torch.empty(T, H * V)
    for i, (lo, hi) in enumerate(((0, 9), (9, 10), (10, 12), (12, 23))):
        retention.retention(proj[lo:hi], torch.arange(lo, hi), rope_inv_freq(4, 30.0, None)[0], decay, memory, torch.tensor([2]),
                            torch.tensor([0, hi - lo]), torch.tensor([int(i == 0)]), out[lo:hi], norm_eps=1e-4, gain=0.7)
    assert torch.allclose(out.double(), want, atol=1e-5) and (memory[:2] == 5).all()


@pytest.mark.parametrize("E,count,keep,k", [(12, 3, 2, 4), (8, 8, 3, 2), (6, 1, 1, 3), (9, 3, 1, 3)])
def test_choice_within_the_best_groups(E, count, keep, k):
    z = torch.randn(40, E, generator=_gen(2)) * 2
    ids, wts = moe.route_choice(z, None, k, 1.0, (count, keep), True)
    want, ww = O.choose(z.double(), k, dict(count=count, keep=keep))
    assert torch.equal(ids.long(), want) and torch.allclose(wts.double(), ww, atol=1e-6)


# ----------------------------------------------------------------------------- whole models
@pytest.mark.parametrize("name", sorted(O.CONFIGS))
def test_prompt_portions_and_decoding_agree_with_the_plain_model(name):
    raw = O.CONFIGS[name]
    t = O.random_tensors(raw, seed=3)
    toks = tokens_for(raw, 67, 7)
    want, layers = O.forward(raw, t, toks, want_layers=True)
    llm = llm_for(raw, t, "cpu", torch.float32)
    for sizes in ([67], [1], [2], [17, 3, 1, 8]):
        assert worst(run_alone(llm.engine, toks, sizes), want) < TOL, sizes
    llm.model.capture_layers = tuple(range(len(layers)))
    assert worst(run_alone(llm.engine, toks, [67]), want) < TOL
    assert len(llm.model.captured) == len(layers)
    for got, ref in zip(llm.model.captured, layers):
        assert torch.allclose(got.double(), ref, atol=3e-4, rtol=1e-4)


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


def _left(**changes):
    """Attention whose record is changed."""
    return lambda f: lambda h, w, m: f(h, w, dict(m, **{k: v(m[k]) for k, v in changes.items()}))


def _right(**changes):
    return lambda f: lambda h, w, m, eps: f(h, w, dict(m, **{k: v(m[k]) for k, v in changes.items()}), eps)


def _late_blocks(f):
    """Blocks that begin one token later."""
    def block_means(x, pool):
        return f(torch.cat([x[1:], x[-1:]]), pool)
    return block_means


def _rotate_neighbours(f):
    def rotate(x, rot, start=0):
        n = rot["dims"]
        order = torch.arange(x.shape[-1])
        order[:n] = torch.cat([torch.arange(0, n, 2), torch.arange(1, n, 2)])
        return f(x[..., order], rot, start)[..., torch.argsort(order)]
    return rotate


def _read_before_write(f):
    return lambda q, k, v, decay: torch.cat([torch.zeros_like(v[:1]), f(q[1:], k[:-1], v[:-1], decay)])


def _no_groups(f):
    return lambda s, groups: f(s, dict(count=1, keep=1))


def _groups_by_worst(f):
    def best_groups(s, groups):
        worst_member = s.view(s.shape[0], groups["count"], -1).amin(-1)
        return f(worst_member.repeat_interleave(s.shape[1] // groups["count"], 1), groups)
    return best_groups


def _spec(change):
    return lambda f: lambda h, w, spec: f(h, w, change(spec))


FAULTS = {
    "window one longer": ("tokens_seen", lambda f: lambda n, size: f(n, size + 1)),
    "window one shorter": ("tokens_seen", lambda f: lambda n, size: f(n, size - 1)),
    "blocks one token early": ("blocks_seen", lambda f: lambda n, size, pool: f(n, size - 1, pool)),
    "blocks one token late": ("blocks_seen", lambda f: lambda n, size, pool: f(n, size + 1, pool)),
    "no blocks": ("blocks_seen", lambda f: lambda n, size, pool: f(n, size + n, pool)),
    "blocks shifted": ("block_means", _late_blocks),
    "sums for means": ("block_means", lambda f: lambda x, pool: f(x, pool) * pool),
    "attention scale": ("pooled_attention", _left(scale=lambda s: s * 1.01)),
    "attention's factor": ("side_by_side", lambda f: lambda a, b, m: f(a, b, dict(m, left_scale=m["left_scale"] * 1.01))),
    "sides exchanged": ("side_by_side", lambda f: lambda a, b, m: f(b, a, m)),
    "neighbours rotated": ("rotate", _rotate_neighbours),
    "rotation base": ("retention", _right(rot=lambda r: dict(r, base=r["base"] * 1.1))),
    "positions from one": ("rotate", lambda f: lambda x, rot, start=0: f(x, dict(rot, base=rot["base"] * 1.01), start)),
    "decay": ("retain", lambda f: lambda q, k, v, decay: f(q, k, v, decay ** 1.02)),
    "read-out before the write": ("retain", _read_before_write),
    "no key scale": ("retain", lambda f: lambda q, k, v, decay: f(q, k + 1e-3, v, decay)),
    "gate": ("silu", lambda f: lambda x: f(1.01 * x)),
    "taps reversed": ("short_conv", lambda f: lambda h, taps: f(h, taps.flip(1))),
    "convolution for its input": ("short_conv", lambda f: lambda h, taps: f(h, taps) - h),
    "layer norm about zero": ("layer_norm", lambda f: lambda x, w, b, eps: O.unit_rms(x, eps) * w + b),
    "no norm bias": ("layer_norm", lambda f: lambda x, w, b, eps: f(x, w, b * 0.99, eps)),
    "mix transposed": ("spread", lambda f: lambda x, y, mix, w_out: f(x, y, mix.T, w_out)),
    "one stream for all": ("gather_streams", lambda f: lambda x, w_in: f(x[:, :1].expand_as(x), w_in)),
    "out weights": ("spread", lambda f: lambda x, y, mix, w_out: f(x, y, mix, w_out.mean().expand_as(w_out))),
    "embedding scale": ("embedding", lambda f: lambda table, tokens, scale: f(table, tokens, scale * 1.01)),
    "no groups": ("best_groups", _no_groups),
    "groups by their worst member": ("best_groups", _groups_by_worst),
    "weights not normalised": ("choose", lambda f: lambda z, top, groups: (f(z, top, groups)[0], f(z, top, groups)[1] * 0.99)),
    "limit": ("dense", _spec(lambda s: dict(s, limit=s["limit"] * 1.05))),
    "glu without the one": ("clipped_glu", lambda f: lambda g, u, limit: f(g, u - 1, limit)),
}


@pytest.mark.parametrize("what", sorted(FAULTS))
def test_a_fault_in_any_mechanism_would_show(what):
    """The comparison's resolution: mistakes planted in the plain model move its logits far beyond the tolerance the engine is
    held to."""
    raw = O.CONFIGS["mixed"]
    t, toks = O.random_tensors(raw, seed=3), tokens_for(raw, 67, 7)
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


def test_copies_of_pages_take_their_means_along():
    from mlxcel_b200.cache.kv_pool import KVPool
    pool = KVPool(ModelConfig.from_dict(O.CONFIGS["mixed"]), 4, 16, dtype=torch.float32)
    for layer in pool.layers:
        for t in (layer.k, layer.v, layer.k_mean, layer.v_mean):
            t[1] = torch.randn_like(t[1])
    pool.copy_blocks([(1, 3)])
    pool.restore_blocks([0], pool.extract_blocks([3]))
    assert all(torch.equal(t[0], t[1]) for layer in pool.layers for t in (layer.k, layer.v, layer.k_mean, layer.v_mean))


def test_loglikelihoods_and_checkpoint_round_trip(tmp_path):
    import argparse

    from safetensors.torch import load_file

    from mlxcel_b200 import cli
    from mlxcel_b200.engine import EngineConfig
    from mlxcel_b200.llm import LLM
    cli.cmd_random_init(argparse.Namespace(preset="tiny-fusolix", out=str(tmp_path), seed=3, quantize=None))
    raw, t = json.loads((tmp_path / "config.json").read_text()), load_file(str(tmp_path / "model.safetensors"))
    assert ModelConfig.from_path(tmp_path).extra == preset("tiny-fusolix").extra
    llm = LLM.from_pretrained(tmp_path, device="cpu", dtype=torch.float32,
                              engine_config=EngineConfig(num_blocks=32, block_size=16, max_batch=4, max_model_len=128))
    toks = tokens_for(raw, 60, 1)
    want = torch.log_softmax(O.forward(raw, t, toks), -1)[:-1].gather(1, torch.tensor(toks[1:])[:, None])[:, 0]
    assert torch.allclose(llm.loglikelihoods(toks).double(), want, atol=1e-4)
    with pytest.raises(ValueError):
        LLM.from_pretrained(tmp_path, device="cpu", engine_config=EngineConfig(num_blocks=32, kv_bits=8))
    fams = {f["name"]: f for f in cli.arch_catalog()["families"]}
    assert fams["fusolix"]["executor"] == fams["pamasun"]["executor"] and fams["fusolix"]["checked_against"] == fams["pamasun"]["checked_against"]


def test_a_missing_tensor_is_named(tmp_path):
    from safetensors.torch import save_file

    from mlxcel_b200.llm import LLM
    raw = O.CONFIGS["odd"]
    t = {k: v.to(torch.bfloat16).contiguous() for k, v in O.random_tensors(raw, 0).items() if k != "l1.hc2.mix"}
    (tmp_path / "config.json").write_text(json.dumps(raw))
    save_file(t, str(tmp_path / "model.safetensors"))
    with pytest.raises(KeyError, match="l1.hc2.mix"):
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
