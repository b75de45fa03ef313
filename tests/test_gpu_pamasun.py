"""Pamasun kernels and engine on a GPU against the plain model (``oracle_pamasun``): every mechanism alone in
fp32 and bf16 over sizes the fast kernels cover and sizes they do not, then whole models."""
import pytest
import torch

import oracle_pamasun as O
from mlxcel_b200 import ops
from mlxcel_b200.engine import SamplingParams
from mlxcel_b200.ops import KVLayer, stream
from design_runs import bf16_ok, interleave, llm_for, oracle_greedy, run_alone, run_mixed, tokens_for, worst

pytestmark = pytest.mark.gpu
DEV = "cuda"
F32, BF16 = torch.float32, torch.bfloat16


def _gen(seed):
    return torch.Generator().manual_seed(seed)


def _close(got, want, dtype, f32=2e-5, bf16=1.5e-2):
    tol = f32 if dtype == F32 else bf16
    got, want = got.double().cpu(), want.double()
    err = (got - want).abs() / (want.abs() + want.pow(2).mean().sqrt())
    assert torch.isfinite(got).all() and err.max() < tol, float(err.max())


# ----------------------------------------------------------------------------- linear
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("M,N,K", [(1, 64, 64), (3, 101, 75), (65, 130, 50), (200, 67, 256), (7, 264, 12)])
def test_linear_of_any_size(M, N, K, dtype):
    g = _gen(M + N)
    x, w = torch.randn(M, K, generator=g).to(dtype), (torch.randn(N, K, generator=g) * K ** -0.5).to(dtype)
    want = x.double() @ w.double().T
    _close(ops.linear(x.to(DEV), w.to(DEV)), want, dtype)
    y = ops.linear(x.to(DEV), w.to(DEV), out_fp32=True)
    assert y.dtype == F32
    _close(y, want, F32)                       # fp32 accumulation whatever the operands


# ----------------------------------------------------------------------------- rows
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("dim", [64, 75, 96, 1000, 1030, 4096, 6001])
def test_stream_rows(dim, dtype):
    g, n, eps = _gen(dim), 5, 1e-5
    h, y = torch.randn(n, dim, generator=g) * 3, torch.randn(n, dim, generator=g).to(dtype)
    w1, w2, ls = 0.3 * torch.randn(dim, generator=g), 0.3 * torch.randn(dim, generator=g), torch.rand(dim, generator=g)
    d = lambda t: None if t is None else t.double()                                     # noqa: E731
    for scale in (ls, None):
        hd = h.to(DEV)
        x = stream.stream_norm(hd, y.to(DEV), w1.to(DEV), None if scale is None else scale.to(DEV), w2.to(DEV), eps, 1.0)
        want = d(h) + O.around_zero_norm(d(y), d(w1), eps) * (1.0 if scale is None else d(scale))
        _close(hd, want, F32)
        _close(x, O.around_zero_norm(want, d(w2), eps), dtype)
        assert x.dtype == dtype
    rows = torch.tensor([3, 0, 3], dtype=torch.int32)
    x = stream.stream_norm(h.to(DEV), None, None, None, w2.to(DEV), eps, 1.0, dtype=dtype, rows=rows.to(DEV))
    _close(x, O.around_zero_norm(d(h)[[3, 0, 3]], d(w2), eps), dtype)
    table, ids = torch.randn(11, dim, generator=g).to(dtype), torch.tensor([10, 0, 7], dtype=torch.int32)
    hh, x = stream.embed_stream(ids.to(DEV), table.to(DEV), 7.25, w2.to(DEV), eps, 1.0)
    _close(hh, d(table)[ids.long()] * 7.25, F32)
    _close(x, O.around_zero_norm(d(table)[ids.long()] * 7.25, d(w2), eps), dtype)
    coef = torch.tensor([0.8, -0.5, 0.4, 0.3])
    _close(stream.polynorm(y.to(DEV), coef.to(DEV), eps), O.polynorm(d(y), d(coef), eps), dtype)


# ----------------------------------------------------------------------------- attention
GEOMETRIES = [(4, 2, 64, 32), (6, 2, 48, 40), (5, 5, 128, 64), (8, 1, 64, 128), (12, 4, 96, 96), (2, 2, 8, 8),   # tensor-core kernels
              (3, 1, 36, 20), (2, 2, 160, 72), (20, 1, 32, 32)]                                             # SIMT kernel in bf16 too


def _attention_case(geo, lens, qlens, dtype, seed):
    """Pool with the sequences' blocks scattered, rows of q | k | v | gate as a projection leaves them; queries
    and keys as they come out of the norms."""
    Hq, Hkv, Dk, Dv = geo
    g, bs = _gen(seed), 16
    need = [(n + bs - 1) // bs for n in lens]
    perm = torch.randperm(sum(need) + 3, generator=g).tolist()
    tables = torch.zeros(len(lens), max(need) + 1, dtype=torch.int32)
    kp, vp = torch.randn(sum(need) + 3, Hkv, bs, Dk, generator=g), torch.randn(sum(need) + 3, Hkv, bs, Dv, generator=g)
    ks, vs = [], []
    for s, n in enumerate(lens):
        blocks = [perm.pop() for _ in range(need[s])]
        tables[s, : need[s]] = torch.tensor(blocks)
        ks.append(torch.randn(n, Hkv, Dk, generator=g))
        vs.append(torch.randn(n, Hkv, Dv, generator=g))
    T = sum(qlens)
    q, gate = torch.randn(T, Hq, Dk, generator=g), torch.randn(T, Hq * Dv, generator=g)
    # single keys that stand out, next to page and tile borders and far away: key n answers query row r
    r = 0
    for s, (n, ql) in enumerate(zip(lens, qlens)):
        spots = [p for p in (0, 1, 15, 16, 17, 31, 32, 63, 64, 127, 128, 129, n - ql, n - 2, n - 1) if 0 <= p < n]
        for i in range(ql):
            p = spots[(i * 7 + s) % len(spots)]
            if p <= n - ql + i:
                for h in range(Hq):
                    q[r + i, h] = 0.3 * q[r + i, h] + 1.2 * ks[s][p, h // (Hq // Hkv)]
        r += ql
    rd = lambda t: t.to(dtype)                                                           # noqa: E731
    ks, vs, q, gate = [rd(k) for k in ks], [rd(v) for v in vs], rd(q), rd(gate)
    for s, n in enumerate(lens):
        for t in range(n):
            kp[tables[s, t // bs], :, t % bs] = ks[s][t].float()
            vp[tables[s, t // bs], :, t % bs] = vs[s][t].float()
    kv = KVLayer(rd(kp).to(DEV), rd(vp).to(DEV), None, None, bs)
    ld = -(-(Hq * Dk + Hq * Dv) // 8) * 8
    row = torch.zeros(T, ld, dtype=dtype)
    row[:, : Hq * Dk], row[:, Hq * Dk: Hq * Dk + Hq * Dv] = q.reshape(T, -1), gate
    return ks, vs, q, gate, kv, tables, row


def _attention_plain(ks, vs, q, gate, lens, qlens, geo, scale, r1, r2, sinks, window):
    Hq, Hkv, Dk, Dv = geo
    out, r = [], 0
    for s, (n, ql) in enumerate(zip(lens, qlens)):
        k, v = ks[s].double(), vs[s].double()
        i = torch.arange(n - ql, n)
        d = i[:, None] - torch.arange(n)[None]
        res = torch.zeros(ql, Hq, Dv, dtype=torch.float64)
        for h in range(Hq):
            sc = q[r:r + ql, h].double() @ k[:, h // (Hq // Hkv)].T * scale
            if r1 is not None:
                sc = sc - O.distance_bias(r1.double(), r2.double(), n)[h][n - ql:]
            sc = sc.masked_fill((d < 0) | ((d >= window) if window else False), float("-inf"))
            p = O.sink_softmax(sc, sinks[h].double()) if sinks is not None else torch.softmax(sc, -1)
            res[:, h] = p @ v[:, h // (Hq // Hkv)]
        res = res.reshape(ql, Hq * Dv)
        out.append(res if gate is None else res * torch.sigmoid(gate[r:r + ql].double()))
        r += ql
    return torch.cat(out)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("geo", GEOMETRIES)
def test_paged_attention(geo, dtype):
    Hq, Hkv, Dk, Dv = geo
    g = _gen(Hq * Dk)
    r1, r2, sinks = 0.1 + torch.rand(Hq, generator=g), 0.05 + torch.rand(Hq, generator=g), 2 * torch.randn(Hq, generator=g)
    scale = Dk ** -0.5 * 1.7
    for lens, qlens in (([1, 16, 17, 33, 300, 129], [1] * 6), ([5, 150, 290, 64, 3], [5, 150, 33, 2, 1])):
        ks, vs, q, gate, kv, tables, row = _attention_case(geo, lens, qlens, dtype, Dk + Dv)
        T = sum(qlens)
        cu = torch.tensor([0] + torch.tensor(qlens).cumsum(0).tolist(), dtype=torch.int32)
        rd, d = row.to(DEV), lambda t: t.to(DEV)
        for window, full in ((0, True), (40, True), (0, False)):
            out = torch.full((T, Hq * Dv), 7.0, dtype=dtype, device=DEV)
            stream.paged_attention(
                rd[:, : Hq * Dk], kv, d(tables), d(torch.tensor(lens, dtype=torch.int32)), None if max(qlens) == 1 else d(cu), out,
                Hq=Hq, Hkv=Hkv, Dk=Dk, Dv=Dv, scale=scale, max_q_len=max(qlens), max_len=max(lens), window=window,
                sinks=d(sinks) if full else None, dist_bias=(d(r1), d(r2)) if full else None,
                gate=rd[:, Hq * Dk: Hq * Dk + Hq * Dv] if full else None)
            want = _attention_plain(ks, vs, q, gate if full else None, lens, qlens, geo, scale, r1 if full else None,
                                    r2 if full else None, sinks if full else None, window)
            _close(out, want, dtype)


def test_decode_splits_of_long_contexts_merge_sink_bias_and_gate_once():
    """Few rows over long contexts: several KV splits per (row, head), merged by the last CTA; then a batch with
    more rows, whose arrival counters must not meet the first call's partial sums."""
    geo = (8, 2, 64, 64)
    g = _gen(5)
    r1, r2, sinks = 0.1 + torch.rand(8, generator=g), 0.02 + 0.1 * torch.rand(8, generator=g), 2 * torch.randn(8, generator=g)
    for lens in ([2100], [1500, 900, 2048, 777], [1100] * 40):
        ks, vs, q, gate, kv, tables, row = _attention_case(geo, lens, [1] * len(lens), BF16, len(lens))
        out, rd = torch.empty(len(lens), 512, dtype=BF16, device=DEV), row.to(DEV)
        stream.paged_attention(rd[:, :512], kv, tables.to(DEV), torch.tensor(lens, dtype=torch.int32, device=DEV), None, out,
                               Hq=8, Hkv=2, Dk=64, Dv=64, scale=0.2, max_q_len=1, max_len=max(lens), sinks=sinks.to(DEV),
                               dist_bias=(r1.to(DEV), r2.to(DEV)), gate=rd[:, 512:1024])
        _close(out, _attention_plain(ks, vs, q, gate, lens, [1] * len(lens), geo, 0.2, r1, r2, sinks, 0), BF16)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("geo", [(6, 2, 48, 24), (3, 1, 20, 13), (4, 4, 128, 96), (2, 1, 160, 200)])
def test_qk_norm_and_append(geo, dtype):
    Hq, Hkv, Dk, Dv = geo
    g, T = _gen(Dk), 9
    n = Hq * Dk + Hkv * (Dk + Dv)
    row = torch.randn(T, -(-n // 8) * 8, generator=g).to(dtype)
    qw, kw = torch.randn(Dk, generator=g), torch.randn(Dk, generator=g)
    slots = torch.tensor([5, 6, 40, -1, 0, 47, 16, 15, 31], dtype=torch.int32)
    kv = KVLayer(torch.zeros(3, Hkv, 16, Dk, dtype=dtype, device=DEV), torch.zeros(3, Hkv, 16, Dv, dtype=dtype, device=DEV), None, None, 16)
    got = row.to(DEV)
    stream.qk_norm_append(got, slots.to(DEV), kv, Hq=Hq, Hkv=Hkv, Dk=Dk, Dv=Dv, q_norm=qw.to(DEV), k_norm=kw.to(DEV), eps=1e-5)
    r = row.double()
    q = O.rms(r[:, : Hq * Dk].view(T, Hq, Dk), 1e-5) * qw.double()
    k = O.rms(r[:, Hq * Dk: Hq * Dk + Hkv * Dk].view(T, Hkv, Dk), 1e-5) * kw.double()
    v = r[:, Hq * Dk + Hkv * Dk: n].view(T, Hkv, Dv)
    _close(got[:, : Hq * Dk], q.reshape(T, -1), dtype)
    assert torch.equal(got[:, Hq * Dk:].cpu(), row[:, Hq * Dk:])
    used = torch.zeros(48, dtype=torch.bool)
    for t, s in enumerate(slots.tolist()):
        if s >= 0:
            used[s] = True
            _close(kv.k[s // 16, :, s % 16], k[t], dtype)
            assert torch.equal(kv.v[s // 16, :, s % 16].cpu().double(), v[t])
    assert not kv.k.cpu().permute(0, 2, 1, 3).reshape(48, -1)[~used].any()


# ----------------------------------------------------------------------------- delta rule
@pytest.mark.parametrize("force_any", [False, True])
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("H,D,R", [(2, 48, 16), (3, 40, 6), (1, 128, 12), (4, 64, 7), (2, 20, 5), (2, 132, 8), (2, 17, 3), (1, 4, 1)])
def test_delta_rule(H, D, R, dtype, force_any):
    g, HD, eps = _gen(D + R), H * D, 1e-5
    pieces = [1, 1, 1, 1, 33, 2, 16, 100, 17]                       # decode rows, then portions
    n_short, slots = 4, torch.tensor([6, 2, -1, 9, 0, 5, 1, 8, 3], dtype=torch.int32)
    reset = torch.tensor([0, 1, 0, 0, 1, 0, 0, 1, 0], dtype=torch.int32)
    cu = torch.tensor([0] + torch.tensor(pieces).cumsum(0).tolist(), dtype=torch.int32)
    T = int(cu[-1])
    ld = -(-(5 * HD + R) // 8) * 8
    proj = torch.randn(T, ld, generator=g).to(dtype)
    w2 = (torch.randn(HD, R, generator=g) * R ** -0.5).to(dtype)
    w0, ab, nw = -3 + 3 * torch.randn(HD, generator=g), torch.randn(HD, generator=g), 1 + 0.3 * torch.randn(HD, generator=g)
    state = torch.randn(10, H, D, D, generator=g)
    p = proj.double()
    z = torch.tanh(p[:, 5 * HD:5 * HD + R]) @ w2.double().T + w0
    decay = torch.exp(-torch.tensor(-0.5, dtype=torch.float64).exp() * torch.sigmoid(z)).view(T, H, D)
    r, k, v, gt, a = (p[:, i * HD:(i + 1) * HD].reshape(T, H, D) for i in range(5))
    a = torch.sigmoid(a + ab.double().view(H, D))
    want, want_state = torch.zeros(T, HD, dtype=torch.float64), state.double().clone()
    for j in range(len(pieces)):
        if slots[j] < 0:
            continue
        s = slice(int(cu[j]), int(cu[j + 1]))
        o, last = O.delta_recurrence(r[s], k[s], v[s], decay[s], a[s], None if reset[j] else state[slots[j]].double())
        want[s] = O.rms(o, eps).reshape(-1, HD) * nw.double() * torch.sigmoid(gt[s].reshape(-1, HD))
        want_state[slots[j]] = last
    d = lambda t: t.to(DEV)                                                              # noqa: E731
    st = d(state)
    got = stream.delta_rule(d(proj), tuple(i * HD for i in range(6)), d(w2), d(w0), d(ab), d(nw), st, d(slots), d(cu), d(reset),
                            D=D, norm_eps=eps, n_short=n_short, force_any=force_any)
    _close(st, want_state, F32, f32=5e-5)               # the state is fp32 whatever the activations are
    for j in range(len(pieces)):                        # (per piece, so that a short one's errors are not averaged away)
        s = slice(int(cu[j]), int(cu[j + 1]))
        if slots[j] >= 0:
            _close(got[s], want[s], dtype, f32=2e-4)
        else:
            assert not got[s].any()


# ----------------------------------------------------------------------------- models
@pytest.mark.parametrize("name", sorted(O.CONFIGS))
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_prompts_portions_and_decoding(name, dtype):
    raw = O.CONFIGS[name]
    t = O.random_tensors(raw, seed=3)
    toks = tokens_for(raw, 150, 7)
    want, layers = O.forward(raw, t, toks, want_layers=True)
    llm = llm_for(raw, t, DEV, dtype)
    whole = run_alone(llm.engine, toks, [150])
    ok = (lambda got: worst(got, want) < 1e-4) if dtype == F32 else (lambda got: bf16_ok(O, raw, t, toks, got, want))   # noqa: E731
    assert ok(whole)
    for sizes in ([1], [130, 1], [2], [17, 3, 1, 64, 16]):
        assert ok(run_alone(llm.engine, toks, sizes)), sizes
    if dtype == F32:
        llm.model.capture_layers = tuple(range(len(layers)))
        run_alone(llm.engine, toks, [150])
        for got, ref in zip(llm.model.captured, layers):
            assert (got.double().cpu() - ref).abs().max() < 1e-3 * ref.abs().max()
    assert llm.engine.stats["graph_replays"] > 150 and ops._lib.read_status(torch.device(DEV, 0)) == 0


@pytest.mark.parametrize("name", ["mixed", "odd", "wide"])
def test_mixed_batches_on_reused_pages_and_slots(name):
    raw = O.CONFIGS[name]
    t = O.random_tensors(raw, seed=5)
    lengths = [170, 7, 133, 1, 40, 18, 2, 141, 90]
    seqs = [tokens_for(raw, n, 20 + i) for i, n in enumerate(lengths)]
    sched = interleave(lengths, [[64, 2, 1, 1, 31], [1], [5, 1, 1, 129], [3, 2]])
    wants = [O.forward(raw, t, s) for s in seqs]
    for dtype in (F32, BF16):
        llm = llm_for(raw, t, DEV, dtype, num_blocks=34, max_model_len=544)
        for s, got, want in zip(seqs, run_mixed(llm.engine, seqs, sched), wants):
            assert worst(got, want) < 1e-4 if dtype == F32 else bf16_ok(O, raw, t, s, got, want)
        assert llm.engine.bm.num_free == 34 and len(llm.model.ssm.free) == 4


def test_long_decoding_keeps_state_and_cache():
    raw = O.CONFIGS["mixed"]
    t = O.random_tensors(raw, seed=8)
    toks = tokens_for(raw, 700, 1)
    want = O.forward(raw, t, toks)
    for dtype in (F32, BF16):
        got = run_alone(llm_for(raw, t, DEV, dtype).engine, toks, [40] + [1] * 660)
        assert worst(got, want) < 1e-4 if dtype == F32 else bf16_ok(O, raw, t, toks, got, want)


def test_greedy_generation_through_the_scheduler():
    raw = O.CONFIGS["mixed"]
    t = O.random_tensors(raw, seed=9)
    prompts = [tokens_for(raw, n, 40 + n) for n in (23, 1, 9, 30, 4)]
    want = [oracle_greedy(O, raw, t, p, 12) for p in prompts]
    sp = SamplingParams(max_tokens=12, temperature=0.0, ignore_eos=True)
    # decode graphs with the lookahead pipeline; without graphs; queueing, prompt portions and preemption
    for kw in (dict(max_batch=8, state_slots=8), dict(cuda_graphs=False), dict(max_batch=2, max_num_batched_tokens=8, num_blocks=6)):
        llm = llm_for(raw, t, DEV, F32, **kw)
        outs = llm.generate(prompt_token_ids=prompts, sampling_params=sp)
        assert [s.output for s in outs] == want, kw
        assert not llm.model.ssm.slot_of and llm.engine.bm.num_free == llm.engine.ecfg.num_blocks
    llm = llm_for(raw, t, DEV, BF16)
    outs = llm.generate(prompt_token_ids=prompts, sampling_params=sp)
    assert sum(s.output[0] == w[0] for s, w in zip(outs, want)) >= 4
