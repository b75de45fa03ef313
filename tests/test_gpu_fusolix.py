"""Fusolix kernels and engine on a GPU against the plain model (``oracle_fusolix``): every mechanism alone in fp32 and bf16
over sizes the fast kernels cover and sizes they do not, then whole models."""
import pytest
import torch

import oracle_fusolix as O
from design_runs import (assert_close, bf16_ok, bounds, fill_pages, interleave, llm_for, oracle_greedy, paged_tables, run_alone, run_mixed,
                         tokens_for, worst)
from mlxcel_b200.engine import SamplingParams
from mlxcel_b200.ops import KVLayer, _lib, block_means, moe, retention, stream, streams
from mlxcel_b200.ops.reference import rope_inv_freq

pytestmark = pytest.mark.gpu
DEV = "cuda"
F32, BF16 = torch.float32, torch.bfloat16


def _gen(seed):
    return torch.Generator().manual_seed(seed)


def _i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


def _status_ok():
    return _lib.read_status(torch.device(DEV, 0)) == 0


# ----------------------------------------------------------------------------- streams
def _around(S, H, K, g, device):
    n = lambda *s: torch.randn(*s, generator=g)      # noqa: E731
    parts = dict(w_in=n(S), w_out=n(S), mix=n(S, S), norm_w=n(H), norm_b=n(H), taps=n(K, H) * K ** -0.5, bias=n(H))
    return parts, streams.Sublayer(**{k: v.to(device) for k, v in parts.items()})


def _conv(n, taps):
    return O.short_conv(n, taps.t())


STREAMS = [  # streams, width, taps
    (4, 64, 3), (1, 75, 1), (3, 1000, 4), (4, 4096, 4), (2, 2048, 2), (5, 33, 6), (16, 256, 3), (8, 1152, 1), (4, 9000, 5), (2, 4099, 3), (4, 1280, 20)]


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("S,H,K", STREAMS)
def test_streams_through_portions_and_single_tokens(S, H, K, dtype):
    """Steps over the same slots: portions of every kind, then single tokens (a padding row among them) beside portions, then
    single tokens alone; a slot that starts anew. Each step: streams, next input, its convolution; results of a row or of experts."""
    g = _gen(S + H)
    n = lambda *s: torch.randn(*s, generator=g)      # noqa: E731
    (da, a), (db, b) = _around(S, H, K, g, DEV), _around(S, H, K, g, DEV)
    da, db = ({k: v.double() for k, v in t.items()} for t in (da, db))
    steps = [[(0, 70), (3, 1), (1, 2), (5, 35)], [(0, 1), (None, 1), (3, 1), (1, 33), (5, 3), (2, 17)], [(5, 1), (0, 1), (2, 1)], [(1, 40), (3, 2)]]
    decode = [0, 3, 3, 0]
    total = {s: sum(c for st in steps for q, c in st if q == s) for s in (0, 1, 2, 3, 5)}
    seq = {s: (n(m, S, H), n(m, H).to(dtype)) for s, m in total.items()}
    new = {s: O.spread(xs.double(), y.double() + da["bias"], da["mix"], da["w_out"]) for s, (xs, y) in seq.items()}
    inp = {s: O.layer_norm(O.gather_streams(x, db["w_in"]), db["norm_w"], db["norm_b"], 1e-5) for s, x in new.items()}
    want = {s: _conv(x, db["taps"]) for s, x in inp.items()}
    tail = torch.full((6, K - 1, H), 7.0, device=DEV)                     # (slots held something before)
    at = {s: 0 for s in seq}
    for i, (st, nd) in enumerate(zip(steps, decode)):
        xs, ys, ex, en, reset = [], [], [], [], []
        for s, c in st:
            if s is None:
                xs.append(n(c, S, H)), ys.append(n(c, H).to(dtype)), ex.append(None), en.append(None), reset.append(0)
                continue
            sl = slice(at[s], at[s] + c)
            xs.append(seq[s][0][sl]), ys.append(seq[s][1][sl]), ex.append(want[s][sl]), en.append(new[s][sl]), reset.append(int(at[s] == 0))
            at[s] += c
        sizes = [c for _, c in st]
        pieces = (_i32([-1 if s is None else s for s, _ in st]), _i32(bounds(sizes)), _i32(reset), nd, max(sizes))
        x_in, y_in = torch.cat(xs).to(DEV), torch.cat(ys).to(DEV)
        total_sum = streams.sum_streams(x_in, a, y_in, None, dtype)
        x = streams.mix_streams(x_in, a, y_in, None, b, 1e-5, dtype, tail, pieces)
        for got, got_new, got_sum, ref, ref_new in zip(x.split(sizes), x_in.split(sizes), total_sum.split(sizes), ex, en):
            if ref is not None:
                assert_close(got, ref, dtype)
                assert_close(got_new, ref_new, F32)
                assert_close(got_sum, ref_new.sum(1), F32)
    if K > 1:
        assert (tail[4] == 7).all()
        for s, m in inp.items():
            have = m[-(K - 1):]
            assert_close(tail[s][K - 1 - have.shape[0]:], have, F32)
            assert not tail[s][:K - 1 - have.shape[0]].any()


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_streams_start_from_the_embedding_and_take_up_experts(dtype):
    g, S, H, K, T, k = _gen(5), 4, 136, 3, 9, 3
    n = lambda *s: torch.randn(*s, generator=g)      # noqa: E731
    (da, a), (db, b) = _around(S, H, K, g, DEV), _around(S, H, K, g, DEV)
    da, db = ({k: v.double() for k, v in t.items()} for t in (da, db))
    table, ids = n(11, H).to(dtype), [3, 0, 10, 3, 1, 7, 2, 9, 9]
    pieces, tail = (_i32([1]), _i32([0, T]), _i32([1]), 0, T), torch.zeros(2, K - 1, H, device=DEV)
    xs, x = streams.embed_streams(_i32(ids), table.to(DEV), 2.5, S, b, 1e-5, tail, pieces)
    e = O.embedding(table.double(), ids, 2.5)[:, None].repeat(1, S, 1)
    norm = lambda u: O.layer_norm(O.gather_streams(u, db["w_in"]), db["norm_w"], db["norm_b"], 1e-5)      # noqa: E731
    assert_close(xs, e, F32)
    assert_close(x, _conv(norm(e), db["taps"]), dtype)
    rows, wts, perm = n(T * k, H).to(dtype), torch.rand(T, k, generator=g), torch.randperm(T * k, generator=g)
    m = moe.MoeRows(rows.to(DEV), x, torch.zeros(T, k, dtype=torch.int32, device=DEV), perm.int().to(DEV), wts.to(DEV), 5)
    y = (rows.double()[perm].view(T, k, H) * wts.double()[..., None]).sum(1)
    new = O.spread(e, y + da["bias"], da["mix"], da["w_out"])
    assert_close(streams.sum_streams(xs, a, None, m, dtype), new.sum(1), F32)
    x = streams.mix_streams(xs, a, None, m, b, 1e-5, dtype, tail, pieces)
    assert_close(xs, new, F32)
    assert_close(x, _conv(norm(new), db["taps"]), dtype)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("H", [64, 75, 4096])
def test_layer_norm_of_chosen_rows(H, dtype):
    g = _gen(H)
    h, w, b, rows = torch.randn(9, H, generator=g) + 5, torch.randn(H, generator=g), torch.randn(H, generator=g), [8, 0, 3]
    for pick in (None, rows):
        got = streams.layer_norm(h.to(DEV), w.to(DEV), b.to(DEV), 1e-3, dtype, None if pick is None else _i32(pick))
        assert_close(got, O.layer_norm((h if pick is None else h[pick]).double(), w.double(), b.double(), 1e-3), dtype)


# ----------------------------------------------------------------------------- experts
@pytest.mark.parametrize("T,E,count,keep,k", [(1, 4, 2, 1, 1), (70, 12, 3, 2, 3), (9, 128, 8, 3, 8), (200, 512, 64, 5, 16), (33, 7, 7, 4, 4),
                                              (40, 6, 1, 1, 3), (17, 500, 250, 100, 7), (5, 600, 3, 1, 2)])
def test_choice_within_the_best_groups(T, E, count, keep, k):
    z = torch.randn(T, E + 3, generator=_gen(T + E)) * 3
    z[0, 0] = 60.0                                                        # one expert takes all of the softmax
    z[0, 1:E] = z[0, 1:E].clamp(max=20)
    want, ww = O.choose(z[:, :E].double(), k, dict(count=count, keep=keep))
    ids, wts = moe.route_choice(z.to(DEV)[:, :E], None, k, 1.0, (count, keep), True)
    full = lambda i, w: torch.zeros(T, E, dtype=torch.float64).scatter_(1, i.cpu().long(), w.cpu().double())      # noqa: E731
    assert ids.dtype == torch.int32 and all(len(set(r)) == k for r in ids.tolist())
    assert torch.allclose(full(ids, wts), full(want, ww), atol=2e-6)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("T,H,I,E,k", [(1, 64, 64, 4, 2), (70, 96, 40, 6, 3), (300, 128, 96, 12, 4), (9, 75, 33, 3, 1), (130, 64, 21, 7, 5)])
def test_plain_gated_experts(T, H, I, E, k, dtype):
    g = _gen(T + I)
    n = lambda *s: torch.randn(*s, generator=g)      # noqa: E731
    x, w = n(T, H).to(dtype), {"router": (n(E, H) * H ** -0.5 * 4).to(dtype)}
    for e in range(E):
        w.update({f"e{e}.gate": (n(I, H) * H ** -0.5 * 2).to(dtype), f"e{e}.up": (n(I, H) * H ** -0.5).to(dtype), f"e{e}.down": (n(H, I) * I ** -0.5).to(dtype)})
    groups = dict(count=1, keep=1)
    want = O.experts(x.double(), {name: t.double() for name, t in w.items()}, O.moe(I, E, 1, 1, k))
    gu = torch.stack([torch.cat([w[f"e{e}.gate"], w[f"e{e}.up"]]) for e in range(E)]).to(DEV)
    dn = torch.stack([w[f"e{e}.down"] for e in range(E)]).to(DEV)
    ids, wts = O.choose(x.double() @ w["router"].double().T, k, groups)
    for force in (False, True):
        m = moe.expert_rows(x.to(DEV), ids.int().to(DEV), wts.float().to(DEV), gu, dn, 1.0, 0.0, force_any=force, act="silu")
        got = (m.y[m.inv.long()].view(T, k, H).float() * m.wts[..., None]).sum(1)
        assert_close(got, want, dtype, bf16=2.5e-2)
    assert _status_ok()


# ----------------------------------------------------------------------------- attention with block means
MEANS = [  # heads, key heads, key width, value width, window, block, page
    (12, 2, 64, 64, 50, 8, 16), (6, 2, 32, 40, 18, 4, 16), (16, 1, 128, 128, 130, 16, 16), (4, 4, 40, 72, 21, 10, 16), (3, 3, 9, 11, 7, 3, 8),
    (8, 4, 128, 64, 33, 32, 16), (2, 1, 64, 128, 1, 1, 16), (5, 1, 24, 16, 27, 23, 32), (4, 2, 96, 48, 200, 5, 16), (8, 8, 8, 8, 2, 2, 16),
    (2, 2, 56, 24, 16, 16, 8), (20, 1, 32, 32, 12, 4, 16)]


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("Hq,Hkv,D,Dv,size,pool,bs", MEANS)
def test_window_and_block_means(Hq, Hkv, D, Dv, size, pool, bs, dtype):
    """Sequences appended in portions that start and end anywhere, then single tokens; the last call's rows are compared. Keys at
    block edges and windows' ends outscore the rest."""
    g = _gen(Hq + D + pool)
    calls = [([300, 40, 17, 700, 3], False), ([1, 1, 1, 1, 1], True), ([100, 2, 21, 33, 64], False), ([1, 1, 1, 1, 1], True)]
    lens = [sum(c[s] for c, _ in calls) for s in range(5)]
    tab, blocks = paged_tables(lens, bs)
    per, fill = -(-bs // pool), lambda w, r: torch.full((blocks, Hkv, r, w), 3.0, dtype=dtype, device=DEV)     # noqa: E731
    kv = KVLayer(fill(D, bs), fill(Dv, bs), None, None, bs, 16, fill(D, per), fill(Dv, per), pool)
    rows = []
    for s, n in enumerate(lens):
        k, v, q = torch.randn(n, Hkv, D, generator=g), torch.randn(n, Hkv, Dv, generator=g), torch.randn(n, Hq, D, generator=g) * 0.3 + 0.5
        for p in {c for e in range(0, n, pool * 7) for c in (e - 1, e, e + pool - 1)} | {n - size - 1, n - size, n - size + 1}:
            if 0 <= p < n:
                k[p] = k[p].abs() + 1.5
        rows.append(torch.cat([q.reshape(n, -1), k.reshape(n, -1), v.reshape(n, -1), torch.randn(n, -(Hq * D + Hkv * (D + Dv)) % 8, generator=g)], 1).to(dtype))
    at, tabd = [0] * 5, tab.to(DEV)
    for counts, single in calls:
        part = torch.cat([rows[s][at[s]:at[s] + c] for s, c in enumerate(counts)]).to(DEV)
        pos = torch.cat([torch.arange(at[s], at[s] + c) for s, c in enumerate(counts)])
        seq = torch.cat([torch.full((c,), s) for s, c in enumerate(counts)])
        slots = tab[seq, pos // bs] * bs + pos % bs
        at = [a + c for a, c in zip(at, counts)]
        cu = None if single else _i32(bounds(counts))
        ld = _i32(at)
        geo = dict(Hq=Hq, Hkv=Hkv, Dk=D, Dv=Dv)
        block_means.append(part, pos.int().to(DEV), slots.int().to(DEV), kv, tabd, cu, **geo)
        b = type("B", (), dict(pf_cu_q_host=None, pf_starts=None, pf_context_lens=ld))()
        means = (None, 0) if single else block_means.portion_means(b, size, pool)
        wide = torch.full((part.shape[0], -(-Hq * Dv // 8) * 8 + 8), 9.0, dtype=dtype, device=DEV)
        for force in (False, True):
            out = wide[:, :Hq * Dv]
            stream.paged_attention(part[:, :Hq * D], kv, tabd, ld, cu, out, scale=D ** -0.5 * 1.3, max_q_len=max(counts), max_len=max(at), window=size,
                                   means=means, gain=0.6, force_any=force, **geo)
            r0 = 0
            for s, c in enumerate(counts):
                n = at[s]
                d = rows[s][:n].double()
                q, k = d[n - c:, :Hq * D].view(c, Hq, D), d[:, Hq * D:(Hq + Hkv) * D].view(n, Hkv, D)
                v = d[:, (Hq + Hkv) * D:(Hq + Hkv) * D + Hkv * Dv].view(n, Hkv, Dv)
                km, vm = (O.block_means(t, pool).to(dtype).double() for t in (k, v))
                keys, vals = torch.cat([k, km]), torch.cat([v, vm])
                seen = torch.cat([O.tokens_seen(n, size), O.blocks_seen(n, size, pool)], 1)[n - c:]
                want = torch.stack([O.attend(q[:, a] @ keys[:, a // (Hq // Hkv)].T * (D ** -0.5 * 1.3), seen, vals[:, a // (Hq // Hkv)])
                                    for a in range(Hq)], 1)
                assert_close(out[r0:r0 + c], want.reshape(c, -1) * 0.6, dtype, f32=5e-5)
                r0 += c
            assert (wide[:, Hq * Dv:] == 9).all()
    assert _status_ok()


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_means_are_those_of_the_pool_and_padding_rows_append_nothing(dtype):
    P, bs, D, Dv, n = 5, 16, 8, 16, 48
    tab, blocks = paged_tables([n], bs)
    kv = KVLayer(*(torch.full((blocks, 1, r, w), 3.0, dtype=dtype, device=DEV) for r, w in ((bs, D), (bs, Dv))), None, None, bs, 16,
                 *(torch.full((blocks, 1, 4, w), 3.0, dtype=dtype, device=DEV) for w in (D, Dv)), P)
    row = torch.randn(n, D + D + Dv, generator=_gen(1)).to(dtype).to(DEV)
    pos = torch.arange(n)
    slots = (tab[0, pos // bs] * bs + pos % bs).int()
    geo = dict(Hq=1, Hkv=1, Dk=D, Dv=Dv)
    block_means.append(row, pos.int().to(DEV), torch.full((n,), -1, dtype=torch.int32, device=DEV), kv, tab.to(DEV), _i32([0, n]), **geo)
    assert all((t == 3).all() for t in (kv.k, kv.v, kv.k_mean, kv.v_mean))
    block_means.append(row, pos.int().to(DEV), slots.to(DEV), kv, tab.to(DEV), _i32([0, n]), **geo)
    k, v = block_means.gather(kv, tab.to(DEV), _i32([0, n // P]), n // P)
    for got, x in ((k, row[:, D:2 * D]), (v, row[:, 2 * D:])):
        assert_close(got[:, 0], O.block_means(x.double().cpu()[:, None], P)[:, 0], dtype, bf16=8e-3)


# ----------------------------------------------------------------------------- retention
def _oracle_retention(p, H, D, V, rot, decay, eps, gain):
    q, k = (O.rotate(p[:, i * H * D:(i + 1) * H * D].view(-1, H, D), rot) for i in (0, 1))
    v, gate = p[:, 2 * H * D:2 * H * D + H * V].view(-1, H, V), p[:, 2 * H * D + H * V:2 * H * (D + V)]
    return O.unit_rms(O.retain(q, k * D ** -0.5, v, decay), eps).reshape(-1, H * V) * O.silu(gate) * gain


RETENTION = [  # heads, key width, value width, rotated
    (4, 64, 32, 64), (2, 128, 128, 128), (3, 10, 7, 6), (1, 34, 13, 2), (5, 40, 24, 20), (2, 16, 64, 8), (8, 8, 8, 8), (1, 256, 64, 128), (2, 200, 40, 100),
    (1, 300, 20, 10), (2, 96, 160, 48), (3, 32, 128, 16), (20, 64, 64, 32), (2, 24, 300, 4), (2, 72, 264, 32), (2, 40, 48, 0), (1, 128, 72, 112)]


@pytest.mark.parametrize("form", [0, 1])
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("H,D,V,rot", RETENTION)
def test_retention(H, D, V, rot, dtype, form):
    """Calls over the same slots: portions of every kind, then decode rows beside portions (a padding row among them), then
    decode rows alone; a slot that starts anew; decays of a few tokens, near one, and one."""
    g = _gen(D + V)
    n = lambda *s: torch.randn(*s, generator=g)          # noqa: E731
    width, rot = 2 * H * (D + V), dict(dims=rot, base=300.0)
    decay = torch.tensor(([0.5, 1.0, 1 - 2.0 ** -10, 0.93] * H)[1:H + 1])
    steps = [[(0, 70), (3, 1), (1, 2), (5, 333)], [(0, 1), (None, 1), (3, 1), (1, 33), (5, 3), (2, 17)], [(5, 1), (0, 1), (2, 1)], [(1, 140), (3, 2)]]
    decode = [0, 3, 3, 0]
    total = {s: sum(c for st in steps for q, c in st if q == s) for s in (0, 1, 2, 3, 5)}
    seq = {s: n(m, width + 8).to(dtype) for s, m in total.items()}
    want = {s: _oracle_retention(p.double(), H, D, V, rot, decay.double(), 1e-5, 0.7) for s, p in seq.items()}
    memory = torch.full((6, H, D, V), 7.0, device=DEV)                    # (slots held something before)
    inv, at = rope_inv_freq(rot["dims"], rot["base"], None)[0].to(DEV), {s: 0 for s in seq}
    for st, nd in zip(steps, decode):
        proj, exp, reset, pos = [], [], [], []
        for s, c in st:
            if s is None:
                proj.append(n(c, width + 8).to(dtype)), exp.append(None), reset.append(0), pos.append(torch.zeros(c))
                continue
            proj.append(seq[s][at[s]:at[s] + c]), exp.append(want[s][at[s]:at[s] + c]), reset.append(int(at[s] == 0))
            pos.append(torch.arange(at[s], at[s] + c))
            at[s] += c
        proj = torch.cat(proj).to(DEV)
        wide = torch.full((proj.shape[0], H * V + 16 + -(H * V) % 8), 9.0, dtype=dtype, device=DEV)
        retention.retention(proj, torch.cat(pos).int().to(DEV), inv, decay.to(DEV), memory, _i32([-1 if s is None else s for s, _ in st]),
                            _i32(bounds([c for _, c in st])), _i32(reset), wide[:, 8:8 + H * V], norm_eps=1e-5, gain=0.7, n_short=nd, form=form)
        for got, ref in zip(wide[:, 8:8 + H * V].cpu().split([c for _, c in st]), exp):
            if ref is not None:
                assert_close(got, ref, dtype, f32=2e-4)
            else:
                assert not got.any()
        assert (wide[:, :8] == 9).all() and (wide[:, 8 + H * V:] == 9).all()
    assert (memory[4] == 7).all() and _status_ok()
    for s, p in seq.items():                              # the state is fp32 whatever the rows are
        m = p.shape[0]
        k = O.rotate(p.double()[:, H * D:2 * H * D].view(m, H, D), rot) * D ** -0.5
        fade = decay.double()[None] ** torch.arange(m - 1, -1, -1)[:, None].double()
        assert_close(memory[s], torch.einsum("nhd,nhv->hdv", k * fade[..., None], p.double()[:, 2 * H * D:2 * H * D + H * V].view(m, H, V)), F32, f32=1e-4)


def test_retention_over_long_portions():
    """Chunks follow chunks: 700 tokens at once, from a state, and again in portions that end inside chunks; far positions."""
    g, H, D, V, rot, n = _gen(1), 3, 64, 96, dict(dims=32, base=1e4), 1500
    proj = torch.randn(n, 2 * H * (D + V), generator=g).to(BF16)
    decay, inv = torch.tensor([0.9, 0.999, 1.0]), rope_inv_freq(32, 1e4, None)[0].to(DEV)
    want = _oracle_retention(proj.double(), H, D, V, rot, decay.double(), 1e-5, 1.0)
    for sizes in ([1500], [700, 800], [130, 127, 1, 128, 129, 600, 385]):
        memory, at, out = torch.full((2, H, D, V), 5.0, device=DEV), 0, torch.empty(n, H * V, dtype=BF16, device=DEV)
        for c in sizes:
            retention.retention(proj[at:at + c].to(DEV), torch.arange(at, at + c, dtype=torch.int32, device=DEV), inv, decay.to(DEV), memory, _i32([1]),
                                _i32([0, c]), _i32([int(at == 0)]), out[at:at + c], norm_eps=1e-5)
            at += c
        assert_close(out, want, BF16)
    assert _status_ok()


# ----------------------------------------------------------------------------- whole models
def _check(raw, t, toks, dtype):
    want = O.forward(raw, t, toks)
    if dtype == F32:
        return lambda got: worst(got, want) < 1e-4
    return lambda got: bf16_ok(O, raw, t, toks, got, want)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", sorted(O.CONFIGS))
def test_prompt_portions_and_decoding(name, dtype):
    raw = O.CONFIGS[name]
    t = O.random_tensors(raw, seed=3)
    toks = tokens_for(raw, 150, 7)
    ok = _check(raw, t, toks, dtype)
    eng = llm_for(raw, t, DEV, dtype).engine
    for sizes in ([150], [2], [97, 1, 1, 1, 30, 2], [17, 64, 1, 33], [1]):
        assert ok(run_alone(eng, toks, sizes)), sizes


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_the_sum_of_the_streams_behind_every_layer(dtype):
    raw = O.CONFIGS["mixed"]
    t, toks = O.random_tensors(raw, seed=3), tokens_for(raw, 90, 7)
    layers = O.forward(raw, t, toks, want_layers=True)[1]
    llm = llm_for(raw, t, DEV, dtype)
    llm.model.capture_layers = tuple(range(len(layers)))
    run_alone(llm.engine, toks, [90])
    assert len(llm.model.captured) == len(layers) == 3
    for got, ref in zip(llm.model.captured, layers):
        assert float((got.cpu().double() - ref).norm() / ref.norm()) < (5e-6 if dtype == F32 else 0.08)


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_mixed_batches_on_reused_pages_and_slots(dtype):
    raw = O.CONFIGS["mixed"]
    t = O.random_tensors(raw, seed=5)
    lengths = [150, 7, 83, 1, 70, 18, 2, 141, 33]
    seqs = [tokens_for(raw, n, 20 + i) for i, n in enumerate(lengths)]
    eng = llm_for(raw, t, DEV, dtype, num_blocks=26, max_model_len=416).engine
    for got, s in zip(run_mixed(eng, seqs, interleave(lengths, [[50, 2, 1], [1], [5, 1, 1, 29], [3, 2]])), seqs):
        assert _check(raw, t, s, dtype)(got)
    assert eng.bm.num_free == 26 and len(eng.model.ssm.free) == 4


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_long_decoding_across_windows_blocks_and_pages(name, dtype):
    raw = O.CONFIGS[name]
    t = O.random_tensors(raw, seed=8)
    toks = tokens_for(raw, 640, 11)
    eng = llm_for(raw, t, DEV, dtype).engine
    assert _check(raw, t, toks, dtype)(run_alone(eng, toks, [390] + [1] * 250))


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_greedy_generation_through_the_scheduler(dtype):
    raw = O.CONFIGS["mixed"]
    t = O.random_tensors(raw, seed=9)
    prompts = [tokens_for(raw, n, 40 + n) for n in (23, 1, 90, 30, 4)]
    sp = SamplingParams(max_tokens=12, temperature=0.0, ignore_eos=True)
    outs = []
    for kw in (dict(), dict(max_batch=2, max_num_batched_tokens=16, num_blocks=12), dict(cuda_graphs=False)):
        llm = llm_for(raw, t, DEV, dtype, **kw)
        outs.append([s.output for s in llm.generate(prompt_token_ids=prompts, sampling_params=sp)])
        assert llm.engine.bm.num_free == llm.engine.ecfg.num_blocks
    if dtype == F32:
        want = [oracle_greedy(O, raw, t, p, 12) for p in prompts]
        assert all(o == want for o in outs)
        return
    for o in outs:                                                         # bf16: each token is the plain model's best up to rounding
        for p, gen in zip(prompts, o):
            lg = O.forward(raw, t, p + gen)[len(p) - 1:-1]
            assert (lg.amax(-1) - lg.gather(1, torch.tensor(gen)[:, None])[:, 0]).max() < 0.35 * float(lg.std())


def test_decode_steps_replay_graphs():
    raw = O.CONFIGS["mixed"]
    llm = llm_for(raw, O.random_tensors(raw, seed=9), DEV, BF16)
    sp = SamplingParams(max_tokens=8, temperature=0.0, ignore_eos=True)
    llm.generate(prompt_token_ids=[tokens_for(raw, 20, 1), tokens_for(raw, 9, 2)], sampling_params=sp)
    assert llm.engine._graphs and llm.engine.stats["decode_steps"] > 0
