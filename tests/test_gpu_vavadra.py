"""Vavadra kernels and engine on a GPU against the plain model (``oracle_vavadra``): every mechanism alone in fp32 and bf16
over sizes the fast kernels cover and sizes they do not, then whole models."""
import pytest
import torch

import oracle_vavadra as O
from design_runs import (assert_close, bf16_ok, bounds, fill_pages, interleave, llm_for, oracle_greedy, paged_tables, run_alone, run_mixed,
                         tokens_for, worst)
from mlxcel_b200.engine import SamplingParams
from mlxcel_b200.models import latent_mixer as LM
from mlxcel_b200.ops import KVLayer, _lib, gated_delta, latent, moe, stream
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


# ----------------------------------------------------------------------------- rows
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("dim", [64, 75, 1000, 4096, 6001, 9000])
def test_stream_adds_branch_experts_embedding_and_vector(dim, dtype):
    g, T, k, E = _gen(dim), 7, 3, 4
    n = lambda *s: torch.randn(*s, generator=g)          # noqa: E731
    table, vec, w = n(9, dim).to(dtype), n(dim), n(dim)
    ids = torch.tensor([3, 0, 8, 3, 1, 7, 2])
    d, dev = lambda t: t.double(), lambda t: t.to(DEV)   # noqa: E731
    h, x = stream.embed_stream(_i32(ids.tolist()), dev(table), 2.5, dev(w), 1e-5, 0.0, vec=dev(vec))
    h0 = d(table)[ids] * 2.5 + d(vec)
    assert_close(h, h0, F32)
    assert_close(x, O.norm(h0, d(w), 1e-5), dtype)
    y = n(T, dim).to(dtype)
    hd = dev(h0.float())
    x = stream.stream_norm(hd, dev(y), None, None, dev(w), 1e-5, 0.0)
    assert_close(hd, h0 + d(y), F32)
    assert_close(x, O.norm(h0 + d(y), d(w), 1e-5), dtype)
    pick = torch.randint(0, E + 2, (T, k), generator=g)                   # two identity experts
    rows, xin, shared, wts = n(T * k, dim).to(dtype), n(T, dim).to(dtype), n(T, dim).to(dtype), torch.rand(T, k, generator=g)
    perm = torch.randperm(T * k, generator=g)
    m = moe.MoeRows(dev(rows), dev(xin), dev(pick.int()), dev(perm.int()), dev(wts), E, dev(shared))
    part = torch.where((pick >= E)[..., None], d(xin)[:, None], d(rows)[perm].view(T, k, dim))
    want = h0 + (part * d(wts)[..., None]).sum(1) + d(shared)
    hd = dev(h0.float())
    x = stream.stream_norm(hd, None, None, None, dev(w), 1e-5, 0.0, dtype=dtype, moe=m)
    assert_close(hd, want, F32)
    assert_close(x, O.norm(want, d(w), 1e-5), dtype)
    m.shared = None
    hd = dev(h0.float())
    entry = stream.Entry(dev(vec), _i32(ids.tolist()), dev(table), 2.5)
    x = stream.stream_norm(hd, None, None, None, None, 1e-5, 0.0, dtype=dtype, plain=True, moe=m, entry=entry)
    want = want - d(shared) + d(table)[ids] * 2.5 + d(vec)
    assert_close(hd, want, F32)
    assert torch.equal(x, hd.to(dtype))
    hd = dev(h0.float())
    stream.stream_norm(hd, None, None, None, None, 1e-5, 0.0, dtype=dtype, entry=stream.Entry(dev(vec)))
    assert_close(hd, h0 + d(vec), F32)


@pytest.mark.parametrize("T,E,k", [(1, 3, 1), (70, 14, 3), (9, 130, 8), (200, 512, 16), (33, 7, 7), (5, 600, 2)])
def test_choice_of_experts(T, E, k):
    g = _gen(T + E)
    z, c = torch.randn(T, E + 3, generator=g) * 3, torch.randn(E, generator=g) * 0.2
    z[0, 0] = 40.0                                                        # one expert takes all of the softmax
    for corr in (c, torch.zeros(E)):
        want, ww = O.choose(z[:, :E].double(), corr.double(), k, 1.7)
        ids, wts = moe.route_choice(z.to(DEV)[:, :E], corr.to(DEV), k, 1.7)
        full = lambda i, w: torch.zeros(T, E, dtype=torch.float64).scatter_(1, i.cpu().long(), w.cpu().double())      # noqa: E731
        assert ids.dtype == torch.int32 and all(len(set(r)) == k for r in ids.tolist())
        assert torch.allclose(full(ids, wts), full(want, ww), atol=1e-6)


MOE = [  # tokens, width, ff, experts, identity, top
    (1, 64, 64, 4, 1, 2), (70, 96, 40, 6, 3, 3), (300, 128, 96, 12, 2, 4), (9, 75, 33, 3, 1, 1), (130, 64, 21, 7, 0, 5), (40, 256, 64, 64, 4, 6),
    (3, 64, 48, 2, 6, 2)]


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("T,H,I,E,Z,k", MOE)
def test_mixture_of_experts(T, H, I, E, Z, k, dtype):
    """The routed rows and their sum; the whole block against the plain statement; tokens that choose identity experts only."""
    g = _gen(T + I)
    n = lambda *s: torch.randn(*s, generator=g)          # noqa: E731
    spec = O.moe(I, E, Z, k, 0.8, 1.3)
    x = n(T, H).to(dtype)
    w = {"router": n(E + Z, H) * H ** -0.5 * 4, "correction": n(E + Z) * 0.1}
    if Z >= k:
        w["correction"][E:] += 5.0 * (T <= 3)                             # everything to the identity experts
    for e in range(E):
        w.update({f"e{e}.gate": n(I, H) * H ** -0.5 * 2, f"e{e}.up": n(I, H) * H ** -0.5, f"e{e}.down": n(H, I) * I ** -0.5})
    w = {name: t.to(dtype) for name, t in w.items()}
    want = O.experts(x.double(), {name: t.double() for name, t in w.items()}, spec)
    gu = torch.stack([torch.cat([w[f"e{e}.gate"], w[f"e{e}.up"]]) for e in range(E)]).to(DEV)
    dn = torch.stack([w[f"e{e}.down"] for e in range(E)]).to(DEV)
    ids, wts = O.choose(x.double() @ w["router"].double().T, w["correction"].double(), k, 1.3)
    for force in (False, True):
        m = moe.expert_rows(x.to(DEV), ids.int().to(DEV), wts.float().to(DEV), gu, dn, 1.702, 0.8, force_any=force)
        h = torch.zeros(T, H, device=DEV)
        stream.stream_norm(h, None, None, None, None, 1e-5, 0.0, dtype=dtype, moe=m)
        assert_close(h, want, dtype, bf16=2.5e-2)
    assert moe.expert_rows(x[:0].to(DEV), ids[:0].int().to(DEV), wts[:0].float().to(DEV), gu, dn, 1.702, 0.8).y.shape == (0, H)
    assert _status_ok()


# ----------------------------------------------------------------------------- differential attention
DIFF = [  # heads, key heads, map width, value width, chunk, page
    (12, 2, 32, 64, 24, 16), (6, 2, 16, 40, 168, 16), (4, 4, 64, 128, 129, 16), (16, 2, 40, 72, 1, 16), (3, 3, 9, 11, 13, 8),
    (8, 1, 64, 128, 64, 16), (9, 1, 64, 64, 100, 16), (2, 1, 96, 128, 256, 16), (2, 1, 24, 48, 128, 32), (4, 2, 128, 64, 48, 16),
    (5, 5, 8, 8, 64, 16)]


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("Hq,Hkv,D,Dv,chunk,bs", DIFF)
def test_differential_attention(Hq, Hkv, D, Dv, chunk, bs, dtype):
    """Prompt portions that start and end anywhere, and decode rows. Keys at the chunks' edges (the last of the chunk before,
    the first two of this one) outscore the rest, each in one map only."""
    g = _gen(Hq + D)
    lens, qlens = [300, 129, 17, 401, 64], [300, 2, 17, 150, 1]
    tab, blocks = paged_tables(lens, bs)
    kp, vp = torch.zeros(blocks, Hkv, bs, 2 * D, dtype=dtype), torch.zeros(blocks, Hkv, bs, Dv, dtype=dtype)
    ks, vs, qs = [], [], []
    for s, (n, ql) in enumerate(zip(lens, qlens)):
        k, v = torch.randn(n, Hkv, 2, D, generator=g).to(dtype), torch.randn(n, Hkv, Dv, generator=g).to(dtype)
        for c in range(0, n, chunk):
            for i, p in enumerate((c - 1, c, c + 1)):
                if 0 <= p < n:
                    k[p, :, (i + c) % 2] = k[p, :, (i + c) % 2].abs() + 1
        ks.append(k), vs.append(v), qs.append((torch.randn(ql, Hq, 2, D, generator=g) * 0.3 + 0.7).to(dtype))
        fill_pages(kp, tab, s, k.reshape(n, Hkv, 2 * D)), fill_pages(vp, tab, s, v)
    scale, lam, gain, eps = 6.0 / D, 0.73, 0.55, 1e-5
    kv = KVLayer(kp.to(DEV), vp.to(DEV), None, None, bs)

    def want(s, rows):
        n, ql = lens[s], qlens[s]
        m = O.chunk_mask(n, chunk)[n - ql:]
        q, k, v = qs[s].double(), ks[s].double(), vs[s].double()
        one = lambda a, i: O.attend(q[:, a, i] @ k[:, a // (Hq // Hkv), i].T * scale, m, v[:, a // (Hq // Hkv)])       # noqa: E731
        out = torch.stack([O.unit_rms(one(a, 0) - lam * one(a, 1), eps) * gain for a in range(Hq)], 1)
        return out[rows].reshape(-1, Hq * Dv)
    q = torch.cat(qs).reshape(-1, Hq * 2 * D).to(DEV)
    cu = bounds(qlens)
    kw = dict(Hq=Hq, Hkv=Hkv, Dk=2 * D, Dv=Dv, scale=scale, chunk=chunk, diff=(lam, gain, eps))
    wp = torch.cat([want(s, slice(None)) for s in range(5)])
    wd = torch.cat([want(s, slice(-1, None)) for s in range(5)])
    qd = torch.cat([x[-1:] for x in qs]).reshape(-1, Hq * 2 * D).to(DEV)
    for force in (False, True):
        out = torch.empty(q.shape[0], Hq * Dv, dtype=dtype, device=DEV)
        stream.paged_attention(q, kv, tab.to(DEV), _i32(lens), _i32(cu), out, max_q_len=300, force_any=force, **kw)
        assert_close(out, wp, dtype, f32=1e-4)
        o = torch.empty(5, Hq * Dv, dtype=dtype, device=DEV)
        stream.paged_attention(qd, kv, tab.to(DEV), _i32(lens), None, o, max_q_len=1, max_len=401, force_any=force, **kw)
        assert_close(o, wd, dtype, f32=1e-4)
    assert _status_ok()


def test_differential_decode_merges_splits_of_long_contexts():
    g, Hq, Hkv, D, Dv, n = _gen(1), 8, 2, 64, 128, 3000
    tab, blocks = paged_tables([n, 700], 16)
    kp, vp = torch.zeros(blocks, Hkv, 16, 2 * D, dtype=BF16), torch.zeros(blocks, Hkv, 16, Dv, dtype=BF16)
    k, v = torch.randn(n, Hkv, 2, D, generator=g).to(BF16), torch.randn(n, Hkv, Dv, generator=g).to(BF16)
    q = torch.randn(2, Hq, 2, D, generator=g).to(BF16)
    k[37, :, 0], k[2500, :, 1] = q[0, ::4, 0], q[0, ::4, 1]                # one key per map that stands out
    for s, m in enumerate((n, 700)):
        fill_pages(kp, tab, s, k[:m].reshape(m, Hkv, 2 * D)), fill_pages(vp, tab, s, v[:m])
    kv = KVLayer(kp.to(DEV), vp.to(DEV), None, None, 16)
    one = lambda s, m, a, i: O.attend(q[s, a, i][None].double() @ k[:m, a // 4, i].double().T * 0.2, torch.ones(1, m).bool(), v[:m, a // 4].double())   # noqa: E731
    want = torch.stack([torch.cat([O.unit_rms(one(s, m, a, 0) - 0.4 * one(s, m, a, 1), 1e-6)[0] * 0.8 for a in range(Hq)])
                        for s, m in enumerate((n, 700))])
    for max_len in (200, n):
        out = torch.empty(2, Hq * Dv, dtype=BF16, device=DEV)
        stream.paged_attention(q.view(2, -1).to(DEV), kv, tab.to(DEV), _i32([n, 700]), None, out, Hq=Hq, Hkv=Hkv, Dk=2 * D, Dv=Dv, scale=0.2,
                               max_q_len=1, max_len=max_len, diff=(0.4, 0.8, 1e-6))
        assert_close(out, want, BF16)


# ----------------------------------------------------------------------------- latent attention
LAT = [  # heads, dim, rot, vdim, latent, window, page
    (7, 48, 32, 56, 80, 130, 16), (16, 128, 64, 128, 512, 64, 16), (3, 24, 16, 40, 56, 1, 16), (20, 72, 64, 128, 512, 200, 16),
    (5, 9, 6, 11, 13, 33, 16), (40, 96, 40, 80, 200, 65, 32), (1, 8, 8, 8, 8, 300, 16), (4, 128, 8, 64, 264, 129, 16)]


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("H,D,R,V,C", [x[:5] for x in LAT])
def test_rotation_of_neighbouring_dimensions(H, D, R, V, C, dtype):
    g, T = _gen(C), 21
    a = torch.randn(T, C + R + 5, generator=g).to(dtype)
    cw, rot = torch.randn(C, generator=g), dict(dims=R, base=900.0)
    inv = rope_inv_freq(R, 900.0, None)[0].to(DEV)
    pool = torch.zeros(4, 1, 16, C + R, dtype=dtype, device=DEV)
    slots, pos = torch.arange(T) * 2 + 1, torch.arange(T) + 90
    slots[3] = -1
    latent.latent_append(a.to(DEV), pos.int().to(DEV), slots.int().to(DEV), KVLayer(pool, pool[..., :0], None, None, 16), Q=0, C=C, R=R, inv_freq=inv,
                         mscale=1.0, q_norm=None, c_norm=cw.to(DEV), eps=1e-5, adjacent=True)
    ad, ok = a.double(), slots >= 0
    entry = torch.cat([O.norm(ad[:, :C], cw.double(), 1e-5), O.rotate(ad[:, None, C:C + R], rot, 90)[:, 0]], -1)
    flat = pool.view(-1, C + R).cpu()
    assert_close(flat[slots[ok]], entry[ok], dtype, f32=5e-5)
    assert int((flat != 0).any(-1).sum()) == T - 1
    q = torch.randn(T, H * (D + R), generator=g).to(dtype)
    want = O.rotate(q.view(T, H, D + R)[..., D:].double(), rot, 90)
    qd = q.to(DEV)
    latent.latent_q_rope(qd, qd, pos.int().to(DEV), H=H, q_at=D, q_head=D + R, d_at=D, d_head=D + R, inv_freq=inv, mscale=1.0, adjacent=True)
    assert_close(qd.view(T, H, D + R)[..., D:], want, dtype, f32=5e-5)
    assert torch.equal(qd.view(T, H, D + R)[..., :D].cpu(), q.view(T, H, D + R)[..., :D])


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("H,D,R,V,C,window,bs", LAT)
def test_absorbed_latent_attention_with_window_and_sink(H, D, R, V, C, window, bs, dtype):
    """Decode rows over contexts of very different length. The rows at both sides of the window's edge outscore the others for
    head 0 (the one outside would take most of the weight); split and unsplit."""
    g, W, scale = _gen(H + C), C + R, 0.1
    lens = [1, 700, 64, 65, 0, 333, window, window + 1, 130]
    tab, blocks = paged_tables(lens, bs)
    pool = torch.zeros(blocks, 1, bs, W, dtype=dtype)
    rows, q = [], (torch.randn(len(lens), H, W, generator=g) * (12 / W ** 0.5)).to(dtype)
    sink = torch.randn(H, generator=g) * 3 + 2
    for s, n in enumerate(lens):
        r = torch.randn(n, W, generator=g).to(dtype)
        for p, lift in ((n - window - 1, 14.0), (n - window, 10.0)):
            if 0 <= p < n - 1:
                r[p] = (q[s, 0] * (lift / scale / float(q[s, 0].float().pow(2).sum()))).to(dtype)
        rows.append(r)
        fill_pages(pool, tab, s, r[:, None])
    want = torch.zeros(len(lens), H, C, dtype=torch.float64)
    for s, n in enumerate(lens):
        if n:
            sc = q[s].double() @ rows[s].double().T * scale
            want[s] = torch.cat([O.attend(sc[a:a + 1], O.window_mask(n, window)[-1:], rows[s][:, :C].double(), sink[a].double()) for a in range(H)])
    kv = KVLayer(pool.to(DEV), pool[..., :0].to(DEV), None, None, bs)
    kw = dict(H=H, C=C, scale=scale, window=window, sinks=sink.to(DEV))
    big = torch.cat([q] * 30).reshape(-1, H * W).to(DEV)                   # more rows than SMs: no split
    for form in (0, 1):                                                    # tcgen05 where it applies; mma.sync
        out = torch.full((len(lens), H * C), 9.0, dtype=dtype, device=DEV)
        latent.latent_attention(q.reshape(-1, H * W).to(DEV), kv, tab.to(DEV), _i32(lens), None, out, max_len=700, form=form, **kw)
        assert_close(out.view(-1, H, C), want, dtype, f32=5e-5)
        out = torch.empty(big.shape[0], H * C, dtype=dtype, device=DEV)
        latent.latent_attention(big, kv, tab.repeat(30, 1).to(DEV), _i32(lens * 30), None, out, max_len=700, form=form, **kw)
        assert_close(out.view(30, -1, H, C), want.expand(30, -1, -1, -1), dtype, f32=5e-5)
    # the whole context in several splits, with sinks
    full = torch.zeros_like(want)
    for s, n in enumerate(lens):
        if n:
            sc = q[s].double() @ rows[s].double().T * scale
            full[s] = torch.cat([O.attend(sc[a:a + 1], torch.ones(1, n).bool(), rows[s][:, :C].double(), sink[a].double()) for a in range(H)])
    kw["window"] = 0
    for form in (0, 1):
        out = torch.full((len(lens), H * C), 9.0, dtype=dtype, device=DEV)
        latent.latent_attention(q.reshape(-1, H * W).to(DEV), kv, tab.to(DEV), _i32(lens), None, out, max_len=5000, form=form, **kw)
        assert_close(out.view(-1, H, C), full, dtype, f32=5e-5)
    assert _status_ok()


@pytest.mark.parametrize("H,D,R,V,C,window,bs", [x for x in LAT if x[4] % 8 == 0])
def test_expanded_latent_attention_with_window_and_sink(H, D, R, V, C, window, bs):
    """Prompt portions against partly gathered rows: what no query's window reaches is left out."""
    g, W, scale = _gen(D), C + R, 2.0 / (D + R)
    lens, qlens = [300, 529, 17, 260, 64], [300, 2, 17, 140, 1]
    tab, blocks = paged_tables(lens, bs)
    pool = torch.zeros(blocks, 1, bs, W, dtype=BF16)
    rows = [torch.randn(n, W, generator=g).to(BF16) for n in lens]
    for s, r in enumerate(rows):
        fill_pages(pool, tab, s, r[:, None])
    kv = KVLayer(pool.to(DEV), pool[..., :0].to(DEV), None, None, bs)

    class Batch:
        pf_cu_q_host, pf_starts, pf_context_lens = bounds(qlens), [n - q for n, q in zip(lens, qlens)], _i32(lens)
    edges, zero, total = LM.context_rows(Batch(), window)
    skips = [max(0, n - q - window + 1) // 128 * 128 for n, q in zip(lens, qlens)]
    ctx = latent.latent_gather(kv, tab.to(DEV), edges, total, zero)
    assert total == sum(lens) - sum(skips) and torch.equal(ctx.cpu(), torch.cat([r[k:] for r, k in zip(rows, skips)]))
    kn, v = ([torch.randn(n, H, d, generator=g).to(BF16) for n in lens] for d in (D, V))
    sink = torch.randn(H, generator=g) * 2 + 1
    q = torch.randn(sum(qlens), H, D + R, generator=g).to(BF16)
    out = torch.full((sum(qlens), H * V + 8), 9.0, dtype=BF16, device=DEV)
    cu, want = bounds(qlens), []
    for s, (n, ql) in enumerate(zip(lens, qlens)):
        qs = q[cu[s]:cu[s] + ql].double()
        for i in (0, ql - 1):                                              # a key just outside this row's window outscores the rest
            p = n - ql + i - window
            if p >= 0:
                kn[s][p] = (kn[s][p].double() + 1.5 * qs[i, :, :D]).to(BF16)
        k = torch.cat([kn[s], rows[s][:, None, C:].expand(n, H, R)], -1).double()
        sc = torch.einsum("qhd,khd->hqk", qs, k) * scale
        m = O.window_mask(n, window)[n - ql:]
        want.append(torch.stack([O.attend(sc[a], m, v[s][:, a].double(), sink[a].double()) for a in range(H)], 1).reshape(ql, H * V))
    part = lambda t, h0, h1, d: torch.cat([x[k:, h0:h1] for x, k in zip(t, skips)]).reshape(-1, (h1 - h0) * d).to(DEV)      # noqa: E731
    qd, h = q.reshape(-1, H * (D + R)).to(DEV), max(1, H // 2)
    for h0, h1 in ((0, h), (h, H)):                                        # two groups of heads into column slices
        if h1 > h0:
            latent.latent_prefill(qd[:, h0 * (D + R):h1 * (D + R)], part(kn, h0, h1, D), ctx[:, C:], part(v, h0, h1, V), _i32(cu), _i32(lens), zero,
                                  out[:, h0 * V:h1 * V], H=h1 - h0, D=D, R=R, V=V, scale=scale, max_q_len=300, window=window,
                                  sinks=sink.to(DEV)[h0:h1])
    assert_close(out[:, :H * V], torch.cat(want), BF16)
    assert (out[:, H * V:] == 9.0).all() and _status_ok()


# ----------------------------------------------------------------------------- gated delta rule
GD = [  # heads, key heads, dim, vdim, taps
    (4, 2, 32, 48, 3), (6, 3, 64, 24, 2), (2, 2, 128, 128, 4), (8, 2, 128, 64, 4), (3, 1, 10, 7, 5), (2, 2, 33, 12, 1), (1, 1, 4, 4, 4), (2, 1, 140, 132, 4),
    (4, 4, 16, 128, 3), (2, 1, 96, 160, 2), (3, 3, 10, 12, 4)]


def _oracle_delta(x, rates, gate, conv, A_log, dt_bias, nw, G, D, V, eps):
    """One sequence from its start, through the plain model's own functions (identity projections)."""
    n, H = x.shape[0], rates.shape[1] // 2
    y = O.short_conv(x, conv)
    q, k = O.unit(y[:, :G * D].view(n, G, D)) * D ** -0.5, O.unit(y[:, G * D:2 * G * D].view(n, G, D))
    q, k = q.repeat_interleave(H // G, 1), k.repeat_interleave(H // G, 1)
    eye = torch.eye(2 * H, dtype=x.dtype)
    beta, g = O.delta_rates(rates, {"b": eye[:H], "a": eye[H:], "A_log": A_log, "dt_bias": dt_bias})
    o = O.norm(O.delta_memory(q, k, y[:, 2 * G * D:].reshape(n, H, V), beta, g), nw, eps).reshape(n, H * V)
    return o * gate * torch.sigmoid(gate)


@pytest.mark.parametrize("force_any", [False, True])
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("H,G,D,V,taps", GD)
def test_gated_delta_rule(H, G, D, V, taps, dtype, force_any):
    """Three calls over the same slots: portions of every kind, then decode rows beside portions (a padding row among them),
    then decode rows alone; a slot that starts anew; long memory (decays near one)."""
    g = _gen(D + V)
    n = lambda *s: torch.randn(*s, generator=g)          # noqa: E731
    ch = 2 * G * D + H * V
    conv, A_log, dt_bias, nw = n(ch, taps) * taps ** -0.5, n(H) * 0.5, n(H) - 4, 1 + 0.3 * n(V)
    steps = [[(0, 70), (3, 1), (1, 2), (5, 150)], [(0, 1), (None, 1), (3, 1), (1, 33), (5, 3), (2, 17)], [(5, 1), (0, 1), (2, 1)], [(1, 40), (3, 2)]]
    decode = [0, 3, 3, 0]
    total = {s: sum(c for st in steps for q, c in st if q == s) for s in (0, 1, 2, 3, 5)}
    seq = {s: (n(m, ch + H * V + 3).to(dtype), n(m, 2 * H)) for s, m in total.items()}
    d = lambda t: t.double()                             # noqa: E731
    want = {s: _oracle_delta(d(p[:, :ch]), d(r), d(p[:, ch:ch + H * V]), d(conv), d(A_log), d(dt_bias), d(nw), G, D, V, 1e-5)
            for s, (p, r) in seq.items()}
    memory, tail = (torch.full(s, 7.0, device=DEV) for s in ((6, H, D, V), (6, taps - 1, ch)))       # (slots held something before)
    w = [t.to(DEV) for t in (conv, A_log, dt_bias, nw)]
    at = {s: 0 for s in seq}
    for st, nd in zip(steps, decode):
        proj, rates, exp, reset = [], [], [], []
        for s, c in st:
            if s is None:
                proj.append(n(c, ch + H * V + 3).to(dtype)), rates.append(n(c, 2 * H)), exp.append(torch.zeros(c, H * V).double()), reset.append(0)
                continue
            sl = slice(at[s], at[s] + c)
            proj.append(seq[s][0][sl]), rates.append(seq[s][1][sl]), exp.append(want[s][sl]), reset.append(int(at[s] == 0))
            at[s] += c
        out = gated_delta.gated_delta(torch.cat(proj).to(DEV), torch.cat(rates).to(DEV), *w, memory, tail,
                                      _i32([-1 if s is None else s for s, _ in st]), _i32(bounds([c for _, c in st])), _i32(reset), G=G,
                                      norm_eps=1e-5, n_short=nd, force_any=force_any)
        for got, ref in zip(out.cpu().split([c for _, c in st]), exp):
            if ref.any():
                assert_close(got, ref, dtype, f32=1e-4)
            else:
                assert not got.any()
    assert (memory[4] == 7).all() and (tail[4] == 7).all()
    for s, (p, _) in seq.items():
        have = p[-(taps - 1):, :ch].float() if taps > 1 else p[:0, :ch].float()
        assert torch.equal(tail[s].cpu()[taps - 1 - have.shape[0]:], have)
    assert _status_ok()


# ----------------------------------------------------------------------------- whole models
def _check(raw, t, toks, dtype):
    want = O.forward(raw, t, toks)
    if dtype == F32:
        return lambda got: worst(got, want) < 1e-4
    return lambda got: bf16_ok(O, raw, t, toks, got, want)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", sorted(O.CONFIGS))
def test_prompt_portions_and_decoding(name, dtype, monkeypatch):
    raw = O.CONFIGS[name]
    t = O.random_tensors(raw, seed=3)
    toks = tokens_for(raw, 150, 7)
    ok = _check(raw, t, toks, dtype)
    eng = llm_for(raw, t, DEV, dtype).engine
    for sizes in ([150], [2], [97, 1, 1, 1, 30, 2], [17, 64, 1, 33]):
        assert ok(run_alone(eng, toks, sizes)), sizes
    assert ok(run_alone(eng, toks, [1]))
    monkeypatch.setattr(LM, "EXPAND_BYTES", 1)                             # one head at a time
    assert ok(run_alone(eng, toks, [100, 50]))


@pytest.mark.parametrize("dtype", [F32, BF16])
def test_the_stream_behind_every_layer(dtype):
    raw = O.CONFIGS["mixed"]
    t, toks = O.random_tensors(raw, seed=3), tokens_for(raw, 90, 7)
    layers = O.forward(raw, t, toks, want_layers=True)[1]
    llm = llm_for(raw, t, DEV, dtype)
    llm.model.capture_layers = tuple(range(len(layers)))
    run_alone(llm.engine, toks, [90])
    assert len(llm.model.captured) == len(layers) == 8
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
def test_long_decoding_across_windows_chunks_and_pages(name, dtype):
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
