"""Govopel kernels and engine on a GPU against the plain model (``oracle_govopel``): every mechanism alone in fp32 and bf16
over sizes the fast kernels cover and sizes they do not, then whole models."""
import pytest
import torch

import oracle_govopel as O
from design_runs import bf16_ok, interleave, llm_for, oracle_greedy, run_alone, run_mixed, tokens_for, worst
from mlxcel_b200 import ops
from mlxcel_b200.engine import SamplingParams
from mlxcel_b200.models import latent_mixer as LM
from mlxcel_b200.models.govopel import rotation_table
from mlxcel_b200.ops import KVLayer, _lib, latent, stream

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


def _i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


def _paged(lens, bs, seed=0):
    """Block tables of sequences of these lengths over a shuffled pool; (tables, blocks in the pool)."""
    need = [-(-n // bs) for n in lens]
    perm = torch.randperm(sum(need) + 3, generator=_gen(seed)).tolist()
    tab, at = torch.zeros(len(lens), max(max(need), 1), dtype=torch.int32), 0
    for s, k in enumerate(need):
        tab[s, :k] = torch.tensor(perm[at:at + k], dtype=torch.int32)
        at += k
    return tab, len(perm)


def _fill(pool, tab, s, rows):
    """rows [n, heads, width] as the first n entries of sequence s."""
    bs = pool.shape[2]
    for i in range(rows.shape[0]):
        pool[int(tab[s, i // bs]), :, i % bs] = rows[i].to(pool.dtype)


# ----------------------------------------------------------------------------- rows
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("dim", [64, 75, 1000, 4096, 6001])
def test_stream_without_inner_norm(dim, dtype):
    g, n = _gen(dim), 6
    table, w, ids = torch.randn(9, dim, generator=g).to(dtype), torch.randn(dim, generator=g), torch.tensor([3, 0, 8, 3, 1, 7])
    h, x = stream.embed_stream(_i32(ids.tolist()), table.to(DEV), 1.0, None, 1e-5, 0.0, w.to(DEV))
    want = O.embed(ids, table.double(), w.double(), 1e-5)
    _close(h, want, F32)
    assert x.dtype == dtype and torch.equal(x, h.to(dtype))
    y, pw, ls = torch.randn(n, dim, generator=g).to(dtype), torch.randn(dim, generator=g), torch.randn(dim, generator=g)
    hc = h.double().cpu()
    x = stream.stream_norm(h, y.to(DEV), pw.to(DEV), None, None, 1e-5, 0.0, plain=True)
    _close(h, hc + O.norm(y.double(), pw.double(), 1e-5), F32)
    assert torch.equal(x, h.to(dtype))
    assert stream.stream_norm(h, y.to(DEV), pw.to(DEV), ls.to(DEV), None, 1e-5, 0.0) is None


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("M,K,I", [(1, 64, 64), (3, 75, 33), (65, 96, 112), (200, 256, 320), (7, 64, 50)])
def test_clipped_glu_projection(M, K, I, dtype):
    g = _gen(M + I)
    x, w = torch.randn(M, K, generator=g).to(dtype) * 2, (torch.randn(2 * I, K, generator=g) * K ** -0.5).to(dtype)
    xd, wd = x.double(), w.double()
    want = O.clipped_glu(xd @ wd[:I].T, xd @ wd[I:].T, 1.25)
    _close(ops.glu_linear(x.to(DEV), w.to(DEV), I, "clipped_swiglu", limit=1.25), want, dtype, bf16=2e-2)


def test_soft_cap_of_logits():
    z = torch.randn(5, 1003, generator=_gen(0)) * 40
    _close(stream.softcap_(z.to(DEV), 11.0), O.soft_cap(z.double(), 11.0), F32, f32=2e-6)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("G,M,N,K,pad", [(7, 1, 80, 56, 32), (7, 5, 56, 80, 0), (3, 130, 56, 40, 8), (4, 70, 264, 24, 16), (3, 9, 11, 13, 5),
                                         (16, 200, 512, 128, 64), (5, 33, 128, 512, 64)])
def test_batched_projection(G, M, N, K, pad, dtype):
    g = _gen(G * M)
    x, w = torch.randn(M, G * (K + pad), generator=g).to(dtype), (torch.randn(G, N, K, generator=g) * K ** -0.5).to(dtype)
    out = torch.full((M, G * (N + pad)), 7.0, dtype=dtype, device=DEV)
    ops.batched_linear(x.to(DEV), w.to(DEV), out, K + pad, N + pad)
    o = out.cpu().view(M, G, N + pad)
    _close(o[..., :N], torch.einsum("mgk,gnk->mgn", x.view(M, G, K + pad)[..., :K].double(), w.double()), dtype)
    assert (o[..., N:] == 7.0).all()


# ----------------------------------------------------------------------------- attention over chunks
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("Hq,Hkv,D,R", [(6, 2, 48, 24), (4, 1, 64, 64), (3, 3, 20, 10), (5, 5, 33, 22), (10, 2, 128, 2), (2, 1, 8, 0)])
@pytest.mark.parametrize("shared", [True, False])
def test_rotation_norm_append(Hq, Hkv, D, R, shared, dtype):
    g, T, Dv = _gen(D), 19, D if shared else D + 4
    rot = O.attn_spec(Hq, Hkv, D, R or 2, 8, 1.0, 1.0, None)["mixer"]["rot"]
    width = (Hq + Hkv) * D + (0 if shared else Hkv * Dv) + 3
    row = torch.randn(T, width, generator=g).to(dtype)
    kv = KVLayer(torch.zeros(4, Hkv, 16, D, dtype=dtype, device=DEV), torch.zeros(4, Hkv, 16, Dv, dtype=dtype, device=DEV), None, None, 16)
    inv, ms = rotation_table(rot, DEV)
    inv = inv[:R // 2].contiguous()
    w = torch.randn(D, generator=g)
    slots, pos = torch.arange(T) * 3 + 2, torch.arange(T) + 700
    slots[5] = -1
    r = row.to(DEV)
    stream.rope_norm_append(r, pos.int().to(DEV), slots.int().to(DEV), kv, Hq=Hq, Hkv=Hkv, Dk=D, Dv=Dv, inv_freq=inv, mscale=ms,
                            values_are_keys=shared, k_norm=w.to(DEV), eps=1e-5)
    turn = lambda z: O.unit_rms(O.rotate(z.double(), rot, 700) if R else z.double(), 1e-5)      # noqa: E731
    q, k = row[:, :Hq * D].view(T, Hq, D), row[:, Hq * D:(Hq + Hkv) * D].view(T, Hkv, D)
    v = k if shared else row[:, (Hq + Hkv) * D:(Hq + Hkv) * D + Hkv * Dv].view(T, Hkv, Dv)
    _close(r[:, :Hq * D].view(T, Hq, D), turn(q), dtype, f32=2e-4)                  # (fp32 angles at position 700)
    assert torch.equal(r[:, Hq * D:].cpu(), row[:, Hq * D:])
    kk = turn(k) * w.double()
    kc, vc = kv.k.cpu(), kv.v.cpu()
    ok = [t for t in range(T) if slots[t] >= 0]
    at = [(int(slots[t]) // 16, int(slots[t]) % 16) for t in ok]
    _close(torch.stack([kc[b, :, o] for b, o in at]), kk[ok], dtype, f32=2e-4)
    assert torch.equal(torch.stack([vc[b, :, o] for b, o in at]), v[ok])
    assert int((vc != 0).any(-1).any(1).sum()) == len(ok)


ATT = [  # heads, key heads, key width, value width, chunk, page
    (12, 1, 64, 64, 24, 16), (6, 2, 48, 48, 168, 16), (4, 4, 128, 128, 129, 16), (16, 1, 128, 64, 1, 16), (3, 3, 20, 20, 13, 8),
    (20, 1, 64, 64, 64, 16), (2, 1, 40, 96, 128, 32), (4, 2, 16, 16, 0, 16)]


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("Hq,Hkv,Dk,Dv,chunk,bs", ATT)
def test_chunked_soft_capped_attention(Hq, Hkv, Dk, Dv, chunk, bs, dtype):
    """Prompt portions that start and end anywhere, and decode rows, with the keys at the chunk's edges planted to outscore the
    rest (the last of the chunk before, the first and second of this one)."""
    g = _gen(Hq + Dk)
    lens, qlens = [300, 129, 17, 401, 64], [300, 2, 17, 150, 1]
    tab, blocks = _paged(lens, bs)
    kp, vp = torch.zeros(blocks, Hkv, bs, Dk, dtype=dtype), torch.zeros(blocks, Hkv, bs, Dv, dtype=dtype)
    ks, vs, qs = [], [], []
    for s, (n, ql) in enumerate(zip(lens, qlens)):
        k, v = torch.randn(n, Hkv, Dk, generator=g).to(dtype), torch.randn(n, Hkv, Dv, generator=g).to(dtype)
        for c in range(0, n, chunk or 100):
            for p in (c - 1, c, c + 1):
                if 0 <= p < n:
                    k[p] = k[p].abs() + 1
        ks.append(k), vs.append(v), qs.append((torch.randn(ql, Hq, Dk, generator=g) * 0.3 + 0.7).to(dtype))
        _fill(kp, tab, s, k), _fill(vp, tab, s, v)
    scale, cap = 6.0 / Dk, 9.0
    kv = KVLayer(kp.to(DEV), vp.to(DEV), None, None, bs)

    def want(s, rows):
        n, ql = lens[s], qlens[s]
        m = O.chunk_mask(n, chunk) if chunk else O.causal_mask(n)
        q, k, v = qs[s].double(), ks[s].double(), vs[s].double()
        return torch.stack([O.attend(O.soft_cap(q[:, a] @ k[:, a // (Hq // Hkv)].T * scale, cap), m[n - ql:], v[:, a // (Hq // Hkv)])
                            for a in range(Hq)], 1)[rows].reshape(-1, Hq * Dv)
    q = torch.cat(qs).reshape(-1, Hq * Dk).to(DEV)
    cu = [0]
    for x in qlens:
        cu.append(cu[-1] + x)
    kw = dict(Hq=Hq, Hkv=Hkv, Dk=Dk, Dv=Dv, scale=scale, softcap=cap, chunk=chunk)
    wp = torch.cat([want(s, slice(None)) for s in range(5)])
    wd = torch.cat([want(s, slice(-1, None)) for s in range(5)])
    qd = torch.cat([x[-1:] for x in qs]).reshape(-1, Hq * Dk).to(DEV)
    for force in (False, True):
        out = torch.empty(q.shape[0], Hq * Dv, dtype=dtype, device=DEV)
        stream.paged_attention(q, kv, tab.to(DEV), _i32(lens), _i32(cu), out, max_q_len=300, force_any=force, **kw)
        _close(out, wp, dtype, f32=5e-5)
        for max_len in (401, 4000):
            o = torch.empty(5, Hq * Dv, dtype=dtype, device=DEV)
            stream.paged_attention(qd, kv, tab.to(DEV), _i32(lens), None, o, max_q_len=1, max_len=max_len, force_any=force, **kw)
            _close(o, wd, dtype, f32=5e-5)
    assert _lib.read_status(torch.device(DEV, 0)) == 0


# ----------------------------------------------------------------------------- latent attention
LAT = [  # heads, dim, rot, vdim, latent, page
    (7, 48, 32, 56, 80, 16), (16, 128, 64, 128, 512, 16), (3, 24, 16, 40, 56, 16), (20, 72, 64, 128, 512, 16), (5, 9, 6, 11, 13, 16),
    (40, 96, 40, 80, 200, 32), (1, 8, 8, 8, 8, 16), (4, 128, 8, 64, 264, 16)]


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("H,D,R,V,C,bs", LAT)
def test_latent_append_and_query_rotation(H, D, R, V, C, bs, dtype):
    g, T, Q = _gen(C), 21, 40 if C % 8 == 0 else 17
    a = torch.randn(T, Q + C + R + 5, generator=g).to(dtype)
    qw, cw = torch.randn(Q, generator=g), torch.randn(C, generator=g)
    rot = dict(dims=R, base=900.0)
    inv = rotation_table(rot, DEV)[0]
    pool = torch.zeros(4, 1, bs, C + R, dtype=dtype, device=DEV)
    slots, pos = torch.arange(T) * 2 + 1, torch.arange(T) + 90
    slots[3] = -1
    d = a.to(DEV)
    latent.latent_append(d, pos.int().to(DEV), slots.int().to(DEV), KVLayer(pool, pool[..., :0], None, None, bs), Q=Q, C=C, R=R, inv_freq=inv,
                         mscale=1.0, q_norm=qw.to(DEV), c_norm=cw.to(DEV), eps=1e-5)
    ad = a.double()
    _close(d[:, :Q], O.norm(ad[:, :Q], qw.double(), 1e-5), dtype)
    assert torch.equal(d[:, Q:].cpu(), a[:, Q:])
    entry = torch.cat([O.norm(ad[:, Q:Q + C], cw.double(), 1e-5), O.rotate(ad[:, None, Q + C:Q + C + R], rot, 90)[:, 0]], -1)
    flat = pool.view(-1, C + R).cpu()
    ok = slots >= 0
    _close(flat[slots[ok]], entry[ok], dtype, f32=5e-5)
    assert int((flat != 0).any(-1).sum()) == T - 1
    q = torch.randn(T, H * (D + R), generator=g).to(dtype)
    want = O.rotate(q.view(T, H, D + R)[..., D:].double(), rot, 90)
    qd, dst = q.to(DEV), torch.zeros(T, H * (C + R), dtype=dtype, device=DEV)
    kw = dict(H=H, q_at=D, q_head=D + R, inv_freq=inv, mscale=1.0)
    latent.latent_q_rope(qd, dst, pos.int().to(DEV), d_at=C, d_head=C + R, **kw)
    _close(dst.view(T, H, C + R)[..., C:], want, dtype, f32=5e-5)
    assert not dst.view(T, H, C + R)[..., :C].any()
    latent.latent_q_rope(qd, qd, pos.int().to(DEV), d_at=D, d_head=D + R, **kw)
    _close(qd.view(T, H, D + R)[..., D:], want, dtype, f32=5e-5)
    assert torch.equal(qd.view(T, H, D + R)[..., :D].cpu(), q.view(T, H, D + R)[..., :D])


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("H,D,R,V,C,bs", LAT)
def test_absorbed_latent_attention(H, D, R, V, C, bs, dtype):
    """Decode rows over contexts of very different length, one planted row among hundreds; split and unsplit."""
    g, W, scale = _gen(H + C), C + R, 0.1
    lens = [1, 700, 64, 65, 0, 333, 128]
    tab, blocks = _paged(lens, bs)
    pool = torch.zeros(blocks, 1, bs, W, dtype=dtype)
    rows, q = [], (torch.randn(len(lens), H, W, generator=g) * (12 / W ** 0.5)).to(dtype)
    for s, n in enumerate(lens):
        r = torch.randn(n, W, generator=g).to(dtype)
        if n > 5:
            r[n // 3] = (q[s, 0] * (100 / float(q[s, 0].float().pow(2).sum()))).to(dtype)      # head 0: a score of 10 more
        rows.append(r)
        _fill(pool, tab, s, r[:, None])
    want = torch.zeros(len(lens), H, C, dtype=torch.float64)
    for s, n in enumerate(lens):
        if n:
            want[s] = torch.softmax(q[s].double() @ rows[s].double().T * scale, -1) @ rows[s][:, :C].double()
    kv = KVLayer(pool.to(DEV), pool[..., :0].to(DEV), None, None, bs)
    big = torch.cat([q] * 30).reshape(-1, H * W).to(DEV)                   # more rows than SMs: no split
    for form in (0, 1):                                                    # tcgen05 where it applies; mma.sync
        for max_len in (100, 400, 5000):
            out = torch.full((len(lens), H * C), 9.0, dtype=dtype, device=DEV)
            latent.latent_attention(q.reshape(-1, H * W).to(DEV), kv, tab.to(DEV), _i32(lens), None, out, H=H, C=C, scale=scale,
                                    max_len=max_len, form=form)
            _close(out.view(-1, H, C), want, dtype, f32=5e-5)
        out = torch.empty(big.shape[0], H * C, dtype=dtype, device=DEV)
        latent.latent_attention(big, kv, tab.repeat(30, 1).to(DEV), _i32(lens * 30), None, out, H=H, C=C, scale=scale, max_len=700, form=form)
        _close(out.view(30, -1, H, C), want.expand(30, -1, -1, -1), dtype, f32=5e-5)
    assert _lib.read_status(torch.device(DEV, 0)) == 0


def test_latent_decode_follows_growing_scores():
    """Scores that grow along the context by far more than the lazy rescaling's threshold, and fall again."""
    H, C, R, n = 16, 128, 64, 1000
    W, g = C + R, _gen(1)
    tab, blocks = _paged([n], 16)
    rows, q = torch.randn(n, W, generator=g), torch.zeros(1, H, W)
    rows[:, 0] = 40 * torch.sin(torch.arange(n) / 150.0) + torch.arange(n) / 50.0
    q[:, :, 0] = torch.linspace(-1, 1, H)
    rows, q = rows.to(BF16), q.to(BF16)
    pool = torch.zeros(blocks, 1, 16, W, dtype=BF16)
    _fill(pool, tab, 0, rows[:, None])
    want = torch.softmax(q[0].double() @ rows.double().T, -1) @ rows[:, :C].double()
    kv = KVLayer(pool.to(DEV), pool[..., :0].to(DEV), None, None, 16)
    for form in (0, 1):
        for max_len in (128, 1000):
            out = torch.empty(1, H * C, dtype=BF16, device=DEV)
            latent.latent_attention(q.view(1, -1).to(DEV), kv, tab.to(DEV), _i32([n]), None, out, H=H, C=C, scale=1.0, max_len=max_len, form=form)
            _close(out.view(H, C), want, BF16)


@pytest.mark.parametrize("H,D,R,V,C,bs", [x for x in LAT if x[4] % 8 == 0])
def test_expanded_latent_attention(H, D, R, V, C, bs):
    """Prompt portions against gathered rows: keys [W_uk c | shared part] and values as two dense matrices."""
    g, W, scale = _gen(D), C + R, 2.0 / (D + R)
    lens, qlens = [300, 129, 17, 260, 64], [300, 2, 17, 140, 1]
    tab, blocks = _paged(lens, bs)
    pool = torch.zeros(blocks, 1, bs, W, dtype=BF16)
    rows = [torch.randn(n, W, generator=g).to(BF16) for n in lens]
    for s, r in enumerate(rows):
        _fill(pool, tab, s, r[:, None])
    kv = KVLayer(pool.to(DEV), pool[..., :0].to(DEV), None, None, bs)
    starts = [0]
    for n in lens:
        starts.append(starts[-1] + n)
    ctx = latent.latent_gather(kv, tab.to(DEV), _i32(starts), starts[-1])
    assert torch.equal(ctx.cpu(), torch.cat(rows))
    kn, v = (torch.randn(starts[-1], H, d, generator=g).to(BF16) for d in (D, V))
    q = torch.randn(sum(qlens), H, D + R, generator=g).to(BF16)
    out = torch.full((sum(qlens), H * V + 8), 9.0, dtype=BF16, device=DEV)
    cu, want = [0], []
    for s, (n, ql) in enumerate(zip(lens, qlens)):
        sl = slice(starts[s], starts[s + 1])
        k = torch.cat([kn[sl], rows[s][:, None, C:].expand(n, H, R)], -1).double()
        sc = torch.einsum("qhd,khd->hqk", q[cu[-1]:cu[-1] + ql].double(), k) * scale
        want.append(O.attend(sc, O.causal_mask(n)[n - ql:], v[sl].double().permute(1, 0, 2)).permute(1, 0, 2).reshape(ql, H * V))
        cu.append(cu[-1] + ql)
    qd = q.reshape(-1, H * (D + R)).to(DEV)
    kw = dict(D=D, R=R, V=V, scale=scale, max_q_len=300)
    h = max(1, H // 2)
    for h0, h1 in ((0, h), (h, H)):                                        # two groups of heads into column slices
        if h1 > h0:
            latent.latent_prefill(qd[:, h0 * (D + R):h1 * (D + R)], kn[:, h0:h1].reshape(-1, (h1 - h0) * D).to(DEV), ctx[:, C:],
                                  v[:, h0:h1].reshape(-1, (h1 - h0) * V).to(DEV), _i32(cu), _i32(lens), _i32(starts),
                                  out[:, h0 * V:h1 * V], H=h1 - h0, **kw)
    _close(out[:, :H * V], torch.cat(want), BF16)
    assert (out[:, H * V:] == 9.0).all() and _lib.read_status(torch.device(DEV, 0)) == 0


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
def test_mixed_batches_on_reused_pages(dtype):
    raw = O.CONFIGS["mixed"]
    t = O.random_tensors(raw, seed=5)
    lengths = [150, 7, 83, 1, 70, 18, 2, 141, 33]
    seqs = [tokens_for(raw, n, 20 + i) for i, n in enumerate(lengths)]
    eng = llm_for(raw, t, DEV, dtype, num_blocks=26, max_model_len=416).engine
    for got, s in zip(run_mixed(eng, seqs, interleave(lengths, [[50, 2, 1], [1], [5, 1, 1, 29], [3, 2]])), seqs):
        assert _check(raw, t, s, dtype)(got)
    assert eng.bm.num_free == 26


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_long_decoding_across_chunks_and_pages(name, dtype):
    raw = O.CONFIGS[name]
    t = O.random_tensors(raw, seed=8)
    toks = tokens_for(raw, 640, 11)
    eng = llm_for(raw, t, DEV, dtype).engine
    assert _check(raw, t, toks, dtype)(run_alone(eng, toks, [390] + [1] * 250))


def test_the_same_logits_however_the_prompt_is_cut():
    """bf16: portions differ from the whole prompt by rounding only (the two forms of the latent attention included)."""
    raw = O.CONFIGS["wide"]
    t = O.random_tensors(raw, seed=4)
    toks = tokens_for(raw, 300, 2)
    eng = llm_for(raw, t, DEV, BF16).engine
    whole = run_alone(eng, toks, [300])
    for sizes in ([2], [130, 1, 1, 40], [1]):
        assert worst(run_alone(eng, toks, sizes), whole.double()) < 0.03


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
            assert (lg.amax(-1) - lg.gather(1, torch.tensor(gen)[:, None])[:, 0]).max() < 0.35


def test_decode_steps_replay_graphs():
    raw = O.CONFIGS["mixed"]
    llm = llm_for(raw, O.random_tensors(raw, seed=9), DEV, BF16)
    sp = SamplingParams(max_tokens=8, temperature=0.0, ignore_eos=True)
    llm.generate(prompt_token_ids=[tokens_for(raw, 20, 1), tokens_for(raw, 9, 2)], sampling_params=sp)
    assert llm.engine._graphs and llm.engine.stats["decode_steps"] > 0
