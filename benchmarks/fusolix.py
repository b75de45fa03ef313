"""Fusolix at sizes that resemble a real model's layers (random weights), beside the framework's closest existing model at
equal size: the Falcon-H1 layout (Mamba2 mixer and attention side by side, gated feed-forward), the same widths, heads, state
and number of layers.

    python bench.py --design fusolix            # engine throughput of both and kernel times, one JSON line each

Kernel times: CUDA events, median of 9 after 3 warm-ups, a 256 MB write between iterations; each new kernel stands beside
the kernel (or chain of kernels) that has its role in the closest model or, for the experts, in the framework's mixture of
experts, both with their share of the measured copy bandwidth or tensor-core peak (``MEASURED_PEAKS.json``)."""
from __future__ import annotations

import json

import torch

from .design_common import DEV, VOCAB, Table, engine_rates, peaks

SIZES = {
    # width, layers, attention heads x 128, key heads, retention heads x 128, dense ff; experts, their ff, chosen, groups, kept groups
    "w2048": dict(width=2048, layers=12, heads=16, kv=4, rheads=16, ff=5632, experts=64, eff=768, top=6, groups=8, keep=3),
    "w4096": dict(width=4096, layers=6, heads=32, kv=8, rheads=32, ff=11264, experts=32, eff=1536, top=4, groups=4, keep=2),
}
DIM, WINDOW, BLOCK, STREAMS, TAPS = 128, 512, 16, 4, 4


def fusolix_llm(s, ecfg):
    from mlxcel_b200.config import ModelConfig
    from mlxcel_b200.llm import LLM
    from mlxcel_b200.models.fusolix import random_fusolix_weights
    left = dict(heads=s["heads"], kv_heads=s["kv"], dim=DIM, vdim=DIM, scale=DIM ** -0.5, mask=dict(size=WINDOW, pool=BLOCK))
    right = dict(heads=s["rheads"], dim=DIM, vdim=DIM, rot=dict(dims=DIM, base=1e4), decay=[1 - 2.0 ** -(5 + 7 * i / s["rheads"]) for i in range(s["rheads"])])
    layer = dict(type="parallel", mixer=dict(left=left, right=right, left_scale=0.5, right_scale=0.5), mlp=dict(kind="dense", ff=s["ff"], limit=7.0))
    cfg = ModelConfig.from_dict(dict(architecture="Fusolix", vocab=VOCAB, width=s["width"], layers=[layer] * s["layers"], streams=STREAMS,
                                     canon=dict(taps=TAPS), embedding=dict(scale=1.0), norm=dict(eps=1e-6)))
    return LLM(cfg, random_fusolix_weights(cfg, device=DEV), ecfg)


def closest_llm(s, ecfg):
    from mlxcel_b200.config import ModelConfig
    from mlxcel_b200.llm import LLM
    from mlxcel_b200.models.hybrid import HybridBlock, HybridWeights
    from mlxcel_b200.models.mamba2 import Mamba2LayerWeights, mamba_dims
    from mlxcel_b200.models.weights import LayerWeights
    W, I, H = s["width"], s["ff"], s["rheads"]
    cfg = ModelConfig.from_dict(dict(
        model_type="falcon_h1", vocab_size=VOCAB, hidden_size=W, num_hidden_layers=s["layers"], num_attention_heads=s["heads"],
        num_key_value_heads=s["kv"], head_dim=DIM, intermediate_size=I, mamba_d_ssm=H * DIM, mamba_d_head=DIM, mamba_d_state=DIM, mamba_n_groups=1,
        mamba_d_conv=4, mamba_rms_norm=True, rms_norm_eps=1e-6, rope_theta=1e7, tie_word_embeddings=False))
    g = torch.Generator(device=DEV).manual_seed(0)
    r = lambda *sh: (torch.randn(*sh, generator=g, device=DEV) * sh[-1] ** -0.5).to(torch.bfloat16)     # noqa: E731
    one = lambda d: torch.ones(d, dtype=torch.bfloat16, device=DEV)                                     # noqa: E731
    d = mamba_dims(cfg)
    blocks, attn = [], []
    for _ in range(s["layers"]):
        mw = Mamba2LayerWeights(norm=one(W), in_proj=r(d["d_inner"] + d["conv_dim"] + d["heads"], W), conv_w=torch.randn(d["conv_dim"], 4, generator=g, device=DEV) * 0.3,
                                conv_b=torch.zeros(d["conv_dim"], device=DEV), dt_bias=torch.zeros(H, device=DEV) - 3, A_log=torch.zeros(H, device=DEV),
                                D=torch.ones(H, device=DEV), gnorm=one(d["d_inner"]), out_proj=r(W, d["d_inner"]))
        lw = LayerWeights(ln1=one(W), ln2=one(W), wqkv=r((s["heads"] + 2 * s["kv"]) * DIM, W), wo=r(W, s["heads"] * DIM))
        attn.append(lw)
        blocks.append(HybridBlock("parallel", one(W), mamba=mw, attn=lw))
        blocks.append(HybridBlock("mlp", one(W), up=r(2 * I, W), down=r(W, I), gated=True))
    return LLM(cfg, HybridWeights(embed=r(VOCAB, W), blocks=blocks, final_norm=one(W), lm_head=r(VOCAB, W), layers=attn), ecfg)


def kernel_rows(s, rows=64, ctx=8192, pieces=8, piece=1024):
    from mlxcel_b200 import ops
    from mlxcel_b200.ops import KVLayer, _lib, block_means, moe, recurrent as R, retention, stream, streams
    W, Hq, Hkv, H, S, K = s["width"], s["heads"], s["kv"], s["rheads"], STREAMS, TAPS
    E, I, top, D, bs = s["experts"], s["eff"], s["top"], DIM, 16
    bf = lambda *sh: torch.randn(*sh, device=DEV).to(torch.bfloat16)                       # noqa: E731
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=DEV)                         # noqa: E731
    f32 = lambda *sh: torch.randn(*sh, device=DEV)                                         # noqa: E731
    empty = lambda *sh: torch.empty(*sh, dtype=torch.bfloat16, device=DEV)                 # noqa: E731
    iota = lambda n: torch.arange(n, dtype=torch.int32, device=DEV)                        # noqa: E731
    table = Table()
    add = table.add
    T = pieces * piece
    around = lambda: streams.Sublayer(f32(S), f32(S), 0.2 * f32(S, S), f32(W), f32(W), f32(K, W))     # noqa: E731
    one_tok = (iota(rows), iota(rows + 1), i32([0] * rows), rows, 1)
    cu = i32([i * piece for i in range(pieces + 1)])
    prompt = (iota(pieces), cu, i32([0] * pieces), 0, piece)
    gu, dn = bf(E, 2 * I, W), bf(E, W, I)
    # ---- row kernels and the mixture of experts (prefill and decode rows)
    for n, batch in ((rows, one_tok), (T, prompt)):
        a, b, tail = around(), around(), torch.zeros(max(rows, pieces), K - 1, W, device=DEV)
        xs, y, x, wb = f32(n, S, W), bf(n, W), bf(n, W), torch.ones(W, dtype=torch.bfloat16, device=DEV)
        state = n * W * 8 * (K - 1) if n == rows else 0                       # (a portion's state is small change)
        name = "streams_step" if n == rows else "streams_step + streams_conv"
        add(f"streams, norm and convolution, {n} rows", "hbm",
            (name, lambda: streams.mix_streams(xs, a, y, None, b, 1e-6, torch.bfloat16, tail, batch)), n * W * (8 * S + 4) + state,
            ("add_rmsnorm", lambda: ops.add_rmsnorm(y, x, wb, 1e-6)), n * W * 8)
        add(f"sum of the streams, {n} rows", "hbm", ("streams_step", lambda: streams.sum_streams(xs, a, y, None, torch.bfloat16)), n * W * (4 * S + 6),
            ("add_rmsnorm", lambda: ops.add_rmsnorm(y, x, wb, 1e-6)), n * W * 8)
        lg = f32(n, E)
        lb = lg.to(torch.bfloat16).contiguous()
        add(f"choice of experts, {n} rows", "hbm", ("moe_route_choice (groups)", lambda: moe.route_choice(lg, None, top, 1.0, (s["groups"], s["keep"]), True)),
            n * (E * 4 + top * 8), ("moe_route", lambda: moe.route(lb, top, "softmax_topk", True)), n * (E * 2 + top * 8))
        ids, wts = moe.route_choice(lg, None, top, 1.0, (s["groups"], s["keep"]), True)
        kind, work = ("hbm", min(E, n * top) * 3 * I * W * 2 + n * top * (3 * W + 2 * I) * 2) if n == rows else ("tensor", n * top * 6 * I * W)
        add(f"experts, {n} rows (alignment, gather, grouped GEMMs)", kind,
            ("expert_rows (silu)", lambda: moe.expert_rows(x, ids, wts, gu, dn, 1.0, 0.0, act="silu")), work,
            ("moe_experts (with its combine)", lambda: moe.moe_experts(x, ids, wts, gu, dn, I, "silu")), work)
        m = moe.expert_rows(x, ids, wts, gu, dn, 1.0, 0.0, act="silu")
        pair, total, inv = torch.arange(n * top, dtype=torch.int32, device=DEV), i32([n * top]), torch.empty(n * top, dtype=torch.int32, device=DEV)
        out, lib = empty(n, W), _lib.load()

        def combine_chain():
            lib.mx_moe_combine_n(m.y.data_ptr(), pair.data_ptr(), total.data_ptr(), inv.data_ptr(), wts.data_ptr(), out.data_ptr(), x.data_ptr(), n, top,
                                 W, n * top, 0, _lib.stream())
            ops.add_rmsnorm(y, out, wb, 1e-6)
        add(f"sum of the experts, streams, norm and convolution, {n} rows", "hbm",
            (name, lambda: streams.mix_streams(xs, a, None, m, b, 1e-6, torch.bfloat16, tail, batch)), n * W * (8 * S + 2 + 2 * top) + state,
            ("moe_combine + add_rmsnorm", combine_chain), n * W * (2 * top + 12))
        flat = f32(n, W)
        add(f"final norm, {n} rows", "hbm", ("layer_norm_rows", lambda: streams.layer_norm(flat, b.norm_w, b.norm_b, 1e-6, torch.bfloat16)), n * W * 6,
            ("rmsnorm", lambda: ops.rmsnorm(y, wb, 1e-6)), n * W * 4)
        del xs, y, x, m, out, flat
        nb = n // bs + rows + 1
        kv = KVLayer(empty(nb, Hkv, bs, D), empty(nb, Hkv, bs, D), None, None, bs, 16, empty(nb, Hkv, 1, D), empty(nb, Hkv, 1, D), BLOCK)
        qkv, inv_f = bf(n, (Hq + 2 * Hkv) * D), f32(D // 2)
        pos = torch.full((n,), bs - 1, dtype=torch.int32, device=DEV) if n == rows else torch.cat([iota(piece)] * pieces)
        tabs = iota(rows)[:, None].contiguous() if n == rows else iota(T // bs).view(pieces, -1)
        slots = iota(rows) * bs + bs - 1 if n == rows else iota(n)
        ends = n if n == rows else n // BLOCK                                  # (every decode row ends a block here)
        add(f"append of keys, values and means, {n} rows", "hbm",
            ("kv_append_means", lambda: block_means.append(qkv, pos, slots, kv, tabs, None if n == rows else cu, Hq=Hq, Hkv=Hkv, Dk=D, Dv=D)),
            (n * 2 + (ends * (BLOCK + 1) if n == rows else n + ends)) * Hkv * D * 4,
            ("rope_append", lambda: ops.rope_append(qkv, pos, slots, inv_f, kv, Hq=Hq, Hkv=Hkv, D=D, rot_dim=D)), n * D * 2 * (2 * Hq + 4 * Hkv))
        del qkv, kv
    del gu, dn
    # ---- attention: a window and the means of 8 x its context against a context of as many keys
    nb = rows * ctx // bs
    kv = KVLayer(bf(nb, Hkv, bs, D), bf(nb, Hkv, bs, D), None, None, bs, 16, bf(nb, Hkv, 1, D), bf(nb, Hkv, 1, D), BLOCK)
    tables, lens = torch.randperm(nb, device=DEV).to(torch.int32).view(rows, -1), i32([ctx] * rows)
    seen = WINDOW + (ctx - WINDOW) // BLOCK
    q1, o, short = bf(rows, Hq * D), empty(rows, Hq * D), i32([seen] * rows)
    geo = dict(Hq=Hq, Hkv=Hkv, Dk=D, Dv=D, scale=D ** -0.5, window=WINDOW)
    pgeo = dict(Hq=Hq, Hkv=Hkv, D=D, scale=D ** -0.5)
    add(f"attention decode, {rows} x {ctx} ({seen} keys)", "hbm",
        ("paged_decode_mma (window, means)", lambda: stream.paged_attention(q1, kv, tables, lens, None, o, max_q_len=1, max_len=ctx, means=(None, 0), **geo)),
        rows * seen * Hkv * D * 4, ("paged_decode_mma", lambda: ops.paged_decode(q1, kv, tables, short, max_len=seen, out=o, **pgeo)))
    q, op, pl, pt = bf(T, Hq * D), empty(T, Hq * D), i32([ctx] * pieces), tables[:pieces]
    batch = type("B", (), dict(pf_cu_q_host=None, pf_starts=None, pf_context_lens=pl))()
    means = block_means.portion_means(batch, WINDOW, BLOCK)
    pairs = sum(WINDOW + (p + 1 - WINDOW) // BLOCK for p in range(ctx - piece, ctx)) * pieces * Hq
    add(f"attention prefill, {pieces} x {piece} behind {ctx - piece}", "tensor",
        ("gather_means + paged_prefill_tc (window, means)", lambda: stream.paged_attention(q, kv, pt, pl, cu, op, max_q_len=piece, means=means, **geo)),
        pairs * 4 * D, ("paged_prefill_tc (window of as many keys)", lambda: ops.paged_prefill(q, kv, pt, cu, pl, max_q_len=piece, out=op, window=1024, **pgeo)),
        pieces * Hq * piece * 1024 * 4 * D)
    add(f"gather of the means, {means[1]} rows", "hbm", ("gather_means", lambda: block_means.gather(kv, pt, *means)), means[1] * Hkv * D * 8,
        ("index_select", lambda: kv.k_mean.view(nb, -1).index_select(0, torch.arange(means[1], device=DEV))), means[1] * Hkv * D * 4)
    del q, q1, kv, op
    # ---- retention
    memory, inv, decay = torch.zeros(rows, H, D, D, device=DEV), f32(D // 2), torch.full((H,), 0.99, device=DEV)
    proj, out = bf(rows, 4 * H * D), empty(rows, H * D)
    state, conv_w, tail = torch.zeros(rows, H, D, D, device=DEV), f32(H * D + 2 * D, 4), torch.zeros(rows, 3, H * D + 2 * D, device=DEV)
    xbc, dt, A, z = bf(rows, H * D + 2 * D), bf(rows, H), -torch.rand(H, device=DEV), bf(rows, H * D)
    sl, one, z0, posd = one_tok[0], one_tok[1], one_tok[2], i32([5] * rows)

    def mamba(n, xbc, dt, z, slots, cu, reset, nd, longest):
        c = R.causal_conv_varlen(xbc, tail, slots, cu, reset, conv_w, None, True, longest)
        y = R.ssm_scan_varlen(state, slots, cu, reset, c[:, :H * D], dt, A, c[:, H * D:H * D + D], c[:, H * D + D:], n_short=nd)
        R.gated_rmsnorm(y, z, wz, 1e-6)
    wz = torch.ones(H * D, dtype=torch.bfloat16, device=DEV)
    add(f"recurrence decode, {rows} rows", "hbm",
        ("retention_step (rotation, recurrence, norm, gate)", lambda: retention.retention(proj, posd, inv, decay, memory, sl, one, z0, out, norm_eps=1e-6, n_short=rows)),
        rows * H * D * D * 8, ("conv + ssm_scan + gated_rmsnorm (Mamba2)", lambda: mamba(rows, xbc, dt, z, sl, one, z0, rows, 1)))
    projp, outp, posp = bf(T, 4 * H * D), empty(T, H * D), torch.cat([iota(piece)] * pieces)
    xbcp, dtp, zp = bf(T, H * D + 2 * D), bf(T, H), bf(T, H * D)
    sp, zr = iota(pieces), i32([0] * pieces)
    for n, c, nm in ((T, cu, f"{pieces} x {piece}"), (piece, cu[:2], f"1 x {piece}")):
        np_ = c.shape[0] - 1
        flops = n * H * D * D * 5
        add(f"recurrence prefill, {nm} (5 flops per state element and token, the sequential form's)", "tensor",
            ("retention", lambda: retention.retention(projp[:n], posp[:n], inv, decay, memory, sp[:np_], c, zr[:np_], outp[:n], norm_eps=1e-6)), flops,
            ("conv + ssm_scan + gated_rmsnorm (Mamba2)", lambda: mamba(n, xbcp[:n], dtp[:n], zp[:n], sp[:np_], c, zr[:np_], 0, piece)), flops)
    return table.rows


def run() -> None:
    how = peaks()[2]
    for name, s in SIZES.items():
        for k in kernel_rows(s):
            print(json.dumps(dict(design="fusolix", size=name, peaks=how, **k)), flush=True)
        torch.cuda.empty_cache()
        ours = engine_rates(fusolix_llm, s)
        ref = engine_rates(closest_llm, s)
        print(json.dumps(dict(design="fusolix", size=name, layers=s["layers"], engine=ours, closest="falcon_h1 layout", closest_engine=ref)), flush=True)
