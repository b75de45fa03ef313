"""Vavadra at sizes that resemble a real model's layers (random weights), beside the framework's closest existing model at
equal size: the Qwen3-Next layout (Gated DeltaNet and gated attention layers, mixture of experts with a shared expert), the
same widths, heads, experts and number of layers.

    python bench.py --design vavadra            # engine throughput of both and kernel times, one JSON line each

Kernel times: CUDA events, median of 9 after 3 warm-ups, a 256 MB write between iterations; each new kernel stands beside
the kernel (or chain of kernels) that has its role in the closest model or, for the latent layers, in a model of latent
attention without window and sink, both with their share of the measured copy bandwidth or tensor-core peak
(``MEASURED_PEAKS.json``)."""
from __future__ import annotations

import json

import torch

from .design_common import DEV, VOCAB, Table, engine_rates, peaks

SIZES = {
    # width, groups of [delta x2, latent, differential] layers, heads x 128, key heads, experts, their ff, chosen, identity experts
    "w2048": dict(width=2048, groups=2, heads=16, kv=4, dkv=8, experts=64, ff=768, top=6, identity=4, shared=1536, kv_rank=512),
    "w4096": dict(width=4096, groups=1, heads=32, kv=8, dkv=16, experts=32, ff=1536, top=4, identity=2, shared=3072, kv_rank=512),
}
DIM, ROT, SPAN = 128, 64, 512           # value width of every head, rotated part of the latent heads, chunk and window


def vavadra_llm(s, ecfg):
    from mlxcel_b200.config import ModelConfig
    from mlxcel_b200.llm import LLM
    from mlxcel_b200.models.vavadra import random_vavadra_weights
    mlp = dict(kind="moe", expert=dict(ff=s["ff"], limit=7.0), shared=dict(ff=s["shared"], limit=7.0),
               router=dict(experts=s["experts"], identity=s["identity"], top=s["top"], scale=2.5))
    delta = dict(type="delta", mlp=mlp, mixer=dict(heads=s["heads"], kv_heads=s["dkv"], dim=DIM, vdim=DIM, conv=4))
    lat = dict(type="latent_attention", mlp=mlp, mixer=dict(heads=s["heads"], dim=DIM, rot_dim=ROT, vdim=DIM, kv_rank=s["kv_rank"],
                                                            scale=(DIM + ROT) ** -0.5, mask=dict(size=SPAN), rot=dict(dims=ROT, base=1e6)))
    att = dict(type="attention", mlp=mlp, mixer=dict(heads=s["heads"], kv_heads=s["kv"], dim=DIM // 2, vdim=DIM, scale=(DIM // 2) ** -0.5, diff=0.7,
                                                     mask=dict(size=SPAN)))
    cfg = ModelConfig.from_dict(dict(architecture="Vavadra", vocab=VOCAB, width=s["width"], layers=[delta, delta, lat, att] * s["groups"],
                                     loop=None, embedding=dict(scale=1.0), norm=dict(eps=1e-6), logit_scale=1.0))
    return LLM(cfg, random_vavadra_weights(cfg, device=DEV), ecfg)


def closest_llm(s, ecfg):
    from mlxcel_b200.config import ModelConfig
    from mlxcel_b200.llm import LLM
    from mlxcel_b200.models.gdn import GdnLayerWeights, gdn_dims
    from mlxcel_b200.models.hybrid import HybridBlock, HybridWeights
    from mlxcel_b200.models.weights import LayerWeights
    W, E, I, n = s["width"], s["experts"], s["ff"], 4 * s["groups"]
    cfg = ModelConfig.from_dict(dict(
        model_type="qwen3_next", vocab_size=VOCAB, hidden_size=W, num_hidden_layers=n, num_attention_heads=s["heads"],
        num_key_value_heads=s["kv"], head_dim=DIM, intermediate_size=I, num_experts=E, num_experts_per_tok=s["top"], moe_intermediate_size=I,
        layer_types=(["linear_attention"] * 2 + ["full_attention"] * 2) * s["groups"], linear_num_key_heads=s["dkv"],
        linear_num_value_heads=s["heads"], linear_key_head_dim=DIM, linear_value_head_dim=DIM, linear_conv_kernel_dim=4,
        rms_norm_eps=1e-6, rope_theta=1e7, partial_rotary_factor=0.25))
    cfg.num_experts_per_tok = s["top"]
    g = torch.Generator(device=DEV).manual_seed(0)
    r = lambda *sh: (torch.randn(*sh, generator=g, device=DEV) * sh[-1] ** -0.5).to(torch.bfloat16)     # noqa: E731
    one = lambda d: torch.ones(d, dtype=torch.bfloat16, device=DEV)                                     # noqa: E731
    d = gdn_dims(cfg)
    blocks, attn = [], []
    for i in range(n):
        if i % 4 < 2:
            blocks.append(HybridBlock("gdn", one(W), mamba=GdnLayerWeights(
                norm=one(W), in_proj=r(d["conv_dim"] + d["value_dim"], W), in_proj_ba=r(2 * d["Hv"], W),
                conv_w=torch.randn(d["conv_dim"], 4, generator=g, device=DEV) * 0.3, dt_bias=torch.zeros(d["Hv"], device=DEV),
                A_log=torch.zeros(d["Hv"], device=DEV), gnorm=one(DIM), out_proj=r(W, d["value_dim"]))))
        else:
            lw = LayerWeights(ln1=one(W), ln2=one(W), wqkv=r((s["heads"] + 2 * s["kv"]) * DIM, W), wo=r(W, s["heads"] * DIM),
                              q_norm=one(DIM), k_norm=one(DIM))
            attn.append(lw)
            blocks.append(HybridBlock("attention", lw.ln1, attn=lw, out_gate=r(s["heads"] * DIM, W)))
        blocks.append(HybridBlock("moe", one(W), moe=LayerWeights(
            ln1=one(W), ln2=one(W), wqkv=None, wo=None, router_w=r(E, W), experts_gate_up=r(E, 2 * I, W), experts_down=r(E, W, I),
            shared_gate_up=r(2 * s["shared"], W), shared_down=r(W, s["shared"]), shared_gate=r(1, W))))
    w = HybridWeights(embed=r(VOCAB, W), blocks=blocks, final_norm=one(W), lm_head=r(VOCAB, W), layers=attn)
    return LLM(cfg, w, ecfg)


def kernel_rows(s, rows=64, ctx=1024, pieces=8, piece=1024):
    from mlxcel_b200 import ops
    from mlxcel_b200.ops import KVLayer, _lib, gated_delta, latent, moe, recurrent as R, stream
    W, Hq, Hkv, H, G, C = s["width"], s["heads"], s["kv"], s["heads"], s["dkv"], s["kv_rank"]
    E, I, top = s["experts"], s["ff"], s["top"]
    bf = lambda *sh: torch.randn(*sh, device=DEV).to(torch.bfloat16)                       # noqa: E731
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=DEV)                         # noqa: E731
    f32 = lambda *sh: torch.randn(*sh, device=DEV)                                         # noqa: E731
    empty = lambda *sh: torch.empty(*sh, dtype=torch.bfloat16, device=DEV)                 # noqa: E731
    table = Table()
    add = table.add
    T, bs, D = pieces * piece, 16, DIM
    # ---- row kernels and the mixture of experts (prefill and decode rows)
    gu, dn = bf(E, 2 * I, W), bf(E, W, I)
    for n in (rows, T):
        h, y, w, x, wb = f32(n, W), bf(n, W), f32(W), bf(n, W), torch.ones(W, dtype=torch.bfloat16, device=DEV)
        add(f"norm and residual, {n} rows", "hbm", ("stream_norm", lambda: stream.stream_norm(h, y, None, None, w, 1e-6, 0.0)), n * W * 12,
            ("add_rmsnorm", lambda: ops.add_rmsnorm(y, x, wb, 1e-6)), n * W * 8)
        lg, corr = f32(n, E + s["identity"]), f32(E + s["identity"]) * 0.01
        lb = lg[:, :E].to(torch.bfloat16).contiguous()
        add(f"choice of experts, {n} rows", "hbm", ("moe_route_choice", lambda: moe.route_choice(lg, corr, top, 2.5)),
            n * ((E + s["identity"]) * 4 + top * 8), ("moe_route", lambda: moe.route(lb, top, "softmax_topk", True)), n * (E * 2 + top * 8))
        ids, wts = moe.route_choice(lg, corr, top, 2.5)
        ids0, _ = moe.route(lb, top, "softmax_topk", True)
        experts_io = min(E, n * top) * 3 * I * W * 2 + n * top * (3 * W + 2 * I) * 2
        kind, work = ("hbm", experts_io) if n == rows else ("tensor", n * top * 6 * I * W)
        real = int((ids < E).sum()) / ids.numel()
        add(f"experts, {n} rows (alignment, gather, grouped GEMMs)", kind,
            ("expert_rows", lambda: moe.expert_rows(x, ids, wts, gu, dn, 1.702, 7.0)), work * (1 if n == rows else real),
            ("moe_experts (with its combine)", lambda: moe.moe_experts(x, ids0, wts, gu, dn, I, "silu")), work)
        m = moe.expert_rows(x, ids, wts, gu, dn, 1.702, 7.0)
        m.shared = y
        pair, total, inv = m.inv.clone(), i32([n * top]), torch.empty(n * top, dtype=torch.int32, device=DEV)
        pair[:] = torch.arange(n * top, dtype=torch.int32, device=DEV)
        out, lib = empty(n, W), _lib.load()

        def combine_chain():
            lib.mx_moe_combine_n(m.y.data_ptr(), pair.data_ptr(), total.data_ptr(), inv.data_ptr(), wts.data_ptr(), out.data_ptr(), x.data_ptr(), n, top,
                                 W, n * top, 0, _lib.stream())
            ops.add_rmsnorm(y, out, wb, 1e-6)
        add(f"sum of the experts, residual and norm, {n} rows", "hbm",
            ("stream_sum", lambda: stream.stream_norm(h, None, None, None, w, 1e-6, 0.0, dtype=torch.bfloat16, moe=m)), n * W * (2 * top + 12),
            ("moe_combine + add_rmsnorm", combine_chain), n * W * (2 * top + 12))
        del h, y, x, m, out
        pos, slots = torch.arange(n, dtype=torch.int32, device=DEV), torch.arange(n, dtype=torch.int32, device=DEV)
        nb = n // bs + 1
        kv = KVLayer(empty(nb, Hkv, bs, D), empty(nb, Hkv, bs, D), None, None, bs)
        qkv, inv_f = bf(n, (Hq + 2 * Hkv) * D), f32(D // 2)
        add(f"append of keys and values, {n} rows", "hbm",
            ("qk_norm_append (no norm)", lambda: stream.qk_norm_append(qkv, slots, kv, Hq=Hq, Hkv=Hkv, Dk=D, Dv=D, q_norm=None, k_norm=None, eps=1e-6)),
            n * D * 2 * 4 * Hkv,
            ("rope_append", lambda: ops.rope_append(qkv, pos, slots, inv_f, kv, Hq=Hq, Hkv=Hkv, D=D, rot_dim=D, q_norm_w=wb[:D], k_norm_w=wb[:D])),
            n * D * 2 * (2 * Hq + 4 * Hkv))
        del qkv, kv
        ld = H * (D + ROT) + C + ROT
        a, pool = bf(n, ld), KVLayer(empty(nb, 1, bs, C + ROT), empty(nb, 1, bs, 0), None, None, bs)
        ir, cn = f32(ROT // 2), f32(C)
        both = lambda adj: (lambda: latent.latent_append(a[:, H * (D + ROT):], pos, slots, pool, Q=0, C=C, R=ROT, inv_freq=ir, mscale=1.0,   # noqa: E731
                                                         q_norm=None, c_norm=cn, eps=1e-6, adjacent=adj))
        add(f"latent norm, rotation and append, {n} rows", "hbm", ("latent_append (neighbours)", both(True)), n * (C + ROT) * 4,
            ("latent_append (halves)", both(False)))
        turn = lambda adj: (lambda: latent.latent_q_rope(a, a, pos, H=H, q_at=D, q_head=D + ROT, d_at=D, d_head=D + ROT, inv_freq=ir,   # noqa: E731
                                                         mscale=1.0, adjacent=adj))
        add(f"query rotation, {n} rows", "hbm", ("latent_q_rope (neighbours)", turn(True)), n * H * ROT * 4, ("latent_q_rope (halves)", turn(False)))
        del a, pool
    del gu, dn
    # ---- differential attention; the context is one chunk, so both kernels have the same keys and values
    nb = rows * ctx // bs
    kv = KVLayer(bf(nb, Hkv, bs, D), bf(nb, Hkv, bs, D), None, None, bs)
    tables, lens = torch.randperm(nb, device=DEV).to(torch.int32).view(rows, -1), i32([ctx] * rows)
    qd, o = bf(rows, Hq * D), empty(rows, Hq * D)
    geo = dict(Hq=Hq, Hkv=Hkv, Dk=D, Dv=D, scale=0.125, chunk=ctx, diff=(0.7, 0.3, 1e-6))
    pgeo = dict(Hq=Hq, Hkv=Hkv, D=D, scale=D ** -0.5)
    add(f"attention decode, {rows} x {ctx}", "hbm",
        ("paged_decode_mma (two maps, chunk)", lambda: stream.paged_attention(qd, kv, tables, lens, None, o, max_q_len=1, max_len=ctx, **geo)),
        rows * ctx * Hkv * D * 4, ("paged_decode_mma", lambda: ops.paged_decode(qd, kv, tables, lens, max_len=ctx, out=o, **pgeo)))
    q, op = bf(T, Hq * D), empty(T, Hq * D)
    cu, pl, pt = i32([i * piece for i in range(pieces + 1)]), i32([piece] * pieces), tables[:pieces]
    pairs = pieces * Hq * piece * piece / 2
    add(f"attention prefill, {pieces} x {piece}", "tensor",
        ("paged_prefill_tc (two maps, chunk)", lambda: stream.paged_attention(q, kv, pt, pl, cu, op, max_q_len=piece, **geo)), pairs * 2 * (D + 2 * D),
        ("paged_prefill_tc", lambda: ops.paged_prefill(q, kv, pt, cu, pl, max_q_len=piece, out=op, **pgeo)), pairs * 2 * (D + D))
    del q, qd, kv
    # ---- latent attention: a window of half the context against the whole of a context that long
    Wd, win = C + ROT, ctx // 2
    pool = KVLayer(bf(nb, 1, bs, Wd), empty(nb, 1, bs, 0), None, None, bs)
    qa, ol, sinks, half = bf(rows, H * Wd), empty(rows, H * C), f32(H), i32([win] * rows)
    add(f"latent attention decode, {rows} x {win} tokens", "hbm",
        ("latent_decode (window, sink)", lambda: latent.latent_attention(qa, pool, tables, lens, None, ol, H=H, C=C, scale=0.1, max_len=ctx,
                                                                         window=win, sinks=sinks)), rows * win * Wd * 2,
        ("latent_decode", lambda: latent.latent_attention(qa, pool, tables, half, None, ol, H=H, C=C, scale=0.1, max_len=win)))
    ctxb = latent.latent_gather(pool, pt, cu, T)
    q, kn, v, op = bf(T, H * (D + ROT)), bf(T, H * D), bf(T, H * D), empty(T, H * D)
    seen = pieces * H * (piece * win - win * win / 2)
    pre = lambda **kw: (lambda: latent.latent_prefill(q, kn, ctxb[:, C:], v, cu, pl, cu, op, H=H, D=D, R=ROT, V=D, scale=0.1, max_q_len=piece, **kw))   # noqa: E731
    add(f"latent attention prefill, {pieces} x {piece}", "tensor", ("latent_prefill (window, sink)", pre(window=win, sinks=sinks)),
        seen * (2 * D + ROT) * 2, ("latent_prefill", pre()), pairs * (2 * D + ROT) * 2)
    del q, kn, v, op, ctxb, pool
    # ---- gated delta rule
    ch = 2 * G * D + H * D
    conv, vec, nw = f32(ch, 4) * 0.3, f32(H) * 0.1, f32(D)
    memory, tail = torch.zeros(rows, H, D, D, device=DEV), torch.zeros(rows, 3, ch, device=DEV)
    proj, rates = bf(rows, ch + H * D), f32(rows, 2 * H)
    sl, one, z0 = torch.arange(rows, dtype=torch.int32, device=DEV), torch.arange(rows + 1, dtype=torch.int32, device=DEV), i32([0] * rows)
    gq, gv, gg, gb = bf(rows, H, D), bf(rows, H, D), -f32(rows, H).abs(), torch.rand(rows, H, device=DEV)

    def gdn_chain():
        R.causal_conv_varlen(proj[:, :ch], tail, sl, one, z0, conv, None, True, 1)
        R.gated_delta_update(memory, gq, gq, gv, gg, gb)
    args = (conv, vec, vec, nw, memory, tail)
    add(f"recurrence decode, {rows} rows", "hbm",
        ("gated_step (convolution, rates, recurrence, norm, gate)", lambda: gated_delta.gated_delta(proj, rates, *args, sl, one, z0, G=G, norm_eps=1e-6,
                                                                                                    n_short=rows)), rows * H * D * D * 8,
        ("conv + gated_delta (state gathered, norm and gate left out)", gdn_chain))
    HD, Rk = H * D, 64
    offs, w2, wide = tuple(i * HD for i in range(6)), bf(HD, Rk), f32(HD)
    proj2, projp, ratesp = bf(T, 5 * HD + Rk), bf(T, ch + H * D), f32(T, 2 * H)
    st, flops = torch.zeros(pieces, H, D, D, device=DEV), T * H * D * D * 7
    add(f"recurrence prefill, {pieces} x {piece} (7 and 8 flops per state element and token; fp32 SIMT peak is 1/20 of the tensor peak)", "tensor",
        ("gated_prep + gated_scan + gated_post", lambda: gated_delta.gated_delta(projp, ratesp, *args, sl[:pieces], cu, z0[:pieces], G=G, norm_eps=1e-6)),
        flops, ("delta_prep + delta_scan + delta_post (general delta rule; the closest model's runs token by token)",
                lambda: stream.delta_rule(proj2, offs, w2, wide, wide, wide, st, sl[:pieces], cu, z0[:pieces], D=D, norm_eps=1e-6)), T * H * D * D * 8)
    return table.rows


def run() -> None:
    how = peaks()[2]
    for name, s in SIZES.items():
        for k in kernel_rows(s):
            print(json.dumps(dict(design="vavadra", size=name, peaks=how, **k)), flush=True)
        torch.cuda.empty_cache()
        ours = engine_rates(vavadra_llm, s)
        ref = engine_rates(closest_llm, s)
        print(json.dumps(dict(design="vavadra", size=name, layers=4 * s["groups"], engine=ours, closest="qwen3_next layout, mixture of experts",
                              closest_engine=ref)), flush=True)
