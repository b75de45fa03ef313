"""Govopel at sizes that resemble a real model's layers (random weights), beside the framework's closest existing model at
equal size: the DeepSeek layout (multi-head latent attention in every layer, per-head keys and values in the pool), dense
feed-forward of equal width, the same number of layers.

    python bench.py --design govopel            # engine throughput of both and kernel times, one JSON line each

Kernel times: CUDA events, median of 9 after 3 warm-ups, a 256 MB write between iterations; each new kernel stands beside
the kernel (or chain of operations) that has its role in the closest model or, for the chunked layers, in the Llama layout,
both with their share of the measured copy bandwidth or tensor-core peak (``MEASURED_PEAKS.json``)."""
from __future__ import annotations

import json

import torch

from .design_common import DEV, VOCAB, Table, engine_rates, peaks

SIZES = {
    # width, ff, groups of [latent x2, chunked x2] layers, heads x 128, key heads of the chunked layers, latent ranks
    "w2048": dict(width=2048, ff=5632, groups=4, heads=16, kv=4, q_rank=768, kv_rank=512),
    "w4096": dict(width=4096, ff=11264, groups=2, heads=32, kv=8, q_rank=1536, kv_rank=512),
}
DIM, ROT, CHUNK = 128, 64, 512


def govopel_llm(s, ecfg):
    from mlxcel_b200.config import ModelConfig
    from mlxcel_b200.llm import LLM
    from mlxcel_b200.models.govopel import random_govopel_weights
    mlp = dict(kind="dense", ff=s["ff"], limit=7.0)
    lat = dict(type="latent_attention", mlp=mlp, mixer=dict(heads=s["heads"], dim=DIM, rot_dim=ROT, vdim=DIM, q_rank=s["q_rank"],
                                                            kv_rank=s["kv_rank"], scale=(DIM + ROT) ** -0.5, rot=dict(dims=ROT, base=1e6)))
    att = dict(type="attention", mlp=mlp, mixer=dict(heads=s["heads"], kv_heads=s["kv"], dim=DIM, vdim=DIM, scale=DIM ** -0.5, softcap=50.0,
                                                     mask=dict(size=CHUNK), rot=dict(dims=DIM, base=1e4, scaling=dict(
                                                         factor=4.0, original=4096, fast=32.0, slow=1.0))))
    cfg = ModelConfig.from_dict(dict(architecture="Govopel", vocab=VOCAB, width=s["width"], layers=[lat, lat, att, att] * s["groups"],
                                     norm=dict(eps=1e-6), logit_softcap=30.0))
    return LLM(cfg, random_govopel_weights(cfg, device=DEV), ecfg)


def closest_llm(s, ecfg):
    from mlxcel_b200.config import ModelConfig
    from mlxcel_b200.llm import LLM
    from mlxcel_b200.models.weights import LayerWeights, ModelWeights
    n, W, I, H = 4 * s["groups"], s["width"], s["ff"], s["heads"]
    cfg = ModelConfig.from_dict(dict(
        model_type="deepseek_v3", vocab_size=VOCAB, hidden_size=W, num_hidden_layers=n, num_attention_heads=H, num_key_value_heads=H,
        intermediate_size=I, n_routed_experts=None, first_k_dense_replace=n, q_lora_rank=s["q_rank"], kv_lora_rank=s["kv_rank"],
        qk_nope_head_dim=DIM, qk_rope_head_dim=ROT, v_head_dim=DIM, rms_norm_eps=1e-6, rope_theta=1e6, max_position_embeddings=8192,
        moe_intermediate_size=I))
    g = torch.Generator(device=DEV).manual_seed(0)
    r = lambda *sh: (torch.randn(*sh, generator=g, device=DEV) * sh[-1] ** -0.5).to(torch.bfloat16)     # noqa: E731
    one = lambda d: torch.ones(d, dtype=torch.bfloat16, device=DEV)                                     # noqa: E731
    layers = [LayerWeights(ln1=one(W), ln2=one(W), wqkv=None, wo=r(W, H * DIM), w_gate_up=r(2 * I, W), w_down=r(W, I), mla=dict(
        q_a=r(s["q_rank"], W), q_a_norm=one(s["q_rank"]), q_b=r(H * (DIM + ROT), s["q_rank"]), kv_a=r(s["kv_rank"] + ROT, W),
        kv_a_norm=one(s["kv_rank"]), kv_b=r(H * 2 * DIM, s["kv_rank"]))) for _ in range(n)]
    return LLM(cfg, ModelWeights(embed=r(VOCAB, W), layers=layers, final_norm=one(W), lm_head=r(VOCAB, W)), ecfg)


def kernel_rows(s, rows=64, ctx=1024, pieces=8, piece=1024):
    from mlxcel_b200 import ops
    from mlxcel_b200.ops import KVLayer, latent, reference as ref, stream
    W, Hq, Hkv, H, Q, C = s["width"], s["heads"], s["kv"], s["heads"], s["q_rank"], s["kv_rank"]
    bf = lambda *sh: torch.randn(*sh, device=DEV).to(torch.bfloat16)                       # noqa: E731
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=DEV)                         # noqa: E731
    f32 = lambda *sh: torch.randn(*sh, device=DEV)                                         # noqa: E731
    empty = lambda *sh: torch.empty(*sh, dtype=torch.bfloat16, device=DEV)                 # noqa: E731
    table = Table()
    add = table.add
    T, bs, D, R, E = pieces * piece, 16, DIM, ROT, C + ROT
    # ---- row kernels (prefill and decode rows)
    for n in (rows, T):
        h, y, w, x = f32(n, W), bf(n, W), f32(W), bf(n, W)
        wb = torch.ones(W, dtype=torch.bfloat16, device=DEV)
        add(f"norm and residual, {n} rows", "hbm", ("stream_norm", lambda: stream.stream_norm(h, y, w, None, None, 1e-6, 0.0, plain=True)),
            n * W * 12, ("add_rmsnorm", lambda: ops.add_rmsnorm(y, x, wb, 1e-6)), n * W * 8)
        del h, y, x
        pos, slots = torch.arange(n, dtype=torch.int32, device=DEV), torch.arange(n, dtype=torch.int32, device=DEV)
        nb = n // bs + 1
        kv = KVLayer(empty(nb, Hkv, bs, D), empty(nb, Hkv, bs, D), None, None, bs)
        q, qkv, inv = bf(n, (Hq + Hkv) * D), bf(n, (Hq + 2 * Hkv) * D), f32(D // 2)
        add(f"rotation, q/k norm and append, {n} rows", "hbm", ("rope_norm_append", lambda: stream.rope_norm_append(
            q, pos, slots, kv, Hq=Hq, Hkv=Hkv, Dk=D, Dv=D, inv_freq=inv, values_are_keys=True, eps=1e-6)), n * D * 2 * (2 * Hq + 3 * Hkv),
            ("rope_append (norm before)", lambda: ops.rope_append(qkv, pos, slots, inv, kv, Hq=Hq, Hkv=Hkv, D=D, rot_dim=D, q_norm_w=wb[:D],
                                                                  k_norm_w=wb[:D])), n * D * 2 * (2 * Hq + 4 * Hkv))
        del q, qkv, kv
        a, pool = bf(n, Q + E), KVLayer(empty(nb, 1, bs, E), empty(nb, 1, bs, 0), None, None, bs)
        ir, qn, cn = f32(R // 2), f32(Q), f32(C)

        def append_chain():
            ops.rmsnorm(a[:, :Q].contiguous(), wb[:Q], 1e-6, 0.0)
            c = ops.rmsnorm(a[:, Q:Q + C].contiguous(), wb[:C], 1e-6, 0.0)
            kr = ref.apply_rope(a[:, Q + C:].view(n, 1, R), pos, ir, R, False, 1.0)
            pool.k.view(-1, E).index_copy_(0, slots.long(), torch.cat([c, kr.view(n, R).to(c.dtype)], 1))
        if Q <= W and C <= W:
            add(f"latent norms, rotation and append, {n} rows", "hbm", ("latent_append", lambda: latent.latent_append(
                a, pos, slots, pool, Q=Q, C=C, R=R, inv_freq=ir, mscale=1.0, q_norm=qn, c_norm=cn, eps=1e-6)), n * (2 * Q + 2 * E) * 2,
                ("norm kernels and tensor operations", append_chain))
        ql = bf(n, H * (D + R))
        add(f"query rotation, {n} rows", "hbm", ("latent_q_rope", lambda: latent.latent_q_rope(
            ql, ql, pos, H=H, q_at=D, q_head=D + R, d_at=D, d_head=D + R, inv_freq=ir, mscale=1.0)), n * H * R * 4,
            ("tensor operations", lambda: ref.apply_rope(ql.view(n, H, D + R)[..., D:], pos, ir, R, False, 1.0)))
        del a, pool, ql
    lg = f32(rows, VOCAB)
    add(f"logit soft cap, {rows} rows", "hbm", ("softcap_rows", lambda: stream.softcap_(lg, 30.0)), rows * VOCAB * 8,
        ("tensor operations", lambda: torch.tanh(lg / 30.0) * 30.0))
    # ---- chunked attention; the context is one chunk, so both kernels have the same work
    nb = rows * ctx // bs
    kv = KVLayer(bf(nb, Hkv, bs, D), bf(nb, Hkv, bs, D), None, None, bs)
    tables, lens = torch.randperm(nb, device=DEV).to(torch.int32).view(rows, -1), i32([ctx] * rows)
    qd, o = bf(rows, Hq * D), empty(rows, Hq * D)
    geo = dict(Hq=Hq, Hkv=Hkv, Dk=D, Dv=D, scale=D ** -0.5, softcap=50.0)
    pgeo = dict(Hq=Hq, Hkv=Hkv, D=D, scale=D ** -0.5)
    add(f"chunked attention decode, {rows} x {ctx}", "hbm",
        ("paged_decode_mma (chunk, soft cap)", lambda: stream.paged_attention(qd, kv, tables, lens, None, o, max_q_len=1, max_len=ctx, chunk=ctx,
                                                                              **geo)), rows * ctx * Hkv * D * 4,
        ("paged_decode_mma", lambda: ops.paged_decode(qd, kv, tables, lens, max_len=ctx, out=o, **pgeo)))
    q, op = bf(T, Hq * D), empty(T, Hq * D)
    cu, pl, pt = i32([i * piece for i in range(pieces + 1)]), i32([piece] * pieces), tables[:pieces]
    add(f"chunked attention prefill, {pieces} x {piece}", "tensor",
        ("paged_prefill_tc (chunk, soft cap)", lambda: stream.paged_attention(q, kv, pt, pl, cu, op, max_q_len=piece, chunk=ctx, **geo)),
        pieces * Hq * D * 4 * (piece * piece / 2),
        ("paged_prefill_tc", lambda: ops.paged_prefill(q, kv, pt, cu, pl, max_q_len=piece, out=op, **pgeo)))
    del q, qd, kv
    # ---- latent attention
    pool = KVLayer(bf(nb, 1, bs, E), empty(nb, 1, bs, 0), None, None, bs)
    qa, ol = bf(rows, H * E), empty(rows, H * C)
    qd, wt, wv = bf(rows, H * (D + R)), bf(H, C, D), bf(H, D, C)
    add(f"query into latent space, {rows} rows", "hbm", ("batched GEMM", lambda: ops.batched_linear(qd, wt, qa, D + R, E)),
        H * C * D * 2 + rows * H * (D + C) * 2,
        ("fp32 einsum", lambda: torch.einsum("thn,hnl->thl", qd.view(rows, H, D + R)[..., :D].float(), wt.transpose(1, 2).float())))
    add(f"values out of latent space, {rows} rows", "hbm", ("batched GEMM", lambda: ops.batched_linear(ol, wv, o, C, D)),
        H * C * D * 2 + rows * H * (D + C) * 2,
        ("fp32 einsum", lambda: torch.einsum("thl,hvl->thv", ol.view(rows, H, C).float(), wv.float())))

    def latent_chain():
        c = pool.k[tables.long()].view(rows, -1, E).float()
        p = torch.softmax(torch.einsum("nhw,nsw->nhs", qa.view(rows, H, E).float(), c) * 0.1, -1)
        return torch.einsum("nhs,nsl->nhl", p, c[..., :C])
    add(f"latent attention decode, {rows} x {ctx}", "hbm",
        ("latent_decode", lambda: latent.latent_attention(qa, pool, tables, lens, None, ol, H=H, C=C, scale=0.1, max_len=ctx)), rows * ctx * E * 2,
        ("gathered rows, fp32 einsum", latent_chain))
    Dp = 256
    kx = KVLayer(bf(nb // 4, H, bs, Dp), bf(nb // 4, H, bs, Dp), None, None, bs)
    qx, ox, tx = bf(rows // 4, H * Dp), empty(rows // 4, H * Dp), torch.randperm(nb // 4, device=DEV).to(torch.int32).view(rows // 4, -1)
    add(f"latent attention decode, {rows // 4} x {ctx}, beside per-head keys and values", "hbm",
        ("latent_decode", lambda: latent.latent_attention(qa[:rows // 4], pool, tables[:rows // 4], lens[:rows // 4], None, ol[:rows // 4], H=H, C=C,
                                                          scale=0.1, max_len=ctx)), rows // 4 * ctx * E * 2,
        ("paged_decode, heads of 256", lambda: ops.paged_decode(qx, kx, tx, lens[:rows // 4], Hq=H, Hkv=H, D=Dp, scale=0.1, max_len=ctx, out=ox)),
        rows // 4 * ctx * H * (D + R + D) * 2)
    starts = cu
    ctxb = latent.latent_gather(pool, pt, starts, T)
    add(f"context gather, {T} rows", "hbm", ("latent_gather", lambda: latent.latent_gather(pool, pt, starts, T)), T * E * 4,
        ("index_select", lambda: pool.k.view(-1, bs * E).index_select(0, pt.reshape(-1))))
    q, kn, v, op = bf(T, H * (D + R)), bf(T, H * D), bf(T, H * D), empty(T, H * D)
    px, ptx, oxx = bf(T, H * Dp), tx[:pieces], empty(T, H * Dp)
    fl = pieces * H * (2 * D + R) * 2 * (piece * piece / 2)
    add(f"latent attention prefill, {pieces} x {piece}", "tensor",
        ("latent_prefill (tcgen05)", lambda: latent.latent_prefill(q, kn, ctxb[:, C:], v, cu, pl, starts, op, H=H, D=D, R=R, V=D, scale=0.1,
                                                                   max_q_len=piece)), fl,
        ("paged_prefill, heads of 256", lambda: ops.paged_prefill(px, kx, ptx, cu, pl, Hq=H, Hkv=H, D=Dp, scale=0.1, max_q_len=piece, out=oxx)))
    return table.rows


def run() -> None:
    how = peaks()[2]
    for name, s in SIZES.items():
        for k in kernel_rows(s):
            print(json.dumps(dict(design="govopel", size=name, peaks=how, **k)), flush=True)
        torch.cuda.empty_cache()
        ours = engine_rates(govopel_llm, s)
        ref = engine_rates(closest_llm, s)
        print(json.dumps(dict(design="govopel", size=name, layers=4 * s["groups"], engine=ours, closest="deepseek_v3 layout, dense",
                              closest_engine=ref)), flush=True)
