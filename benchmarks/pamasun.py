"""Pamasun at sizes that resemble a real model's layers (random weights), beside the framework's closest
existing model at equal size: the Qwen3-Next stack (Gated DeltaNet + gated attention with per-head q/k
norms), dense feed-forward of equal parameter count.

    python bench.py --design pamasun            # engine throughput of both and kernel times, one JSON line each

Kernel times: CUDA events, median of 9 after 3 warm-ups, a 256 MB write between iterations; each new kernel
stands beside the kernel that has its role in the closest model, both with their share of the measured copy
bandwidth or tensor-core peak (``MEASURED_PEAKS.json``)."""
from __future__ import annotations

import json

import torch

from .design_common import DEV, VOCAB, Table, engine_rates, peaks

SIZES = {
    # width, ff, layers of [delta x3, attention] groups, query / kv heads x 128, delta heads x 128
    "w2048": dict(width=2048, ff=8192, groups=4, heads=16, kv=4, delta=16),
    "w4096": dict(width=4096, ff=16384, groups=2, heads=32, kv=8, delta=32),
}
DIM = 128


def pamasun_llm(s, ecfg):
    from mlxcel_b200.config import ModelConfig
    from mlxcel_b200.llm import LLM
    from mlxcel_b200.models.pamasun import random_pamasun_weights
    delta = dict(type="general_delta", mixer=dict(heads=s["delta"], dim=DIM), mlp=dict(kind="dense", ff=s["ff"]))
    attn = dict(type="attention", mixer=dict(heads=s["heads"], kv_heads=s["kv"], dim=DIM, vdim=DIM, scale=DIM ** -0.5),
                mlp=dict(kind="dense", ff=s["ff"]))
    cfg = ModelConfig.from_dict(dict(architecture="Pamasun", vocab=VOCAB, width=s["width"], layers=[delta, delta, delta, attn] * s["groups"],
                                     loop=None, embedding=dict(scale=1.0), norm=dict(eps=1e-6)))
    return LLM(cfg, random_pamasun_weights(cfg, device=DEV, rank=64), ecfg)


def closest_llm(s, ecfg):
    """Qwen3-Next layout with the same mixers' sizes; SwiGLU width 2/3 of ff (equal parameters)."""
    from mlxcel_b200.config import ModelConfig
    from mlxcel_b200.llm import LLM
    from mlxcel_b200.models.gdn import GdnLayerWeights, gdn_dims
    from mlxcel_b200.models.hybrid import HybridBlock, HybridWeights
    from mlxcel_b200.models.weights import LayerWeights
    W, I = s["width"], s["ff"] * 2 // 3 // 128 * 128
    n = 4 * s["groups"]
    cfg = ModelConfig.from_dict(dict(
        model_type="qwen3_next", vocab_size=VOCAB, hidden_size=W, num_hidden_layers=n, num_attention_heads=s["heads"],
        num_key_value_heads=s["kv"], head_dim=DIM, intermediate_size=I, num_experts=0, full_attention_interval=4,
        layer_types=(["linear_attention"] * 3 + ["full_attention"]) * s["groups"], linear_num_key_heads=s["delta"],
        linear_num_value_heads=s["delta"], linear_key_head_dim=DIM, linear_value_head_dim=DIM, linear_conv_kernel_dim=4,
        rms_norm_eps=1e-6, rope_theta=1e7, partial_rotary_factor=0.25))
    g = torch.Generator(device=DEV).manual_seed(0)
    r = lambda *sh: (torch.randn(*sh, generator=g, device=DEV) * sh[-1] ** -0.5).to(torch.bfloat16)     # noqa: E731
    one = lambda d: torch.ones(d, dtype=torch.bfloat16, device=DEV)                                     # noqa: E731
    d = gdn_dims(cfg)
    blocks, attn = [], []
    for i in range(n):
        if i % 4 != 3:
            blocks.append(HybridBlock("gdn", one(W), mamba=GdnLayerWeights(
                norm=one(W), in_proj=r(d["conv_dim"] + d["value_dim"], W), in_proj_ba=r(2 * d["Hv"], W),
                conv_w=torch.randn(d["conv_dim"], 4, generator=g, device=DEV) * 0.3, dt_bias=torch.zeros(d["Hv"], device=DEV),
                A_log=torch.zeros(d["Hv"], device=DEV), gnorm=one(DIM), out_proj=r(W, d["value_dim"]))))
        else:
            lw = LayerWeights(ln1=one(W), ln2=one(W), wqkv=r((s["heads"] + 2 * s["kv"]) * DIM, W), wo=r(W, s["heads"] * DIM),
                              q_norm=one(DIM), k_norm=one(DIM))
            attn.append(lw)
            blocks.append(HybridBlock("attention", lw.ln1, attn=lw, out_gate=r(s["heads"] * DIM, W)))
        blocks.append(HybridBlock("mlp", one(W), up=r(2 * I, W), down=r(W, I), gated=True))
    w = HybridWeights(embed=r(VOCAB, W), blocks=blocks, final_norm=one(W), lm_head=r(VOCAB, W), layers=attn)
    return LLM(cfg, w, ecfg)


def kernel_rows(s, rows=64, ctx=1024, pieces=8, piece=1024):
    """(name, new kernel us, share of roofline, its counterpart, us, share) per role."""
    from mlxcel_b200 import ops
    from mlxcel_b200.ops import KVLayer, recurrent as R, stream
    W, ff, Hq, Hkv, H = s["width"], s["ff"], s["heads"], s["kv"], s["delta"]
    bf = lambda *sh: torch.randn(*sh, device=DEV).to(torch.bfloat16)                       # noqa: E731
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=DEV)                         # noqa: E731
    f32 = lambda *sh: torch.randn(*sh, device=DEV)                                         # noqa: E731
    table = Table()
    add = table.add
    # ---- row kernels (prefill and decode rows)
    for n in (rows, pieces * piece):
        h, y, w, x = f32(n, W), bf(n, W), f32(W), bf(n, W)
        wb = torch.ones(W, dtype=torch.bfloat16, device=DEV)
        add(f"norms and residual, {n} rows", "hbm", ("stream_norm", lambda: stream.stream_norm(h, y, w, w, w, 1e-6, 1.0)), n * W * 12,
            ("add_rmsnorm", lambda: ops.add_rmsnorm(y, x, wb, 1e-6)), n * W * 8)
        z, coef = bf(n, ff), f32(4)
        gu = bf(n, 2 * (ff * 2 // 3))
        add(f"activation, {n} rows", "hbm", ("polynorm", lambda: stream.polynorm(z, coef, 1e-6)), n * ff * 4,
            ("swiglu (unfused form)", lambda: ops.swiglu(gu, gu.shape[1] // 2)), n * gu.shape[1] * 3)
        del h, y, x, z, gu
    # ---- attention
    D, bs = DIM, 16
    nb = rows * ctx // bs
    kv = KVLayer(bf(nb, Hkv, bs, D), bf(nb, Hkv, bs, D), None, None, bs)
    tables = torch.randperm(nb, device=DEV).to(torch.int32).view(rows, -1)
    lens = i32([ctx] * rows)
    r1, r2, sinks = f32(Hq).abs(), f32(Hq).abs() * 0.1, f32(Hq)
    qd = bf(rows, (2 * Hq + 2 * Hkv) * D)
    o = torch.empty(rows, Hq * D, dtype=torch.bfloat16, device=DEV)
    geo = dict(Hq=Hq, Hkv=Hkv, Dk=D, Dv=D, scale=D ** -0.5, sinks=sinks, dist_bias=(r1, r2))
    g0 = (Hq + 2 * Hkv) * D
    add(f"attention decode, {rows} x {ctx}", "hbm",
        ("paged_decode_mma (bias, sink, gate)", lambda: stream.paged_attention(qd[:, :Hq * D], kv, tables, lens, None, o, max_q_len=1,
                                                                               max_len=ctx, gate=qd[:, g0:], **geo)), rows * ctx * Hkv * D * 4,
        ("paged_decode_mma", lambda: ops.paged_decode(qd[:, :Hq * D], kv, tables, lens, Hq=Hq, Hkv=Hkv, D=D, scale=D ** -0.5, max_len=ctx,
                                                      out=o)), rows * ctx * Hkv * D * 4)
    T = pieces * piece
    q = bf(T, (2 * Hq + 2 * Hkv) * D)
    op = torch.empty(T, Hq * D, dtype=torch.bfloat16, device=DEV)
    cu, pl = i32([i * piece for i in range(pieces + 1)]), i32([piece] * pieces)
    pt = tables[:pieces]
    fl = pieces * Hq * D * 4 * (piece * piece / 2)
    add(f"attention prefill, {pieces} x {piece}", "tensor",
        ("paged_prefill_tc (bias, sink, gate)", lambda: stream.paged_attention(q[:, :Hq * D], kv, pt, pl, cu, op, max_q_len=piece,
                                                                               gate=q[:, g0:], **geo)), fl,
        ("paged_prefill_tc", lambda: ops.paged_prefill(q[:, :Hq * D], kv, pt, cu, pl, Hq=Hq, Hkv=Hkv, D=D, scale=D ** -0.5,
                                                       max_q_len=piece, out=op)), fl)
    slots = torch.arange(T, dtype=torch.int32, device=DEV) % (nb * bs)
    qn, pos, inv = f32(D), torch.arange(T, dtype=torch.int32, device=DEV), f32(D // 2)
    qb = torch.ones(D, dtype=torch.bfloat16, device=DEV)
    qkv = q[:, :g0].contiguous()
    io = T * D * 2 * (2 * Hq + 4 * Hkv)
    add(f"q/k norm and append, {T} rows", "hbm", ("qk_norm_append", lambda: stream.qk_norm_append(
        q, slots, kv, Hq=Hq, Hkv=Hkv, Dk=D, Dv=D, q_norm=qn, k_norm=qn, eps=1e-6)), io,
        ("rope_append", lambda: ops.rope_append(qkv, pos, slots, inv, kv, Hq=Hq, Hkv=Hkv, D=D, rot_dim=D, q_norm_w=qb, k_norm_w=qb)), io)
    del q, qkv, op, kv
    # ---- recurrence
    HD, Rk = H * D, 64
    offs = tuple(i * HD for i in range(6))
    w2, vec = bf(HD, Rk), f32(HD)
    st = torch.zeros(rows, H, D, D, device=DEV)
    proj = bf(rows, 5 * HD + Rk)
    sl = torch.arange(rows, dtype=torch.int32, device=DEV)
    cud, z0 = torch.arange(rows + 1, dtype=torch.int32, device=DEV), torch.zeros(rows, dtype=torch.int32, device=DEV)
    gq, gk, gv = bf(rows, H, D), bf(rows, H, D), bf(rows, H, D)
    gg, gb = -f32(rows, H).abs(), torch.rand(rows, H, device=DEV)
    state_io = rows * H * D * D * 8
    add(f"recurrence decode, {rows} rows", "hbm",
        ("delta_step", lambda: stream.delta_rule(proj, offs, w2, vec, vec, vec, st, sl, cud, z0, D=D, norm_eps=1e-6, n_short=rows)), state_io,
        ("gated_delta (state already gathered)", lambda: R.gated_delta_update(st, gq, gk, gv, gg, gb)), state_io)
    del proj
    proj = bf(T, 5 * HD + Rk)
    flops = T * H * D * D * 8
    N = 128
    mst = torch.zeros(pieces, H, D, N, device=DEV)
    mx, mdt, mB, A = bf(T, HD), bf(T, H), bf(T, 2 * N), -f32(H).abs()
    add(f"recurrence prefill, {pieces} x {piece} (8 flops per state element and token; fp32 SIMT peak is 1/20 of the tensor peak)", "tensor",
        ("delta_prep + delta_scan + delta_post", lambda: stream.delta_rule(proj, offs, w2, vec, vec, vec, st, sl[:pieces], cu, z0[:pieces],
                                                                            D=D, norm_eps=1e-6)), flops,
        ("ssm_scan (Mamba2, same state; the delta rule of the closest model runs token by token)",
         lambda: R.ssm_scan_varlen(mst, sl[:pieces], cu, z0[:pieces], mx, mdt, A, mB[:, :N], mB[:, N:])), T * H * D * N * 5)
    return table.rows


def run() -> None:
    how = peaks()[2]
    for name, s in SIZES.items():
        for k in kernel_rows(s):
            print(json.dumps(dict(design="pamasun", size=name, peaks=how, **k)), flush=True)
        torch.cuda.empty_cache()
        ours = engine_rates(pamasun_llm, s)
        ref = engine_rates(closest_llm, s)
        print(json.dumps(dict(design="pamasun", size=name, layers=4 * s["groups"], engine=ours, closest="qwen3_next layout, dense",
                              closest_engine=ref)), flush=True)
