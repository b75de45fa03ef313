"""Attention mixer without rotation: positions enter through a logarithmic distance bias.

Per query head h with its key head: ``score = q.k * scale - r1_h ln(1 + r2_h (i - j))`` over all earlier
tokens (or a window of them), softmax with ``exp(sink_h)`` in the denominator, q and k RMS-normalised per
head, key and value heads of different widths, and a sigmoid gate computed from the mixer's input on the
concatenated heads. Every one of bias, sink, q/k norm and gate is optional, and the geometry belongs to
the layer, so models may mix layers of different shapes.

One GEMM produces q | k | v | gate; one kernel normalises q and k and appends k, v to the paged pool; the
attention kernels apply the gate on the way out. Scores, bias, softmax and accumulation are fp32.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch

from .. import ops
from ..ops import stream


@dataclass
class AttentionMixerWeights:
    w_in: torch.Tensor                    # rows q | k | v (| gate), zero rows up to a multiple of 8
    out_proj: torch.Tensor                # [H, heads * vdim]
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    gated: bool = False
    q_norm: torch.Tensor | None = None    # fp32 [dim], shared by the heads
    k_norm: torch.Tensor | None = None
    r1: torch.Tensor | None = None        # fp32 [heads]
    r2: torch.Tensor | None = None
    sinks: torch.Tensor | None = None     # fp32 [heads]
    window: int = 0


def stack_rows(parts: list[torch.Tensor]) -> torch.Tensor:
    """Projections that read the same input as one matrix; zero rows bring the row stride of its output to a
    multiple of 16 bytes, which the tensor-memory loads of the kernels behind it need."""
    w = torch.cat(parts, 0)
    pad = -w.shape[0] % 8
    return torch.cat([w, w.new_zeros(pad, w.shape[1])], 0).contiguous() if pad else w.contiguous()


def attention_mixer(w: AttentionMixerWeights, x: torch.Tensor, b, kv, eps: float) -> torch.Tensor:
    """x [T, H] normalised input, ``b`` the step's batch, ``kv`` this run's pool layer. Returns the gated heads
    [T, heads * vdim] (the input of ``out_proj``)."""
    T, nd = x.shape[0], b.num_decode
    row = ops.linear(x, w.w_in)
    geo = dict(Hq=w.heads, Hkv=w.kv_heads, Dk=w.dim, Dv=w.vdim)
    stream.qk_norm_append(row, b.slot_mapping, kv, q_norm=w.q_norm, k_norm=w.k_norm, eps=eps, **geo)
    q = row[:, : w.heads * w.dim]
    g0 = w.heads * w.dim + w.kv_heads * (w.dim + w.vdim)
    gate = row[:, g0:g0 + w.heads * w.vdim] if w.gated else None
    out = torch.empty(T, w.heads * w.vdim, dtype=row.dtype, device=row.device)
    common = dict(scale=w.scale, window=w.window, sinks=w.sinks, dist_bias=None if w.r1 is None else (w.r1, w.r2), **geo)
    if nd > 0:
        stream.paged_attention(q[:nd], kv, b.dec_block_tables, b.dec_context_lens, None, out[:nd], max_q_len=1,
                               max_len=b.dec_max_len, gate=None if gate is None else gate[:nd], **common)
    if b.num_prefill_seqs > 0:
        stream.paged_attention(q[nd:], kv, b.pf_block_tables, b.pf_context_lens, b.pf_cu_q, out[nd:],
                               max_q_len=b.pf_max_q_len, gate=None if gate is None else gate[nd:], **common)
    return out
