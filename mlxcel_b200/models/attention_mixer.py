"""Attention mixer with optional parts, each a field of its layer's record, so models may mix layers of different shapes:

* positions: a rotation of the first dimensions of q and k (``inv_freq``, ``mscale``), a logarithmic distance bias
  (``- r1_h ln(1 + r2_h (i - j))``), or none;
* q/k norm per head: with weights and without a rotation, or behind the rotation (``unit``: division by the root mean
  square, weights optional);
* visibility: all earlier tokens, a window of them, or the earlier tokens of the query's own chunk (runs of ``chunk``
  positions counted from the sequence's start); beside a window, one key and value for every block of ``means`` tokens that lies
  wholly before it, the means of the block's keys and values, in the same softmax;
* scores: ``q.k * scale``, soft-capped (``softcap tanh(s / softcap)``) where a cap is given; ``exp(sink_h)`` in the
  denominator;
* values: heads of their own width, or the keys as projected (``values_are_keys``: no value projection);
* a sigmoid gate computed from the mixer's input on the concatenated heads;
* differential heads (``diff``): query and key rows hold two maps of ``dim / 2`` each, attentions of their own over the same
  values; the head is ``a1 - factor * a2``, divided by its root mean square, times a gain.

One GEMM produces q | k | v | gate; one kernel rotates and normalises q and k and appends k, v (and the means of the blocks that
become full) to the paged pool; the attention kernels cap, mask, gate and combine the maps. Scores, bias, softmax and accumulation are fp32.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch

from .. import ops
from ..ops import block_means, stream


@dataclass
class AttentionMixerWeights:
    w_in: torch.Tensor                    # rows q | k (| v) (| gate), zero rows up to a multiple of 8
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
    chunk: int = 0
    softcap: float = 0.0
    inv_freq: torch.Tensor | None = None  # fp32 [rotated dimensions / 2]
    mscale: float = 1.0
    unit: bool = False                    # with a rotation: q and k divided by their root mean square behind it
    values_are_keys: bool = False
    b_in: torch.Tensor | None = None      # biases of w_in's rows
    diff: tuple | None = None             # (factor of the second map, gain)
    means: int = 0                        # tokens of a block that is seen as one key once it has left the window
    gain: float = 1.0                     # factor of the heads (no differential heads)


def stack_rows(parts: list[torch.Tensor]) -> torch.Tensor:
    """Projections that read the same input as one matrix; zero rows bring the row stride of its output to a
    multiple of 16 bytes, which the tensor-memory loads of the kernels behind it need."""
    w = torch.cat(parts, 0)
    pad = -w.shape[0] % 8
    return torch.cat([w, w.new_zeros(pad, w.shape[1])], 0).contiguous() if pad else w.contiguous()


def attention_mixer(w: AttentionMixerWeights, x: torch.Tensor, b, kv, eps: float) -> torch.Tensor:
    """x [T, H] normalised input, ``b`` the step's batch, ``kv`` this run's pool layer. Returns the gated heads
    [T, heads * vdim] (the input of ``out_proj``)."""
    row = ops.linear(x, w.w_in, bias=w.b_in)
    out = torch.empty(x.shape[0], w.heads * w.vdim, dtype=row.dtype, device=row.device)
    attention_heads(w, row, b, kv, eps, out)
    return out


def attention_heads(w: AttentionMixerWeights, row: torch.Tensor, b, kv, eps: float, out: torch.Tensor) -> None:
    """:func:`attention_mixer` behind its projection: rows q | k (| v) (| gate) -> ``out`` [T, heads * vdim] (may be a column
    slice of wider rows)."""
    nd = b.num_decode
    geo = dict(Hq=w.heads, Hkv=w.kv_heads, Dk=w.dim, Dv=w.vdim)
    # (rows, tables, lengths, bounds, longest piece, longest context) of the decode rows and of the prompt portions
    groups = []
    if nd > 0:
        groups.append((slice(0, nd), b.dec_block_tables, b.dec_context_lens, None, 1, b.dec_max_len))
    if b.num_prefill_seqs > 0:
        groups.append((slice(nd, row.shape[0]), b.pf_block_tables, b.pf_context_lens, b.pf_cu_q, b.pf_max_q_len, 0))
    if w.means:
        assert w.inv_freq is None and w.q_norm is None and w.k_norm is None and w.window > 0, "block means: a window, keys as projected"
        for at, tables, _, cu, _, _ in groups:
            block_means.append(row[at], b.positions[at], b.slot_mapping[at], kv, tables, cu, **geo)
    elif w.inv_freq is not None:
        stream.rope_norm_append(row, b.positions, b.slot_mapping, kv, inv_freq=w.inv_freq, mscale=w.mscale, unit=w.unit,
                                values_are_keys=w.values_are_keys, q_norm=w.q_norm, k_norm=w.k_norm, eps=eps, **geo)
    else:
        stream.qk_norm_append(row, b.slot_mapping, kv, q_norm=w.q_norm, k_norm=w.k_norm, eps=eps, **geo)
    q = row[:, : w.heads * w.dim]
    g0 = w.heads * w.dim + w.kv_heads * (w.dim + (0 if w.values_are_keys else w.vdim))
    gate = row[:, g0:g0 + w.heads * w.vdim] if w.gated else None
    common = dict(scale=w.scale, window=w.window, chunk=w.chunk, softcap=w.softcap, sinks=w.sinks, gain=w.gain,
                  dist_bias=None if w.r1 is None else (w.r1, w.r2), diff=None if w.diff is None else (*w.diff, eps), **geo)
    for at, tables, lens, cu, longest, max_len in groups:
        means = None
        if w.means:
            means = (None, 0) if cu is None else block_means.portion_means(b, w.window, w.means)
        stream.paged_attention(q[at], kv, tables, lens, cu, out[at], max_q_len=longest, max_len=max_len, means=means,
                               gate=None if gate is None else gate[at], **common)
