"""Multi-head latent attention mixer on a latent pool: one ``[normalised latent | rotated key part]`` row per token.

Queries come through a latent of their own (``q = W_uq norm(W_dq h)``) or straight from the input (``w_uq`` None); per head they have an unrotated part scored
against ``W_uk c`` and a rotated part scored against one key part that all heads share, and the value is ``W_uv c``. Only c
and the rotated key part are stored. Optional: a sliding window, a sink (``exp(sink_h)`` in the denominator), the rotation
of neighbouring dimensions instead of halves (``adjacent``).

Decode rows run absorbed (``W_uk`` moves into the query, ``W_uv`` behind the attention): the context is read as stored,
once for all heads. Prompt portions run expanded: their context's rows are gathered and projected to per-head keys and
values (fewer operations per query-key pair), a group of heads at a time where the context is long. One GEMM produces query
latent | latent | key part; one kernel normalises, rotates and appends."""
from __future__ import annotations

from dataclasses import dataclass

import torch

from .. import ops
from ..ops import latent

EXPAND_BYTES = 1 << 30        # most that expanded keys and values of one group of heads take


@dataclass
class LatentMixerWeights:
    w_in: torch.Tensor                    # rows query latent (or queries) | latent | key part, zero rows up to a multiple of 8
    q_norm: torch.Tensor | None           # fp32 [q_rank]
    c_norm: torch.Tensor                  # fp32 [kv_rank]
    w_uq: torch.Tensor | None             # [heads * (dim + rot_dim), q_rank]
    w_uk: torch.Tensor                    # [heads * dim, kv_rank]
    w_uk_t: torch.Tensor                  # the same per head, transposed: [heads, kv_rank, dim]
    w_uv: torch.Tensor                    # [heads * vdim, kv_rank]
    out_proj: torch.Tensor                # [H, heads * vdim]
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    inv_freq: torch.Tensor                # fp32 [rot_dim / 2]
    mscale: float = 1.0
    adjacent: bool = False                # the rotation turns dimension 2i with 2i + 1
    window: int = 0                       # a token sees itself and the window - 1 tokens before it (0: all)
    sinks: torch.Tensor | None = None     # fp32 [heads]


def context_rows(b, window: int = 0) -> tuple[torch.Tensor, torch.Tensor, int]:
    """The rows of the gathered matrix the prompt portions' contexts take: (bounds [portions + 1] int32, the row token 0
    of each context would have [portions] int32, rows in all), computed once per batch and window. With a window only the
    tokens some query sees are gathered, from a multiple of the attention kernel's tile on."""
    cache = b.__dict__.setdefault("_context_rows", {})
    got = cache.get(window)
    if got is None:
        if b.pf_cu_q_host is not None and b.pf_starts is not None:
            spans = [(s, s + b.pf_cu_q_host[i + 1] - b.pf_cu_q_host[i]) for i, s in enumerate(b.pf_starts)]
        else:
            q = b.pf_cu_q.tolist()
            spans = [(n - (q[i + 1] - q[i]), n) for i, n in enumerate(b.pf_context_lens.tolist())]
        bounds, zero = [0], []
        for start, end in spans:
            skip = max(0, start - window + 1) // latent.EXPANDED_TILE * latent.EXPANDED_TILE if window > 0 else 0
            zero.append(bounds[-1] - skip)
            bounds.append(bounds[-1] + end - skip)
        both = torch.tensor(bounds + zero, dtype=torch.int32).to(b.pf_context_lens.device)
        got = cache[window] = (both[:len(bounds)], both[len(bounds):], bounds[-1])
    return got


def _absorbed(w: LatentMixerWeights, q, positions, kv, tables, lens, cu, out, max_len: int = 0) -> None:
    H, D, R, C, V = w.heads, w.dim, w.rot_dim, w.kv_rank, w.vdim
    n, W = q.shape[0], C + R
    qa = torch.empty(n, H * W, dtype=q.dtype, device=q.device)
    ops.batched_linear(q, w.w_uk_t, qa, D + R, W)
    latent.latent_q_rope(q, qa, positions, H=H, q_at=D, q_head=D + R, d_at=C, d_head=W, inv_freq=w.inv_freq, mscale=w.mscale, adjacent=w.adjacent)
    o = torch.empty(n, H * C, dtype=q.dtype, device=q.device)
    latent.latent_attention(qa, kv, tables, lens, cu, o, H=H, C=C, scale=w.scale, max_len=max_len, window=w.window, sinks=w.sinks)
    ops.batched_linear(o, w.w_uv.view(H, V, C), out, C, V)


def _expanded(w: LatentMixerWeights, q, positions, b, kv, out) -> None:
    H, D, R, C, V = w.heads, w.dim, w.rot_dim, w.kv_rank, w.vdim
    latent.latent_q_rope(q, q, positions, H=H, q_at=D, q_head=D + R, d_at=D, d_head=D + R, inv_freq=w.inv_freq, mscale=w.mscale, adjacent=w.adjacent)
    bounds, zero, rows = context_rows(b, w.window)
    ctx = latent.latent_gather(kv, b.pf_block_tables, bounds, rows, zero)
    c, kr = ctx[:, :C], ctx[:, C:]
    group = max(1, min(H, EXPAND_BYTES // max(1, 2 * rows * (D + V))))
    for h0 in range(0, H, group):
        h1 = min(H, h0 + group)
        kn, v = ops.linear(c, w.w_uk[h0 * D:h1 * D]), ops.linear(c, w.w_uv[h0 * V:h1 * V])
        latent.latent_prefill(q[:, h0 * (D + R):h1 * (D + R)], kn, kr, v, b.pf_cu_q, b.pf_context_lens, zero,
                              out[:, h0 * V:h1 * V], H=h1 - h0, D=D, R=R, V=V, scale=w.scale, max_q_len=b.pf_max_q_len,
                              window=w.window, sinks=None if w.sinks is None else w.sinks[h0:h1])


def latent_mixer(w: LatentMixerWeights, x: torch.Tensor, b, kv, eps: float) -> torch.Tensor:
    """x [T, H] the mixer's input, ``b`` the step's batch, ``kv`` this layer's pool. Returns the heads [T, heads * vdim]
    (the input of ``out_proj``)."""
    T, nd = x.shape[0], b.num_decode
    a = ops.linear(x, w.w_in)
    nq = 0 if w.w_uq is not None else w.heads * (w.dim + w.rot_dim)       # columns of queries in front of the latent
    latent.latent_append(a[:, nq:], b.positions, b.slot_mapping, kv, Q=w.q_rank, C=w.kv_rank, R=w.rot_dim, inv_freq=w.inv_freq,
                         mscale=w.mscale, q_norm=w.q_norm, c_norm=w.c_norm, eps=eps, adjacent=w.adjacent)
    q = a[:, :nq] if w.w_uq is None else ops.linear(a[:, :w.q_rank], w.w_uq)
    out = torch.empty(T, w.heads * w.vdim, dtype=q.dtype, device=q.device)
    if nd > 0:
        _absorbed(w, q[:nd], b.positions[:nd], kv, b.dec_block_tables, b.dec_context_lens, None, out[:nd], b.dec_max_len)
    if b.num_prefill_seqs > 0:
        if latent.expanded_covered(q.dtype, w.dim, w.rot_dim, w.vdim, w.kv_rank, q.is_cuda):
            _expanded(w, q[nd:], b.positions[nd:], b, kv, out[nd:])
        else:
            _absorbed(w, q[nd:], b.positions[nd:], kv, b.pf_block_tables, b.pf_context_lens, b.pf_cu_q, out[nd:])
    return out
