"""Attention and retention side by side on the same input, their results added with a factor each.

One GEMM projects both (attention's q | k | v, then retention's q | k | v | gate), both write their heads, times their factors,
into the columns of one matrix, and one GEMM with both output projections side by side adds them up."""
from __future__ import annotations

from dataclasses import dataclass

import torch

from .. import ops
from .attention_mixer import AttentionMixerWeights, attention_heads, stack_rows
from .retention import RetentionModel, RetentionWeights


def _up8(n: int) -> int:
    return (n + 7) // 8 * 8


@dataclass
class ParallelMixerWeights:
    attn: AttentionMixerWeights      # (its projections are here)
    ret: RetentionWeights
    w_in: torch.Tensor               # attention's rows, zero rows up to a multiple of 8, retention's rows, likewise
    b_in: torch.Tensor
    w_out: torch.Tensor              # [H, attention's columns | retention's columns], each with zero columns up to a multiple of 8

    @property
    def in_split(self) -> int:
        a = self.attn
        return _up8(a.heads * a.dim + a.kv_heads * (a.dim + a.vdim))

    @property
    def out_split(self) -> int:
        return _up8(self.attn.heads * self.attn.vdim)


def stack_parallel(left: list, left_bias: list, right: list) -> tuple[torch.Tensor, torch.Tensor]:
    """(w_in, b_in) of the projections' rows."""
    a, r = stack_rows(left), stack_rows(right)
    b = stack_rows([t[:, None] for t in left_bias])[:, 0]
    return torch.cat([a, r]).contiguous(), torch.cat([b, b.new_zeros(r.shape[0])]).contiguous()


def join_columns(left: torch.Tensor, right: torch.Tensor) -> torch.Tensor:
    pad = lambda w: torch.cat([w, w.new_zeros(w.shape[0], -w.shape[1] % 8)], 1)      # noqa: E731
    return torch.cat([pad(left), pad(right)], 1).contiguous()


def parallel_mixer(w: ParallelMixerWeights, ssm: RetentionModel, run: int, x: torch.Tensor, b, kv, pieces, eps: float) -> torch.Tensor:
    """x [T, H] the mixer's input, ``kv`` / ``run`` this layer's pool and state slab. Returns [T, H]."""
    row = ops.linear(x, w.w_in, bias=w.b_in)
    left, right, at = w.attn.heads * w.attn.vdim, w.ret.heads * w.ret.vdim, w.out_split
    padded = at != left or w.w_out.shape[1] != at + right
    both = (torch.zeros if padded else torch.empty)(x.shape[0], w.w_out.shape[1], dtype=row.dtype, device=row.device)
    attention_heads(w.attn, row[:, :w.in_split], b, kv, eps, both[:, :left])
    ssm.heads(run, w.ret, row[:, w.in_split:], b, pieces, both[:, at:at + right])
    return ops.linear(both, w.w_out)
