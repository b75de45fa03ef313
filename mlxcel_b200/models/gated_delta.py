"""Gated delta-rule mixer with one decay per head and per-sequence state slots (stream layout).

q, k and v pass a short causal convolution per channel and silu; q and k become unit vectors per head (``heads`` value heads
share ``kv_heads`` q/k heads). Per value head with state S [dim, vdim]: ``S <- g S; u = beta (v - S^T k); S <- S + k u^T;
o = S^T q``, ``g = exp(-exp(A_log) softplus(a + dt_bias))``, ``beta = sigmoid(b)``; o is divided by its root mean square per
head, weighted and gated by ``silu``. Kernels: ``csrc/gated_delta.cu``.

State slots, decode graphs and the interface to the engine are those of :class:`GeneralDeltaModel`; the last ``taps - 1``
convolution inputs are part of the state."""
from __future__ import annotations

from dataclasses import dataclass

import torch

from .. import ops
from ..ops import gated_delta
from .general_delta import GeneralDeltaModel


@dataclass
class GatedDeltaWeights:
    w_in: torch.Tensor        # rows q | k | v | gate, zero rows up to a multiple of 8
    w_rates: torch.Tensor     # rows write rate | decay, [2 * heads, H]
    conv_w: torch.Tensor      # fp32 [channels of q | k | v, taps], the last tap is the current token's
    A_log: torch.Tensor       # fp32 [heads]
    dt_bias: torch.Tensor     # fp32 [heads]
    norm_w: torch.Tensor      # fp32 [vdim], shared by the heads
    out_proj: torch.Tensor    # [H, heads * vdim]
    heads: int
    kv_heads: int
    dim: int
    vdim: int


class GatedDeltaModel(GeneralDeltaModel):
    """State slots + mixer of the gated delta layers (a component of the hybrid executor). ``runs``: the layer weights in
    execution order, a recurrent and a convolution slab each."""

    def _slabs(self, runs: list[GatedDeltaWeights], max_seqs: int) -> list:
        new = lambda *s: torch.zeros(max_seqs, *s, dtype=torch.float32, device=self.device)      # noqa: E731
        self.memory = [new(w.heads, w.dim, w.vdim) for w in runs]
        self.tail = [new(w.conv_w.shape[1] - 1, w.conv_w.shape[0]) for w in runs]
        return self.memory + self.tail

    def mixer(self, run: int, w: GatedDeltaWeights, x: torch.Tensor, pieces) -> torch.Tensor:
        """x [T, H] normalised input. Returns [T, heads * vdim] (the input of ``out_proj``)."""
        slots, cu, reset, nd, _ = pieces
        proj, rates = ops.linear(x, w.w_in), ops.linear(x, w.w_rates, out_fp32=True)
        return gated_delta.gated_delta(proj, rates, w.conv_w, w.A_log, w.dt_bias, w.norm_w, self.memory[run], self.tail[run], slots,
                                       cu, reset, G=w.kv_heads, norm_eps=self.norm_eps, n_short=nd)
