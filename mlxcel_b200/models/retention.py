"""Retention with per-sequence state slots: linear attention with a fixed decay per head and no softmax.

Per head with state S [dim, vdim]: ``S <- decay S + k v^T; o = S^T q``; q and k are rotated by their positions, k times
dim^(-1/2) behind the rotation; o is divided by its root mean square per head and gated by ``silu``. Rotation, state,
decay and norm are fp32. Kernels: ``csrc/retention.cu``.

State slots, decode graphs and the interface to the engine are those of :class:`GeneralDeltaModel`. The short convolutions of
a model with several residual streams (``ops/streams.py``) keep their last inputs in the same slots."""
from __future__ import annotations

from dataclasses import dataclass

import torch

from ..ops import retention
from .general_delta import GeneralDeltaModel


@dataclass
class RetentionWeights:
    inv_freq: torch.Tensor    # fp32 [rotated dimensions / 2]
    decay: torch.Tensor       # fp32 [heads]
    heads: int
    dim: int
    vdim: int
    gain: float = 1.0         # factor of the gated heads

    @property
    def rows(self) -> int:
        """Rows of the input projection: q | k | v | gate."""
        return 2 * self.heads * (self.dim + self.vdim)


class RetentionModel(GeneralDeltaModel):
    """State slots + mixer of the retention layers (a component of the hybrid executor). ``runs``: the layers in execution
    order, a state slab each; ``convs``: (taps, width) of every short convolution, a slab of its last taps - 1 inputs each."""

    def __init__(self, runs: list[RetentionWeights], convs: list[tuple[int, int]], norm_eps: float, device, max_seqs: int = 256, comm=None):
        self.convs = convs
        super().__init__(runs, norm_eps, device, max_seqs, comm)

    def _slabs(self, runs: list[RetentionWeights], max_seqs: int) -> list:
        new = lambda *s: torch.zeros(max_seqs, *s, dtype=torch.float32, device=self.device)      # noqa: E731
        self.memory = [new(w.heads, w.dim, w.vdim) for w in runs]
        self.tail = [new(taps - 1, width) for taps, width in self.convs]
        return self.memory + self.tail

    def heads(self, run: int, w: RetentionWeights, proj: torch.Tensor, b, pieces, out: torch.Tensor) -> None:
        """proj [T, rows] as projected -> the gated heads, into ``out`` [T, heads * vdim]."""
        slots, cu, reset, nd, _ = pieces
        retention.retention(proj, b.positions, w.inv_freq, w.decay, self.memory[run], slots, cu, reset, out, norm_eps=self.norm_eps,
                            gain=w.gain, n_short=nd)
