"""Generalized delta-rule mixer with per-sequence state slots.

Per head with state S [D, D] (key channel, value channel), decay w and removal rate a per key channel and
unit key u: ``S <- diag(w) S - (a u)(u^T S) + k v^T``, both terms from the old state, ``o = S^T r``; o is divided
by its root mean square per head, weighted and gated. The decay comes from a low-rank projection,
``w = exp(-exp(-1/2) sigmoid(w0 + W2 tanh(W1 h)))``. Kernels: ``csrc/delta_rule.cu``.

State slots and the interface to the engine are those of :class:`Mamba2Model`; there is no convolution. Every run
of a layer that is executed several times owns a slab of its own, and layers may differ in heads and
width, so the slabs are a list. Decode steps read the slots from a fixed device buffer when the engine
provides one (``StepBatch.state_slots``), which makes them replayable from a CUDA graph.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch

from .. import ops
from ..ops import stream
from .decoder import LocalComm
from .mamba2 import Mamba2Model


@dataclass
class GeneralDeltaWeights:
    w_in: torch.Tensor        # rows r | k | v | gate | removal rate | low-rank decay, zero rows up to a multiple of 8
    w2: torch.Tensor          # [heads * dim, rank]
    w0: torch.Tensor          # fp32 [heads * dim]
    a_bias: torch.Tensor      # fp32 [heads * dim]
    norm_w: torch.Tensor      # fp32 [heads * dim]
    out_proj: torch.Tensor    # [H, heads * dim]
    heads: int
    dim: int

    @property
    def offsets(self) -> tuple:
        return tuple(i * self.heads * self.dim for i in range(6))


class GeneralDeltaModel(Mamba2Model):
    """State slots + mixer of the delta layers (a component of the hybrid executor). ``runs``: the layer
    weights in execution order, one state slab each."""

    def __init__(self, runs: list[GeneralDeltaWeights], norm_eps: float, device, max_seqs: int = 256, comm=None):
        self.runs, self.norm_eps, self.device = runs, norm_eps, device
        self.comm = comm or LocalComm()
        if self.comm.tp_size != 1:
            raise NotImplementedError("the delta-rule executor is single-GPU")
        self.state = self._slabs(runs, max_seqs)
        self.slot_of: dict[int, int] = {}
        self.free = list(range(max_seqs - 1, -1, -1))
        self._iota = torch.arange(max_seqs + 1, dtype=torch.int32, device=device)
        self._no_reset = torch.zeros(max_seqs + 1, dtype=torch.int32, device=device)

    def _slabs(self, runs: list, max_seqs: int) -> list:
        return [torch.zeros(max_seqs, w.heads, w.dim, w.dim, dtype=torch.float32, device=self.device) for w in runs]

    def _slot(self, seq_id: int, resets: bool) -> int:
        s = self.slot_of.get(seq_id)
        if s is None:
            if not self.free:
                raise RuntimeError("no free recurrent-state slot (raise max_seqs)")
            s = self.slot_of[seq_id] = self.free.pop()
            if not resets:
                for st in self.state:
                    st[s].zero_()
        return s

    def slot(self, seq_id: int) -> int:
        """Slot of a sequence that has state already (decode rows)."""
        return self._slot(seq_id, False)

    def pieces(self, b):
        slots = getattr(b, "state_slots", None)
        if slots is not None and b.num_prefill_seqs == 0:
            nd = b.num_decode
            if nd >= self._iota.shape[0]:
                raise RuntimeError("more decode rows than state slots")
            return slots[:nd], self._iota[: nd + 1], self._no_reset[:nd], nd, 1
        return super().pieces(b)

    def mixer(self, run: int, w: GeneralDeltaWeights, x: torch.Tensor, pieces) -> torch.Tensor:
        """x [T, H] normalised input. Returns [T, heads * dim] (the input of ``out_proj``)."""
        slots, cu, reset, nd, _ = pieces
        proj = ops.linear(x, w.w_in)
        return stream.delta_rule(proj, w.offsets, w.w2, w.w0, w.a_bias, w.norm_w, self.state[run], slots, cu, reset,
                                 D=w.dim, norm_eps=self.norm_eps, n_short=nd)
