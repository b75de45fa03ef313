"""Retention: linear attention with a fixed decay per head (``csrc/retention.cu``; CPU tensors take the PyTorch statement). bf16
or fp32 projections; rotation, decay, state and norm are fp32."""
from __future__ import annotations

import torch

from . import _lib
from .stream import _call, _f, _fp32, _i, _ll, _rms, _SIG, _vp, rotate_half

_SIG["mx_retention"] = [_vp, _ll] + [_vp] * 8 + [_ll, _vp] + [_i] * 7 + [_f, _f, _i, _i, _vp, _vp]


def retention_ref(proj, positions, inv_freq, decay, memory, slots, cu, reset, out, norm_eps: float, gain: float):
    H, D, V = memory.shape[1:]
    T, HD, HV = proj.shape[0], H * D, H * V
    turn = lambda at: rotate_half(proj[:, at:at + HD].float().view(T, H, D), positions, inv_freq, 1.0)      # noqa: E731
    q, k, v = turn(0), turn(HD) * D ** -0.5, proj[:, 2 * HD:2 * HD + HV].float().view(T, H, V)
    o = torch.zeros(T, H, V, device=proj.device)
    sl, rs, c = slots.tolist(), reset.tolist(), cu.tolist()
    for j in range(len(sl)):
        if sl[j] < 0 or c[j + 1] <= c[j]:
            continue
        S = torch.zeros_like(memory[0]) if rs[j] else memory[sl[j]].clone()
        for t in range(c[j], c[j + 1]):
            S = S * decay[:, None, None] + k[t][:, :, None] * v[t][:, None, :]
            o[t] = (S * q[t][:, :, None]).sum(1)
        memory[sl[j]] = S
    gate = proj[:, 2 * HD + HV:2 * (HD + HV)].float()
    out.copy_((_rms(o, norm_eps).reshape(T, HV) * torch.nn.functional.silu(gate) * gain).to(out.dtype))


def retention(proj, positions, inv_freq, decay, memory, slots, cu, reset, out, *, norm_eps: float, gain: float = 1.0, n_short: int = 0,
              form: int = 0) -> None:
    """Retention over a ragged batch, into ``out`` [rows, H * V] (may be a column slice).

    ``proj`` rows: q [H * D] | k [H * D] | v [H * V] | gate [H * V] as projected; ``positions`` [rows] int32; ``inv_freq`` fp32 [rotated
    dimensions / 2] (dimension i turns with i + dims / 2); ``decay`` fp32 [H]; ``memory`` [slots, H, D, V] fp32 is advanced in
    place; ``slots`` / ``reset`` [pieces], ``cu`` [pieces + 1] int32 (the first ``n_short`` pieces are decode rows of one token; a
    negative slot marks a padding row). The result is the read-out over its root mean square per head, times silu(gate),
    times ``gain``. Longer pieces of bf16 rows with key heads of up to 128 run in chunks on the tensor cores; ``form`` 1 keeps
    them on the token-by-token kernel, which takes the rest."""
    if proj.shape[0] == 0:
        return
    if not proj.is_cuda:
        return retention_ref(proj, positions, inv_freq, decay, memory, slots, cu, reset, out, norm_eps, gain)
    (H, D, V), rows, pieces = memory.shape[1:], proj.shape[0], slots.shape[0]
    assert proj.stride(1) == 1 and out.stride(1) == 1 and out.dtype == proj.dtype and positions.dtype == torch.int32
    assert memory.is_contiguous() and decay.dtype == inv_freq.dtype == torch.float32 and 2 * inv_freq.shape[0] <= D
    lib = _lib.load()
    floats = lib.mx_retention_scratch_floats
    if not floats.argtypes:
        floats.argtypes, floats.restype = [_i] * 7, _ll
    bf, rot = (0 if proj.dtype == torch.float32 else 1), 2 * inv_freq.shape[0]
    if (proj.data_ptr() | out.data_ptr()) % 16 or proj.stride(0) % 8 or out.stride(0) % 8:
        form = 1
    scratch = torch.empty(int(floats(rows - n_short, H, D, V, rot, bf, form)), dtype=torch.float32, device=proj.device) if pieces > n_short else None
    _call("mx_retention", proj.data_ptr(), proj.stride(0), positions.data_ptr(), inv_freq.data_ptr(), decay.data_ptr(), memory.data_ptr(),
          slots.data_ptr(), cu.data_ptr(), reset.data_ptr(), out.data_ptr(), out.stride(0), _lib.ptr(scratch), pieces, n_short, rows, H, D, V,
          rot, float(norm_eps), float(gain), _fp32(proj), form, _lib.workspace(proj.device).data_ptr(), _lib.stream())
    chunks = bf and form == 0 and lib.mx_retention_chunk_covered(D, V, rot)
    _lib.count_launch((1 if n_short and pieces > n_short else 0) + ((1 if chunks and V <= 128 else 2) if pieces > n_short else 0))
