"""Gated delta rule with a short convolution in front and a gated norm behind (``csrc/gated_delta.cu``; CPU tensors take the
PyTorch statement). bf16 or fp32 projections; rates, norms, decays and the state are fp32."""
from __future__ import annotations

import torch

from . import _lib
from .stream import _call, _f, _fp32, _i, _ll, _rms, _SIG, _vp

_SIG["mx_gated_delta"] = [_vp, _ll] + [_vp] * 12 + [_i] * 8 + [_f, _f, _i, _i, _vp]
UNIT_EPS = 1e-6                          # inside the root of the unit queries and keys


def gated_delta_ref(proj, rates, conv_w, A_log, dt_bias, norm_w, memory, tail, slots, cu, reset, G: int, norm_eps: float, unit_eps: float):
    H, D, V = memory.shape[1:]
    ch, taps = conv_w.shape
    x, out = proj[:, :ch].float(), torch.zeros(proj.shape[0], H, V, device=proj.device)
    beta = torch.sigmoid(rates[:, :H])
    g = torch.exp(-torch.exp(A_log) * torch.nn.functional.softplus(rates[:, H:2 * H] + dt_bias))
    unit = lambda t: t / torch.sqrt(t.pow(2).sum(-1, keepdim=True) + unit_eps)      # noqa: E731
    sl, rs, c = slots.tolist(), reset.tolist(), cu.tolist()
    for j in range(len(sl)):
        if sl[j] < 0 or c[j + 1] <= c[j]:
            continue
        rows = slice(c[j], c[j + 1])
        S, before = (torch.zeros_like(t[0]) if rs[j] else t[sl[j]].clone() for t in (memory, tail))
        past = torch.cat([before, x[rows]], 0)
        n = c[j + 1] - c[j]
        y = torch.nn.functional.silu(sum(past[i:i + n] * conv_w[:, i] for i in range(taps)))
        q, k = unit(y[:, :G * D].view(n, G, D)) * D ** -0.5, unit(y[:, G * D:2 * G * D].view(n, G, D))
        q, k, v = q.repeat_interleave(H // G, 1), k.repeat_interleave(H // G, 1), y[:, 2 * G * D:].reshape(n, H, V)
        for t in range(n):
            r = c[j] + t
            S = S * g[r][:, None, None]
            u = beta[r][:, None] * (v[t] - (S * k[t][:, :, None]).sum(1))
            S = S + k[t][:, :, None] * u[:, None, :]
            out[r] = (S * q[t][:, :, None]).sum(1)
        memory[sl[j]], tail[sl[j]] = S, past[n:]
    gate = proj[:, ch:ch + H * V].float()
    return ((_rms(out, norm_eps) * norm_w).reshape(-1, H * V) * torch.nn.functional.silu(gate)).to(proj.dtype)


def gated_delta(proj, rates, conv_w, A_log, dt_bias, norm_w, memory, tail, slots, cu, reset, *, G: int, norm_eps: float, n_short: int = 0,
                unit_eps: float = UNIT_EPS, force_any: bool = False):
    """Gated delta rule over a ragged batch.

    ``proj`` rows: q [G * D] | k [G * D] | v [H * V] | gate [H * V] as projected; ``rates`` rows (fp32): write rate [H] |
    decay [H] pre-activations; ``conv_w`` fp32 [channels of q | k | v, taps]; ``memory`` [slots, H, D, V] and ``tail``
    [slots, taps - 1, channels] fp32 are advanced in place; ``slots`` / ``reset`` [pieces], ``cu`` [pieces + 1] int32 (the first
    ``n_short`` pieces are decode rows of one token; a negative slot marks a padding row). Returns [rows, H * V] in
    proj's type, ready for the output projection."""
    if not proj.is_cuda:
        return gated_delta_ref(proj, rates, conv_w, A_log, dt_bias, norm_w, memory, tail, slots, cu, reset, G, norm_eps, unit_eps)
    (H, D, V), taps, rows, pieces = memory.shape[1:], conv_w.shape[1], proj.shape[0], slots.shape[0]
    assert proj.stride(1) == 1 and rates.dtype == torch.float32 and rates.is_contiguous() and rates.shape[1] == 2 * H
    assert memory.is_contiguous() and tail.is_contiguous() and conv_w.is_contiguous() and proj.shape[1] >= 2 * (G * D + H * V)
    out = torch.empty(rows, H * V, dtype=proj.dtype, device=proj.device)
    lib = _lib.load()
    floats = lib.mx_gated_delta_scratch_floats
    if not floats.argtypes:
        floats.argtypes, floats.restype = [_i] * 5, _ll
    short = 0 if force_any or not lib.mx_gated_delta_step_covered(H, G, D, V, taps) else n_short
    scratch = torch.empty(int(floats(rows - short, H, G, D, V)), dtype=torch.float32, device=proj.device) if pieces > short else None
    _call("mx_gated_delta", proj.data_ptr(), proj.stride(0), rates.data_ptr(), conv_w.data_ptr(), A_log.data_ptr(), dt_bias.data_ptr(),
          norm_w.data_ptr(), memory.data_ptr(), tail.data_ptr(), slots.data_ptr(), cu.data_ptr(), reset.data_ptr(), out.data_ptr(),
          _lib.ptr(scratch), pieces, short, rows, H, G, D, V, taps, float(unit_eps), float(norm_eps), _fp32(proj),
          1 if force_any else 0, _lib.stream())
    _lib.count_launch((1 if short and pieces > short else 0) + (2 if pieces > short else 0))
    return out
