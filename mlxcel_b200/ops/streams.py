"""Several residual streams around each sub-layer (``csrc/streams.cu``; CPU tensors take the PyTorch statements).

``xs`` fp32 [tokens, streams, width]. A sub-layer reads ``u = sum_s w_in[s] x_s``, layer-normalised with weight and bias, plus a
causal convolution of that over time (``taps`` fp32 [K, width], the last row for the current token); with its result y the
streams become ``x_t <- sum_s mix[s, t] x_s + w_out[t] y``. One kernel does the step between two sub-layers: what the last one
returned (a row, or a token's chosen experts, plus a bias), the mixing, the next one's input and norm, and for rows of one
token (decode) the convolution and its state; a second one convolves prompt portions. All arithmetic is fp32."""
from __future__ import annotations

import ctypes
from dataclasses import dataclass

import torch

from . import _lib
from .stream import _call, _f, _fp32, _i, _SIG, _vp

MAX_STREAMS = 16


@dataclass
class Sublayer:
    """What surrounds one sub-layer; fp32 vectors."""

    w_in: torch.Tensor                        # [streams]
    w_out: torch.Tensor                       # [streams]
    mix: torch.Tensor                         # [streams, streams], [from, to]
    norm_w: torch.Tensor                      # [width]
    norm_b: torch.Tensor
    taps: torch.Tensor                        # [K, width]
    bias: torch.Tensor | None = None          # [width], added to the sub-layer's result


class _Step(ctypes.Structure):
    """Mirror of ``MxStreamsStep`` (csrc/api.h)."""

    _fields_ = [("xs", _vp), ("ids", _vp), ("table", _vp), ("y", _vp), ("moe_y", _vp), ("moe_inv", _vp), ("moe_w", _vp), ("bias", _vp),
                ("mix", _vp), ("w_out", _vp), ("w_in", _vp), ("norm_w", _vp), ("norm_b", _vp), ("taps_w", _vp), ("tail", _vp), ("slots", _vp),
                ("x", _vp), ("normed", _vp), ("sum", _vp), ("rows", _i), ("dim", _i), ("streams", _i), ("vocab", _i), ("moe_k", _i), ("taps", _i),
                ("n_short", _i), ("emb_scale", _f), ("eps", _f)]


_SIG["mx_streams_step"] = [ctypes.POINTER(_Step), _i, _vp]
_SIG["mx_streams_conv"] = [_vp] * 7 + [_i] * 7 + [_vp]
_SIG["mx_layer_norm_rows"] = [_vp] * 5 + [_i, _i, _f, _i, _vp]


def layer_norm_ref(x, w, b, eps: float):
    c = x - x.mean(-1, keepdim=True)
    return c * torch.rsqrt(c.pow(2).mean(-1, keepdim=True) + eps) * w + b


def conv_ref(n, taps, tail, slots, cu, reset):
    """n [T, width] fp32 plus its convolution over each piece; ``tail`` [slots, K - 1, width] is advanced in place."""
    K, out = taps.shape[0], n.clone()
    sl, rs, c = slots.tolist(), reset.tolist(), cu.tolist()
    for j in range(len(sl)):
        if sl[j] < 0 or c[j + 1] <= c[j]:
            continue
        m = c[j + 1] - c[j]
        past = torch.cat([torch.zeros_like(tail[0]) if rs[j] else tail[sl[j]], n[c[j]:c[j + 1]]])
        out[c[j]:c[j + 1]] += sum(past[i:i + m] * taps[i] for i in range(K))
        tail[sl[j]] = past[m:]
    return out


def _result(y, moe, bias):
    r = y.float() if moe is None else moe.summed()
    return r if bias is None else r + bias


def _enter_ref(xs, nxt, eps, dtype, tail, pieces):
    slots, cu, reset, _, _ = pieces
    n = layer_norm_ref((xs * nxt.w_in[:, None]).sum(1), nxt.norm_w, nxt.norm_b, eps)
    return conv_ref(n, nxt.taps, tail, slots, cu, reset).to(dtype)


def _step(xs, done: Sublayer | None, y, moe, nxt: Sublayer | None, eps, dtype, tail, pieces, total=None, embed=None):
    """The kernels of one step. Returns the next sub-layer's input, or None without ``nxt``."""
    T, S, H = xs.shape
    if T == 0:
        return None if nxt is None else torch.empty(0, H, dtype=dtype, device=xs.device)
    assert xs.is_contiguous() and xs.dtype == torch.float32 and S <= MAX_STREAMS
    p = _Step(xs=xs.data_ptr(), rows=T, dim=H, streams=S, eps=float(eps))
    if embed is not None:
        ids, table, p.emb_scale = embed
        assert table.dtype == dtype and ids.dtype == torch.int32
        p.ids, p.table, p.vocab = ids.data_ptr(), table.data_ptr(), table.shape[0]
    else:
        p.mix, p.w_out, p.bias = done.mix.data_ptr(), done.w_out.data_ptr(), _lib.ptr(done.bias)
        if moe is not None:
            assert moe.y.dtype == dtype and moe.shared is None and moe.y.shape[1] == H and int(moe.experts) > 0
            p.moe_y, p.moe_inv, p.moe_w, p.moe_k = moe.y.data_ptr(), moe.inv.data_ptr(), moe.wts.data_ptr(), moe.ids.shape[1]
        else:
            assert y.is_contiguous() and y.dtype == dtype and y.shape == (T, H)
            p.y = y.data_ptr()
    x = normed = None
    fp32 = 1 if dtype == torch.float32 else 0
    if total is not None:
        p.sum = total.data_ptr()
    if nxt is not None:
        slots, cu, reset, nd, longest = pieces
        K = nxt.taps.shape[0]
        x = torch.empty(T, H, dtype=dtype, device=xs.device)
        if nd < T and K > 1:
            normed = torch.empty(T - nd, H, dtype=torch.float32, device=xs.device)
        p.w_in, p.norm_w, p.norm_b, p.taps_w = (t.data_ptr() for t in (nxt.w_in, nxt.norm_w, nxt.norm_b, nxt.taps))
        p.taps = K
        p.tail, p.slots, p.x, p.normed, p.n_short = tail.data_ptr(), slots.data_ptr(), x.data_ptr(), _lib.ptr(normed), nd
    _call("mx_streams_step", ctypes.byref(p), fp32, _lib.stream())
    if normed is not None:
        _call("mx_streams_conv", normed.data_ptr(), nxt.taps.data_ptr(), tail.data_ptr(), slots[nd:].data_ptr(), cu[nd:].data_ptr(),
              reset[nd:].data_ptr(), x.data_ptr(), slots.shape[0] - nd, nd, T, H, K, longest, fp32, _lib.stream())
    return x


def embed_streams(ids, table, scale: float, streams: int, nxt: Sublayer, eps: float, tail, pieces):
    """Every stream starts as ``scale * table[ids]``. Returns (xs, the first sub-layer's input)."""
    dim = table.shape[1]
    if not table.is_cuda:
        ok = (ids >= 0) & (ids < table.shape[0])
        e = table[ids.clamp(0, table.shape[0] - 1).long()].float() * scale * ok[:, None]
        xs = e[:, None].repeat(1, streams, 1)
        return xs, _enter_ref(xs, nxt, eps, table.dtype, tail, pieces)
    xs = torch.empty(ids.shape[0], streams, dim, dtype=torch.float32, device=table.device)
    return xs, _step(xs, None, None, None, nxt, eps, table.dtype, tail, pieces, embed=(ids, table, float(scale)))


def mix_streams(xs, done: Sublayer, y, moe, nxt: Sublayer, eps: float, dtype, tail, pieces):
    """The step between two sub-layers, in place on ``xs``: ``done`` returned ``y`` (or the experts' rows ``moe``), ``nxt`` comes next;
    ``tail`` [slots, K - 1, width] is the state of its convolution, ``pieces`` the ragged batch. Returns its input as ``dtype``."""
    if not xs.is_cuda:
        xs.copy_(torch.einsum("nsd,st->ntd", xs, done.mix) + done.w_out[:, None] * _result(y, moe, done.bias)[:, None])
        return _enter_ref(xs, nxt, eps, dtype, tail, pieces)
    return _step(xs, done, y, moe, nxt, eps, dtype, tail, pieces)


def sum_streams(xs, done: Sublayer, y, moe, dtype):
    """Behind the last sub-layer: the sum of the streams, fp32 [tokens, width] (``xs`` itself is not advanced)."""
    if not xs.is_cuda:
        return torch.einsum("nsd,st->nd", xs, done.mix) + done.w_out.sum() * _result(y, moe, done.bias)
    total = torch.empty(xs.shape[0], xs.shape[2], dtype=torch.float32, device=xs.device)
    _step(xs, done, y, moe, None, 0.0, dtype, None, None, total=total)
    return total


def layer_norm(h, w, b, eps: float, dtype, rows=None):
    """Layer norm of fp32 rows (or of the rows ``rows``, int32) as ``dtype``."""
    if not h.is_cuda:
        return layer_norm_ref(h if rows is None else h[rows.long()], w, b, eps).to(dtype)
    n = h.shape[0] if rows is None else rows.shape[0]
    out = torch.empty(n, h.shape[1], dtype=dtype, device=h.device)
    assert h.is_contiguous() and h.dtype == torch.float32 and (rows is None or rows.dtype == torch.int32)
    if n:
        _call("mx_layer_norm_rows", h.data_ptr(), _lib.ptr(rows), w.data_ptr(), b.data_ptr(), out.data_ptr(), n, h.shape[1], float(eps),
              _fp32(out), _lib.stream())
    return out
