"""Operators of layers with an fp32 residual stream: sub-layer norms before and / or behind a branch,
polynomial-norm activation, soft cap, q/k norm (before or behind a rotation) + KV append, paged attention with
chunks, soft cap, a logarithmic distance bias, sink, output gate and separate key and value widths, the
generalized delta rule.

Every operator exists for bf16 and fp32 activations on CUDA (``csrc/stream_norm.cu``, ``csrc/rope_norm.cu``,
``csrc/simt.cu``, ``csrc/attention*.cu``, ``csrc/delta_rule.cu``); CPU tensors take the PyTorch statements below. Norm weights,
layer scales and per-head constants are fp32 vectors."""
from __future__ import annotations

import ctypes
import math
from dataclasses import dataclass

import torch

from . import _lib
from .reference import _gather_kv

_vp, _i, _f, _ll = ctypes.c_void_p, ctypes.c_int, ctypes.c_float, ctypes.c_longlong
_SIG = {
    "mx_stream_norm": [_vp] * 7 + [_i, _i, _f, _f, _i, _vp, _vp],
    "mx_embed_stream": [_vp] * 7 + [_i, _i, _i, _f, _f, _f, _i, _vp],
    "mx_polynorm": [_vp, _vp, _vp, _i, _i, _f, _i, _vp],
    "mx_softcap_rows": [_vp, _ll, _f, _vp],
    "mx_rope_norm_append": [_vp, _ll, _vp, _vp, _vp, _f] + [_vp] * 4 + [_i] * 9 + [_f, _i, _vp],
    "mx_qk_norm_append": [_vp, _ll, _vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _i, _f, _i, _vp],
    "mx_paged_attention_any": [_vp, _ll] + [_vp] * 9 + [_ll, _vp, _ll] + [_i] * 12 + [_f, _f, _i, _f, _f, _f, _vp, _vp, _i, _i, _vp],
    "mx_paged_decode_ext": [_vp, _ll] + [_vp] * 8 + [_ll, _vp, _ll, _vp] + [_i] * 9 + [_f, _f, _i, _f, _f, _f, _vp, _vp, _i, _i, _vp],
    "mx_paged_prefill_ext": [_vp, _ll, _vp, _vp, _ll] + [_vp] * 7 + [_ll, _vp, _ll] + [_i] * 11 + [_f, _f, _i, _f, _f, _f, _vp, _vp, _vp, _i, _i,
                                                                                                    _vp, _vp],
    "mx_delta_rule": [_vp, _ll] + [_vp] * 11 + [_i] * 6 + [_f, _f, _f, _i, _i, _vp],
}
NOT_COVERED = -10        # a tensor-core kernel refuses the geometry: the shape-agnostic one takes it


def _fn(name):
    fn = getattr(_lib.load(), name)
    if not fn.argtypes:
        fn.argtypes, fn.restype = _SIG[name], _i
    return fn


def _call(name, *args) -> None:
    rc = _fn(name)(*args)
    _lib.count_launch()
    _lib.check(rc, name)


def _fp32(t: torch.Tensor) -> int:
    if t.dtype not in (torch.float32, torch.bfloat16):
        raise TypeError(f"activations must be fp32 or bf16, not {t.dtype}")
    return 1 if t.dtype == torch.float32 else 0


def visible(max_len: int, span: int, means: int = 0) -> int:
    """Keys a query sees at most: a window or chunk of ``span`` tokens (0: all) of ``max_len`` and, with ``means``, one for every
    block of so many tokens before the window."""
    if span <= 0:
        return max_len
    return min(max_len, span) + (max(0, max_len - span) // means if means else 0)


def _rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + eps)


# ----------------------------------------------------------------------------- residual stream
class _StreamExtras(ctypes.Structure):
    """Mirror of ``MxStreamExtras`` (csrc/api.h): what a step of the stream adds besides a branch."""

    _fields_ = [("moe_y", _vp), ("moe_shared", _vp), ("moe_x", _vp), ("moe_ids", _vp), ("moe_inv", _vp), ("moe_w", _vp),
                ("moe_k", _i), ("moe_experts", _i), ("vec", _vp), ("ids", _vp), ("table", _vp), ("vocab", _i), ("emb_scale", _f)]


@dataclass
class Entry:
    """What is added to the stream ahead of a run of layers: a vector and, with ``ids``, the tokens' embedding again."""

    vec: torch.Tensor                     # fp32 [dim]
    ids: torch.Tensor | None = None
    table: torch.Tensor | None = None
    scale: float = 1.0

    def add_to(self, h) -> None:
        if self.ids is not None:
            ok = (self.ids >= 0) & (self.ids < self.table.shape[0])
            h += self.table[self.ids.clamp(0, self.table.shape[0] - 1).long()].float() * self.scale * ok[:, None]
        h += self.vec


def embed_stream(ids, table, scale: float, pre_w, eps: float, w_bias: float, own_w=None, vec=None):
    """``h = scale * table[ids]`` (fp32 stream; with ``own_w`` the embedding's own norm: ``rmsnorm(.) * (w_bias + own_w)``;
    plus the fp32 vector ``vec``) and ``x = rmsnorm(h) * (w_bias + pre_w)`` in the table's type; without ``pre_w``, x is h itself."""
    n, dim = ids.shape[0], table.shape[1]
    if not table.is_cuda:
        ok = (ids >= 0) & (ids < table.shape[0])
        h = table[ids.clamp(0, table.shape[0] - 1).long()].float() * scale * ok[:, None]
        h = h if own_w is None else _rms(h, eps) * (w_bias + own_w)
        h = h if vec is None else h + vec
        return h, _stream_as(h, table.dtype) if pre_w is None else (_rms(h, eps) * (w_bias + pre_w)).to(table.dtype)
    h = torch.empty(n, dim, dtype=torch.float32, device=table.device)
    alias = pre_w is None and table.dtype == torch.float32       # (the branch has read the stream before it is added to it)
    x = None if alias else torch.empty(n, dim, dtype=table.dtype, device=table.device)
    if n:
        _call("mx_embed_stream", ids.data_ptr(), table.data_ptr(), h.data_ptr(), _lib.ptr(own_w), _lib.ptr(vec), _lib.ptr(pre_w),
              _lib.ptr(x), n, dim, table.shape[0], float(scale), float(eps), float(w_bias), _fp32(table), _lib.stream())
    return h, h if alias else x


def _stream_as(h, dtype):
    return h if h.dtype == dtype else h.to(dtype)


def stream_norm(h, y, post_w, layer_scale, pre_w, eps: float, w_bias: float, dtype=None, rows=None, plain: bool = False,
                moe=None, entry: Entry | None = None):
    """One step of the stream between two sub-layers, in place on ``h`` (fp32): with a branch ``y``,
    ``h += rmsnorm(y) * (w_bias + post_w) * layer_scale`` (without ``post_w``, y as it is; layer_scale optional); with ``moe``
    (:class:`~mlxcel_b200.ops.moe.MoeRows`) the weighted sum of a token's experts; then what ``entry`` adds. With ``pre_w``,
    returns ``rmsnorm(h) * (w_bias + pre_w)`` as ``dtype`` (default: y's type); with ``plain`` (and no ``pre_w``) the
    stream itself as ``dtype``. ``rows`` (int32, nothing to add) selects the rows of h to normalise."""
    dtype = dtype or y.dtype
    assert rows is None or (y is None and moe is None and entry is None)
    if not h.is_cuda:
        if y is not None:
            b = y.float() if post_w is None else _rms(y.float(), eps) * (w_bias + post_w)
            h += b if layer_scale is None else b * layer_scale
        if moe is not None:
            h += moe.summed()
        if entry is not None:
            entry.add_to(h)
        if pre_w is None:
            return _stream_as(h, dtype) if plain else None
        return (_rms(h if rows is None else h[rows.long()], eps) * (w_bias + pre_w)).to(dtype)
    dim = h.shape[1]
    n = h.shape[0] if rows is None else rows.shape[0]
    alias = plain and pre_w is None and dtype == torch.float32
    x = torch.empty(n, dim, dtype=dtype, device=h.device) if pre_w is not None or (plain and not alias) else None
    assert h.is_contiguous() and (y is None or (y.is_contiguous() and y.dtype == dtype))
    assert rows is None or rows.dtype == torch.int32
    ex = None
    if moe is not None or entry is not None:
        ex = _StreamExtras()
        if moe is not None:
            assert moe.x.dtype == dtype and moe.x.is_contiguous() and moe.y.dtype == dtype and moe.x.shape == h.shape
            ex.moe_y, ex.moe_x, ex.moe_ids, ex.moe_inv, ex.moe_w = (t.data_ptr() for t in (moe.y, moe.x, moe.ids, moe.inv, moe.wts))
            ex.moe_shared, ex.moe_k, ex.moe_experts = _lib.ptr(moe.shared), moe.ids.shape[1], moe.experts
        if entry is not None:
            ex.vec = entry.vec.data_ptr()
            if entry.ids is not None:
                assert entry.table.dtype == dtype
                ex.ids, ex.table, ex.vocab, ex.emb_scale = entry.ids.data_ptr(), entry.table.data_ptr(), entry.table.shape[0], entry.scale
    if n:
        fp32 = 1 if dtype == torch.float32 else 0
        _call("mx_stream_norm", _lib.ptr(y), h.data_ptr(), _lib.ptr(rows), _lib.ptr(post_w), _lib.ptr(layer_scale),
              _lib.ptr(pre_w), _lib.ptr(x), n, dim, float(eps), float(w_bias), fp32, _lib.ref_or_null(ex), _lib.stream())
    return h if alias else x


def polynorm(z, coef, eps: float):
    """``a N(z) + b N(z^2) + c N(z^3) + e`` over the last dimension, N(x) = x / rms(x); coef = (a, b, c, e) fp32."""
    if not z.is_cuda:
        f = z.float()
        return (coef[0] * _rms(f, eps) + coef[1] * _rms(f ** 2, eps) + coef[2] * _rms(f ** 3, eps) + coef[3]).to(z.dtype)
    assert z.is_contiguous()
    out = torch.empty_like(z)
    if z.shape[0]:
        _call("mx_polynorm", z.data_ptr(), coef.data_ptr(), out.data_ptr(), z.shape[0], z.shape[1], float(eps), _fp32(z),
              _lib.stream())
    return out


def softcap_(x, cap: float):
    """``cap tanh(x / cap)`` on fp32 values, in place."""
    if not x.is_cuda:
        return x.copy_(cap * torch.tanh(x / cap))
    assert x.dtype == torch.float32 and x.is_contiguous()
    if x.numel():
        _call("mx_softcap_rows", x.data_ptr(), x.numel(), float(cap), _lib.stream())
    return x


# ----------------------------------------------------------------------------- attention
def rotate_half(x, positions, inv_freq, mscale: float, adjacent: bool = False):
    """x [T, H, D] fp32: dimension i turned with i + R / 2 by ``positions * inv_freq[i]`` (R = 2 len(inv_freq)), both
    times ``mscale``; dimensions from R on pass. ``adjacent``: dimension 2 i turned with 2 i + 1 instead."""
    half = inv_freq.shape[0]
    a = (positions.float()[:, None] * inv_freq)[:, None]
    c, s = a.cos() * mscale, a.sin() * mscale
    if adjacent:
        u, v = x[..., 0:2 * half:2], x[..., 1:2 * half:2]
        turned = torch.stack([u * c - v * s, v * c + u * s], -1).flatten(-2)
        return torch.cat([turned, x[..., 2 * half:]], -1)
    u, v = x[..., :half], x[..., half:2 * half]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * half:]], -1)


def rope_norm_append(row, positions, slots, kv, *, Hq: int, Hkv: int, Dk: int, Dv: int, inv_freq, mscale: float = 1.0,
                     unit: bool = True, values_are_keys: bool = False, q_norm=None, k_norm=None, eps: float = 1e-6) -> None:
    """Rows ``q | k (| v)``: q (in place) and k are rotated by their positions, then divided per head by their root
    mean square (``unit``) and multiplied by an optional weight; k and v go into the paged pool (negative slots append
    nothing). ``values_are_keys``: no v columns, the values are the keys as projected."""
    if not row.is_cuda:
        T, nq, nk = row.shape[0], Hq * Dk, Hkv * Dk
        q, k = row[:, :nq].float().view(T, Hq, Dk), row[:, nq:nq + nk].float().view(T, Hkv, Dk)
        v = row[:, nq:nq + nk] if values_are_keys else row[:, nq + nk:nq + nk + Hkv * Dv]
        v = v.reshape(T, Hkv, Dv).clone()

        def turned(x, w):
            x = rotate_half(x, positions, inv_freq, mscale)
            x = _rms(x, eps) if unit else x
            return x if w is None else x * w
        row[:, :nq] = turned(q, q_norm).reshape(T, nq).to(row.dtype)
        ok = slots >= 0
        s = slots[ok].long()
        blk, off = s // kv.block_size, s % kv.block_size
        kv.k[blk, :, off] = turned(k, k_norm)[ok].to(kv.k.dtype)
        kv.v[blk, :, off] = v[ok].to(kv.v.dtype)
        return
    assert kv.k.dtype == row.dtype and row.stride(1) == 1 and slots.dtype == torch.int32 and positions.dtype == torch.int32
    if row.shape[0]:
        _call("mx_rope_norm_append", row.data_ptr(), row.stride(0), positions.data_ptr(), slots.data_ptr(), inv_freq.data_ptr(),
              float(mscale), kv.k.data_ptr(), kv.v.data_ptr(), _lib.ptr(q_norm), _lib.ptr(k_norm), row.shape[0], Hq, Hkv, Dk, Dv,
              2 * inv_freq.shape[0], 1 if values_are_keys else 0, 1 if unit else 0, kv.block_size, float(eps), _fp32(row),
              _lib.stream())


def qk_norm_append(qkv, slots, kv, *, Hq: int, Hkv: int, Dk: int, Dv: int, q_norm, k_norm, eps: float) -> None:
    """Rows ``q | k | v | ...``: per-head RMS norm of q (in place) and k, then k and v into the paged pool
    (negative slots append nothing). No positional encoding."""
    if not qkv.is_cuda:
        T, nq, nk = qkv.shape[0], Hq * Dk, Hkv * Dk
        q, k, v = qkv[:, :nq].float().view(T, Hq, Dk), qkv[:, nq:nq + nk].float().view(T, Hkv, Dk), \
            qkv[:, nq + nk:nq + nk + Hkv * Dv].view(T, Hkv, Dv)
        if q_norm is not None:
            qkv[:, :nq] = (_rms(q, eps) * q_norm).reshape(T, nq).to(qkv.dtype)
        k = _rms(k, eps) * k_norm if k_norm is not None else k
        ok = slots >= 0
        s = slots[ok].long()
        blk, off = s // kv.block_size, s % kv.block_size
        kv.k[blk, :, off] = k[ok].to(kv.k.dtype)
        kv.v[blk, :, off] = v[ok].to(kv.v.dtype)
        return
    assert kv.k.dtype == qkv.dtype and qkv.stride(1) == 1 and slots.dtype == torch.int32
    if qkv.shape[0]:
        _call("mx_qk_norm_append", qkv.data_ptr(), qkv.stride(0), slots.data_ptr(), kv.k.data_ptr(), kv.v.data_ptr(),
              _lib.ptr(q_norm), _lib.ptr(k_norm), qkv.shape[0], Hq, Hkv, Dk, Dv, kv.block_size, float(eps), _fp32(qkv),
              _lib.stream())


def paged_attention_ref(q, kv, tables, lens, cu, *, Hq, Hkv, Dk, Dv, scale, window=0, sinks=None, dist_bias=None, gate=None,
                        softcap=0.0, chunk=0, diff=None, means=False, gain=1.0):
    if diff is not None:
        # the maps as two attentions whose queries are zero in the other map's columns
        factor, gain, eps = diff
        q3, a, common = q.reshape(-1, Hq, 2, Dk // 2), [], dict(Hq=Hq, Hkv=Hkv, Dk=Dk, Dv=Dv, scale=scale, window=window, chunk=chunk)
        for i in (0, 1):
            one = torch.zeros_like(q3)
            one[:, :, i] = q3[:, :, i]
            a.append(paged_attention_ref(one.reshape(q.shape[0], -1).float(), kv, tables, lens, cu, **common).view(-1, Hq, Dv))
        return (_rms(a[0] - factor * a[1], eps) * gain).reshape(-1, Hq * Dv).to(q.dtype)
    T, G = q.shape[0], Hq // Hkv
    out = torch.zeros(T, Hq * Dv, dtype=q.dtype, device=q.device)
    cu_l, lens_l = cu.tolist(), lens.tolist()
    for s in range(len(lens_l)):
        q0, q1, n = cu_l[s], cu_l[s + 1], lens_l[s]
        ql = q1 - q0
        if ql == 0 or n == 0:
            continue
        k, v = _gather_kv(kv, tables[s], n)
        qs = q[q0:q1].float().reshape(ql, Hkv, G, Dk).permute(1, 2, 0, 3)
        sc = torch.einsum("hgqd,hkd->hgqk", qs, k) * scale
        sc = softcap * torch.tanh(sc / softcap) if softcap > 0 else sc
        qp, kp = torch.arange(n - ql, n, device=q.device)[:, None], torch.arange(n, device=q.device)[None, :]
        d = qp - kp
        if dist_bias is not None:
            r1, r2 = (t.float().reshape(Hkv, G, 1, 1) for t in dist_bias)
            sc = sc - r1 * torch.log1p(r2 * d.clamp(min=0).float())
        vis = (d >= 0) & (d < window) if window > 0 else d >= 0
        vis = vis & (kp // chunk == qp // chunk) if chunk > 0 else vis
        sc = sc.masked_fill(~vis, float("-inf"))
        if means:
            # blocks of tokens that lie wholly before a query's window, as one key and value each
            from .block_means import mean_rows_ref
            nb = max(0, n - window) // kv.mean_of
            km, vm = mean_rows_ref(kv, tables[s], nb)
            old = (torch.arange(nb, device=q.device)[None] + 1) * kv.mean_of <= qp - window + 1
            ms = torch.einsum("hgqd,hkd->hgqk", qs, km) * scale
            sc, v = torch.cat([sc, ms.masked_fill(~old, float("-inf"))], -1), torch.cat([v, vm], 1)
        if sinks is not None:
            sc = torch.cat([sc, sinks.float().reshape(Hkv, G, 1, 1).expand(Hkv, G, ql, 1)], -1)
        p = torch.softmax(sc, -1)[..., :v.shape[1]]
        o = gain * torch.einsum("hgqk,hkd->hgqd", p, v).permute(2, 0, 1, 3).reshape(ql, Hq * Dv)
        if gate is not None:
            o = o * torch.sigmoid(gate[q0:q1].float())
        out[q0:q1] = o.to(q.dtype)
    return out


def paged_attention(q, kv, tables, lens, cu, out, *, Hq: int, Hkv: int, Dk: int, Dv: int, scale: float, max_q_len: int,
                    max_len: int = 0, window: int = 0, sinks=None, dist_bias=None, gate=None, softcap: float = 0.0, chunk: int = 0,
                    diff: tuple | None = None, means: tuple | None = None, gain: float = 1.0, force_any: bool = False) -> None:
    """Causal paged attention of the query rows of every sequence (the last ``cu[s+1] - cu[s]`` of its ``lens[s]``
    tokens) into ``out`` [rows, Hq * Dv]. ``cu=None`` says one row per sequence (decode).

    scores: ``q.k * scale``, with ``softcap`` > 0 ``softcap tanh(. / softcap)``, then ``- r1 ln(1 + r2 distance)`` with
    ``dist_bias = (r1, r2)`` per query head; ``chunk`` > 0: a token sees only keys of its own run of ``chunk`` positions
    (counted from the sequence's start); ``sinks`` adds ``exp(sink)`` to the denominator; ``gate`` ([rows, Hq * Dv], may be a column slice) multiplies the result by
    its sigmoid; ``diff = (factor, gain, eps)``: differential heads, the Dk columns of a query and key head are two maps of
    Dk / 2 (scores and softmax of their own, the same values) and the result is ``a1 - factor a2`` over its root mean square,
    times ``gain``; ``means`` (with a window): the blocks of ``kv.mean_of`` tokens wholly before a query's window are keys too, by
    their means; for prompt portions ``(bounds, rows)`` of :func:`block_means.portion_means`, for decode rows any tuple;
    ``gain`` multiplies the heads. ``out`` may be a column slice. bf16 pools with row widths that are multiples of 8 up to 128 take the tensor-core kernels
    (flash decoding with split KV; tcgen05 prefill); the rest the SIMT one."""
    rows = q.shape[0]
    if rows == 0:
        return
    if not q.is_cuda:
        c = torch.arange(rows + 1) if cu is None else cu
        out.copy_(paged_attention_ref(q, kv, tables, lens, c, Hq=Hq, Hkv=Hkv, Dk=Dk, Dv=Dv, scale=scale, window=window,
                                      sinks=sinks, dist_bias=dist_bias, gate=gate, softcap=softcap, chunk=chunk, diff=diff,
                                      means=means is not None, gain=gain))
        return
    assert gain == 1.0 or diff is None
    assert means is None or (window > 0 and kv.mean_of > 0 and chunk == 0 and dist_bias is None and diff is None), "block means stand beside a window"
    assert diff is None or (Dk % 2 == 0 and sinks is None and dist_bias is None and gate is None), "differential heads: plain scores"
    maps, (lam, gain, eps) = (1, (0.0, gain, 0.0)) if diff is None else (2, diff)
    dargs = (maps, float(lam), float(gain), float(eps))
    r1, r2 = dist_bias if dist_bias is not None else (None, None)
    assert kv.k.dtype == q.dtype and q.stride(1) == 1 and out.stride(1) == 1 and out.dtype == q.dtype
    km, vm, P = (kv.k_mean.data_ptr(), kv.v_mean.data_ptr(), kv.mean_of) if means is not None else (None, None, 0)
    assert gate is None or (gate.stride(1) == 1 and gate.dtype == q.dtype)
    gs = gate.stride(0) if gate is not None else 0
    head = (q.data_ptr(), q.stride(0), kv.k.data_ptr(), kv.v.data_ptr())
    tail = (_lib.ptr(sinks), _lib.ptr(r1), _lib.ptr(r2), _lib.ptr(gate), gs, out.data_ptr(), out.stride(0))
    if q.dtype == torch.bfloat16 and not force_any and Dk % 8 == Dv % 8 == 0:
        from . import _decode_scratch, decode_splits
        if cu is None:
            splits = decode_splits(rows, Hkv, visible(max_len or tables.shape[1] * kv.block_size, window or chunk, P))
            scratch = _decode_scratch(q.device, int(_lib.load().mx_paged_decode_scratch_floats(rows, maps * Hq, Dv, splits)))
            rc = _fn("mx_paged_decode_ext")(*head, tables.data_ptr(), lens.data_ptr(), *tail, scratch.data_ptr(), rows, Hq,
                                            Hkv, Dk, Dv, kv.block_size, tables.shape[1], window, chunk, float(scale),
                                            float(softcap), *dargs, km, vm, P, splits, _lib.stream())
        else:
            gathered = (None, None, None, 0)
            if means is not None and means[1]:
                from .block_means import gather
                gk, gv = gather(kv, tables, *means)
                gathered = (gk.data_ptr(), gv.data_ptr(), means[0].data_ptr(), means[1])
            rc = _fn("mx_paged_prefill_ext")(*head, kv.k.shape[0], tables.data_ptr(), cu.data_ptr(), lens.data_ptr(), *tail,
                                             lens.shape[0], rows, max_q_len, Hq, Hkv, Dk, Dv, kv.block_size, tables.shape[1],
                                             window, chunk, float(scale), float(softcap), *dargs, *gathered, P,
                                             _lib.workspace(q.device).data_ptr(), _lib.stream())
        if rc != NOT_COVERED:
            _lib.count_launch()
            _lib.check(rc, "paged attention")
            return
    if cu is None:
        cu = torch.arange(rows + 1, dtype=torch.int32, device=q.device)
    _call("mx_paged_attention_any", *head, tables.data_ptr(), cu.data_ptr(), lens.data_ptr(), *tail, lens.shape[0], rows, Hq,
          Hkv, Dk, Dv, Dk, Dv, kv.block_size, tables.shape[1], window, chunk, float(scale), float(softcap), *dargs, km, vm, P,
          _fp32(q), _lib.stream())


# ----------------------------------------------------------------------------- generalized delta rule
DELTA_DECAY_SCALE = math.exp(-0.5)       # largest decay exponent: w = exp(-exp(-1/2) sigmoid(.))
DELTA_UNIT_EPS = 1e-6                    # inside the root of the unit key


def delta_rule_ref(proj, offs, w2, w0, a_bias, norm_w, state, slots, cu, reset, D: int, norm_eps: float,
                   decay_scale: float = DELTA_DECAY_SCALE, unit_eps: float = DELTA_UNIT_EPS):
    H = state.shape[1]
    HD, R = H * D, w2.shape[1]
    f = proj.float()
    r, k, v, g, a = (f[:, o:o + HD].reshape(-1, H, D) for o in offs[:5])
    z = torch.tanh(f[:, offs[5]:offs[5] + R]) @ w2.float().t() + w0
    w = torch.exp(-decay_scale * torch.sigmoid(z)).reshape(-1, H, D)
    a = torch.sigmoid(a + a_bias.reshape(H, D))
    u = k / torch.sqrt(k.pow(2).sum(-1, keepdim=True) + unit_eps)
    o = torch.zeros(f.shape[0], H, D, device=proj.device)
    sl, rs, c = slots.tolist(), reset.tolist(), cu.tolist()
    for j in range(len(sl)):
        if sl[j] < 0 or c[j + 1] <= c[j]:
            continue
        S = torch.zeros_like(state[0]) if rs[j] else state[sl[j]].clone()
        for t in range(c[j], c[j + 1]):
            read = (u[t][:, :, None] * S).sum(1)
            S = w[t][:, :, None] * S - (a[t] * u[t])[:, :, None] * read[:, None, :] + k[t][:, :, None] * v[t][:, None, :]
            o[t] = (S * r[t][:, :, None]).sum(1)
        state[sl[j]] = S
    y = _rms(o, norm_eps).reshape(-1, HD) * norm_w * torch.sigmoid(g.reshape(-1, HD))
    return y.to(proj.dtype)


def delta_rule(proj, offs, w2, w0, a_bias, norm_w, state, slots, cu, reset, *, D: int, norm_eps: float, n_short: int = 0,
               decay_scale: float = DELTA_DECAY_SCALE, unit_eps: float = DELTA_UNIT_EPS, force_any: bool = False):
    """Generalized delta rule over a ragged batch with its preparation, per-head output norm and gate.

    ``proj`` rows hold r, k, v, gate, removal-rate and low-rank decay pre-activations at the element offsets
    ``offs = (r, k, v, g, a, l)``; ``w2`` [H*D, R] lifts ``tanh(l)``; ``w0``, ``a_bias``, ``norm_w`` [H*D] fp32;
    ``state`` [slots, H, D, D] fp32 is advanced in place; ``slots`` / ``reset`` [pieces], ``cu`` [pieces + 1] int32
    (the first ``n_short`` pieces are decode rows of one token; a negative slot marks a padding row).
    Returns [rows, H * D] in proj's type, ready for the output projection."""
    if not proj.is_cuda:
        return delta_rule_ref(proj, offs, w2, w0, a_bias, norm_w, state, slots, cu, reset, D, norm_eps, decay_scale, unit_eps)
    H, rows = state.shape[1], proj.shape[0]
    assert proj.stride(1) == 1 and w2.is_contiguous() and w2.dtype == proj.dtype and state.is_contiguous()
    out = torch.empty(rows, H * D, dtype=proj.dtype, device=proj.device)
    pieces = slots.shape[0]
    scratch = None
    if pieces > n_short and not force_any:
        scratch = torch.empty((rows - n_short) * H * (6 * D + 2), dtype=torch.float32, device=proj.device)
    arr = (ctypes.c_int * 6)(*[int(o) for o in offs])
    _call("mx_delta_rule", proj.data_ptr(), proj.stride(0), ctypes.cast(arr, ctypes.c_void_p), w2.data_ptr(), w0.data_ptr(),
          a_bias.data_ptr(), norm_w.data_ptr(), state.data_ptr(), slots.data_ptr(), cu.data_ptr(), reset.data_ptr(),
          out.data_ptr(), _lib.ptr(scratch), pieces, n_short, rows, H, D, w2.shape[1], float(decay_scale), float(unit_eps),
          float(norm_eps), _fp32(proj), 1 if force_any else 0, _lib.stream())
    if not force_any:
        _lib.count_launch((1 if n_short and pieces > n_short else 0) + (2 if pieces > n_short else 0))
    return out
