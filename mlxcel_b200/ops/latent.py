"""Operators of multi-head latent attention over a latent pool (one ``[latent C | rotated key part R]`` row per token,
shared by the heads; pool ``[blocks, 1, block_size, C + R]`` in the K slab of its :class:`KVLayer`).

Two forms of the same attention: absorbed (queries ``[q W_uk | q_rot]`` against the pool rows, their first C columns as
values; decode rows, fp32, sizes the expanded form does not take) and expanded (per-head keys and values of the whole
context projected from gathered rows; prompt portions on the tcgen05 kernel). ``csrc/latent.cu``, ``csrc/attention_tc.cu``,
``csrc/simt.cu``; CPU tensors take the PyTorch statements below."""
from __future__ import annotations

import torch

from . import _decode_scratch, _lib
from .stream import NOT_COVERED, _call, _f, _fn, _fp32, _i, _ll, _rms, _SIG, _vp, rotate_half, visible

_SIG.update({
    "mx_latent_append": [_vp, _ll, _vp, _vp, _vp, _f, _vp, _vp, _vp, _i, _i, _i, _i, _f, _i, _i, _vp],
    "mx_latent_q_rope": [_vp, _ll, _i, _vp, _ll, _i, _vp, _vp, _f, _i, _i, _i, _i, _i, _vp],
    "mx_latent_gather": [_vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _vp],
    "mx_latent_head_tile": [_i],
    "mx_latent_decode": [_vp, _ll, _vp, _ll, _vp, _vp, _vp, _vp, _vp, _i, _i, _i, _i, _i, _i, _i, _f, _i, _i, _vp, _vp],
    "mx_latent_prefill": [_vp, _ll, _vp, _vp, _ll, _vp, _ll, _vp, _vp, _vp, _vp, _vp, _ll] + [_i] * 8 + [_f, _vp, _vp],
})
EXPANDED_TILE = 128      # keys per tile of the expanded form: a context gathered in part starts at a multiple of it


def latent_append(a, positions, slots, kv, *, Q: int, C: int, R: int, inv_freq, mscale: float, q_norm, c_norm, eps: float,
                  adjacent: bool = False) -> None:
    """Rows ``q latent [Q] | latent [C] | key part [R]``: the query latent is RMS-normalised in place, the latent normalised
    and the key part rotated into the pool (negative slots append nothing)."""
    if not a.is_cuda:
        f = a.float()
        if Q:
            a[:, :Q] = (_rms(f[:, :Q], eps) * q_norm).to(a.dtype)
        entry = torch.cat([_rms(f[:, Q:Q + C], eps) * c_norm, rotate_half(f[:, None, Q + C:Q + C + R], positions, inv_freq, mscale, adjacent)[:, 0]], -1)
        ok = slots >= 0
        kv.k.view(-1, C + R)[slots[ok].long()] = entry[ok].to(kv.k.dtype)
        return
    assert kv.k.dtype == a.dtype and a.stride(1) == 1 and slots.dtype == positions.dtype == torch.int32 and kv.k.shape[-1] == C + R
    if a.shape[0]:
        _call("mx_latent_append", a.data_ptr(), a.stride(0), positions.data_ptr(), slots.data_ptr(), inv_freq.data_ptr(), float(mscale),
              _lib.ptr(q_norm), c_norm.data_ptr(), kv.k.data_ptr(), a.shape[0], Q, C, R, float(eps), 1 if adjacent else 0, _fp32(a),
              _lib.stream())


def latent_q_rope(q, dst, positions, *, H: int, q_at: int, q_head: int, d_at: int, d_head: int, inv_freq, mscale: float,
                  adjacent: bool = False) -> None:
    """Rotates the R dimensions from ``q_at`` of every head (``q_head`` apart in the rows of q) into those from ``d_at`` of
    dst's heads; q and dst may be the same rows. ``adjacent``: neighbouring dimensions are turned, not the halves."""
    R = 2 * inv_freq.shape[0]
    if not q.is_cuda:
        n = q.shape[0]
        src = torch.stack([q[:, q_at + h * q_head:q_at + h * q_head + R] for h in range(H)], 1).float()
        rot = rotate_half(src, positions, inv_freq, mscale, adjacent).to(dst.dtype)
        for h in range(H if n else 0):
            dst[:, d_at + h * d_head:d_at + h * d_head + R] = rot[:, h]
        return
    assert q.stride(1) == 1 and dst.stride(1) == 1 and q.dtype == dst.dtype and positions.dtype == torch.int32
    if q.shape[0] and R:
        e = q.element_size()
        _call("mx_latent_q_rope", q.data_ptr() + q_at * e, q.stride(0), q_head, dst.data_ptr() + d_at * e, dst.stride(0), d_head,
              positions.data_ptr(), inv_freq.data_ptr(), float(mscale), q.shape[0], H, R, 1 if adjacent else 0, _fp32(q), _lib.stream())


def latent_splits(B: int, H: int, max_len: int, sms: int = 148) -> int:
    """KV splits of the absorbed decode kernel: one CTA per SM, at least two 64-token tiles each."""
    pairs = max(1, B * -(-H // (32 if H > 16 else 16)))
    return max(1, min(sms // pairs, max_len // 128, 64))


def latent_attention_ref(q, kv, tables, lens, cu, *, H: int, C: int, scale: float, window: int = 0, sinks=None):
    W = kv.k.shape[-1]
    flat = kv.k.view(-1, W)
    out = torch.zeros(q.shape[0], H * C, dtype=q.dtype, device=q.device)
    cu_l, lens_l = cu.tolist(), lens.tolist()
    for s, n in enumerate(lens_l):
        q0, q1 = cu_l[s], cu_l[s + 1]
        if q1 == q0 or n == 0:
            continue
        t = torch.arange(n)
        rows = flat[tables[s].long()[t // kv.block_size] * kv.block_size + t % kv.block_size].float()
        sc = torch.einsum("qhw,kw->hqk", q[q0:q1].float().view(-1, H, W), rows) * scale
        d = torch.arange(n - (q1 - q0), n)[:, None] - t[None, :]
        sc = sc.masked_fill((d < 0) | (d >= window) if window > 0 else d < 0, float("-inf"))
        if sinks is not None:
            sc = torch.cat([sc, sinks[:, None, None].expand(-1, q1 - q0, 1)], -1)
        out[q0:q1] = torch.einsum("hqk,kc->qhc", torch.softmax(sc, -1)[..., :n], rows[:, :C]).reshape(q1 - q0, H * C).to(q.dtype)
    return out


def latent_attention(q, kv, tables, lens, cu, out, *, H: int, C: int, scale: float, max_len: int = 0, window: int = 0, sinks=None,
                     force_any: bool = False, form: int = 0) -> None:
    """Causal attention of absorbed query rows [rows, H * (C + R)] over the latent pool into ``out`` [rows, H * C];
    ``window`` > 0: the last ``window`` tokens only; ``sinks`` adds ``exp(sink)`` to the denominator.
    ``cu=None`` says one row per sequence (decode): bf16 rows of at most 576 (latent 512) take the tensor-core kernels, which
    read every pool row once for up to 32 heads (tcgen05 for pages of 16 tokens; ``form`` 1: the mma.sync one everywhere); the
    rest the SIMT one."""
    rows, W = q.shape[0], kv.k.shape[-1]
    if rows == 0:
        return
    if not q.is_cuda:
        out.copy_(latent_attention_ref(q, kv, tables, lens, torch.arange(rows + 1) if cu is None else cu, H=H, C=C, scale=scale,
                                       window=window, sinks=sinks))
        return
    assert kv.k.dtype == q.dtype == out.dtype and q.stride(1) == 1 and out.is_contiguous()
    if q.dtype == torch.bfloat16 and cu is None and not force_any:
        splits = latent_splits(rows, H, visible(max_len or tables.shape[1] * kv.block_size, window))
        lib = _lib.load()
        floats = lib.mx_latent_decode_scratch_floats
        if not floats.argtypes:
            floats.argtypes, floats.restype = [_i] * 4, _ll
        scratch = _decode_scratch(q.device, int(floats(rows, H, C, splits)) if splits > 1 else 0)
        rc = _fn("mx_latent_decode")(q.data_ptr(), q.stride(0), kv.k.data_ptr(), kv.k.shape[0] * kv.block_size, tables.data_ptr(),
                                     lens.data_ptr(), _lib.ptr(sinks), out.data_ptr(), scratch.data_ptr(), rows, H, W, C, kv.block_size,
                                     tables.shape[1], window, float(scale), splits, form, _lib.workspace(q.device).data_ptr(), _lib.stream())
        if rc != NOT_COVERED:
            _lib.count_launch(2 if splits > 1 else 1)
            _lib.check(rc, "mx_latent_decode")
            return
    if cu is None:
        cu = torch.arange(rows + 1, dtype=torch.int32, device=q.device)
    _call("mx_paged_attention_any", q.data_ptr(), q.stride(0), kv.k.data_ptr(), kv.k.data_ptr(), tables.data_ptr(), cu.data_ptr(),
          lens.data_ptr(), _lib.ptr(sinks), None, None, None, 0, out.data_ptr(), out.stride(0), lens.shape[0], rows, H, 1, W, C, W, W,
          kv.block_size, tables.shape[1], window, 0, float(scale), 0.0, 1, 0.0, 1.0, 0.0, None, None, 0, _fp32(q), _lib.stream())


def latent_gather(kv, tables, bounds, rows: int, zero=None):
    """The pool rows of the sequences' contexts back to back: sequence s fills rows ``bounds[s]`` .. ``bounds[s + 1] - 1`` of
    the result, row r with its token ``r - zero[s]`` (default: from the first token on, ``zero = bounds``)."""
    W = kv.k.shape[-1]
    out = torch.empty(rows, W, dtype=kv.k.dtype, device=kv.k.device)
    _call("mx_latent_gather", kv.k.data_ptr(), tables.data_ptr(), bounds.data_ptr(), (bounds if zero is None else zero).data_ptr(),
          out.data_ptr(), rows, bounds.shape[0] - 1, W * kv.k.element_size(), kv.block_size, tables.shape[1], _lib.stream())
    return out


def expanded_covered(dtype, D: int, R: int, V: int, C: int, cuda: bool) -> bool:
    """Whether :func:`latent_prefill` takes these head sizes."""
    return cuda and dtype == torch.bfloat16 and not (D % 8 or R % 8 or V % 8 or C % 8) and D <= 128 and 0 < R <= 64 and V <= 128


def latent_prefill(q, kn, kr, v, cu, lens, starts, out, *, H: int, D: int, R: int, V: int, scale: float, max_q_len: int,
                   window: int = 0, sinks=None) -> None:
    """Causal attention of prompt portions over expanded rows: q [rows, H * (D + R)] (rotated), kn [ctx, H * D],
    kr [ctx, R] (columns of the gathered rows), v [ctx, H * V], token 0 of context s in row ``starts[s]`` (which may lie
    before the gathered rows if its window does not); into ``out`` [rows, H * V]. q and out may be column slices (a group of heads)."""
    _call("mx_latent_prefill", q.data_ptr(), q.stride(0), kn.data_ptr(), kr.data_ptr(), kr.stride(0), v.data_ptr(), kn.shape[0],
          cu.data_ptr(), lens.data_ptr(), starts.data_ptr(), _lib.ptr(sinks), out.data_ptr(), out.stride(0), lens.shape[0], q.shape[0],
          max_q_len, H, D, R, V, window, float(scale), _lib.workspace(q.device).data_ptr(), _lib.stream())
