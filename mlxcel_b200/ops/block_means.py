"""Block means beside a paged KV pool (``csrc/block_means.cu``; CPU tensors take the PyTorch statements): the mean key and
value of every full run of ``kv.mean_of`` tokens, counted from the sequence's start.

The mean of block b is kept in the page that holds the block's last token, at place ``b - (page * block_size) // mean_of`` of
that page. A token whose window begins at w sees the blocks ``b < w // mean_of`` beside the window's tokens."""
from __future__ import annotations

import torch

from . import _lib
from .stream import _call, _fp32, _i, _ll, _SIG, _vp

_SIG["mx_kv_append_means"] = [_vp, _ll] + [_vp] * 8 + [_i] * 10 + [_vp]
_SIG["mx_gather_means"] = [_vp] * 6 + [_i] * 9 + [_vp]


def mean_rows_ref(kv, table, n: int):
    """Dense fp32 means [Hkv, n, width] of keys and values of the first n blocks of one sequence."""
    b = torch.arange(n)
    page = ((b + 1) * kv.mean_of - 1) // kv.block_size
    at = b - page * kv.block_size // kv.mean_of
    t = table[page].long()
    return kv.k_mean[t, :, at].float().transpose(0, 1), kv.v_mean[t, :, at].float().transpose(0, 1)


def append_ref(row, positions, slots, kv, tables, cu, Hq, Hkv, Dk, Dv):
    T, nq, nk, P, bs = row.shape[0], Hq * Dk, Hkv * Dk, kv.mean_of, kv.block_size
    k, v = row[:, nq:nq + nk].reshape(T, Hkv, Dk), row[:, nq + nk:nq + nk + Hkv * Dv].reshape(T, Hkv, Dv)
    for t in range(T):
        if int(slots[t]) >= 0:
            blk, off = divmod(int(slots[t]), bs)
            kv.k[blk, :, off], kv.v[blk, :, off] = k[t].to(kv.k.dtype), v[t].to(kv.v.dtype)
    c = list(range(T + 1)) if cu is None else cu.tolist()
    for s in range(len(c) - 1):
        for t in range(c[s], c[s + 1]):
            pos = int(positions[t])
            if int(slots[t]) < 0 or (pos + 1) % P:
                continue
            p = torch.arange(pos + 1 - P, pos + 1)
            pages, off = tables[s][p // bs].long(), p % bs
            page = pos // bs
            at = (pos + 1) // P - 1 - page * bs // P
            dst = int(tables[s][page])
            for mean, pool in ((kv.k_mean, kv.k), (kv.v_mean, kv.v)):
                mean[dst, :, at] = pool[pages, :, off].float().mean(0).to(mean.dtype)


def append(row, positions, slots, kv, tables, cu, *, Hq: int, Hkv: int, Dk: int, Dv: int) -> None:
    """Rows ``q | k | v | ...`` of one group of sequences (``cu=None``: one row each): k and v into the paged pool (negative
    slots append nothing), and the means of the blocks these tokens complete."""
    if row.shape[0] == 0:
        return
    if not row.is_cuda:
        return append_ref(row, positions, slots, kv, tables, cu, Hq, Hkv, Dk, Dv)
    assert kv.k.dtype == row.dtype and row.stride(1) == 1 and slots.dtype == torch.int32 and positions.dtype == torch.int32
    _call("mx_kv_append_means", row.data_ptr(), row.stride(0), positions.data_ptr(), slots.data_ptr(), tables.data_ptr(), _lib.ptr(cu),
          kv.k.data_ptr(), kv.v.data_ptr(), kv.k_mean.data_ptr(), kv.v_mean.data_ptr(), row.shape[0], tables.shape[0], Hq, Hkv,
          Dk, Dv, kv.block_size, tables.shape[1], kv.mean_of, _fp32(row), _lib.stream())


def seen(context: int, window: int, mean_of: int) -> int:
    """Blocks the last of ``context`` tokens sees."""
    return max(0, context - window) // mean_of


def portion_means(b, window: int, mean_of: int):
    """Rows of the gathered matrix the prompt portions' means take: (bounds [portions + 1] int32, rows in all), computed once
    per batch, window and block size."""
    cache = b.__dict__.setdefault("_portion_means", {})
    got = cache.get((window, mean_of))
    if got is None:
        if b.pf_cu_q_host is not None and b.pf_starts is not None:
            ends = [s + b.pf_cu_q_host[i + 1] - b.pf_cu_q_host[i] for i, s in enumerate(b.pf_starts)]
        else:
            ends = b.pf_context_lens.tolist()
        bounds = [0]
        for n in ends:
            bounds.append(bounds[-1] + seen(n, window, mean_of))
        got = cache[(window, mean_of)] = (torch.tensor(bounds, dtype=torch.int32).to(b.pf_context_lens.device), bounds[-1])
    return got


def gather(kv, tables, bounds, rows: int):
    """The first ``bounds[s + 1] - bounds[s]`` block means of every sequence as dense matrices ([rows, Hkv, Dk], [rows, Hkv, Dv])."""
    (_, H, per, Dk), Dv = kv.k_mean.shape, kv.v_mean.shape[3]
    k, v = (torch.empty(rows, H, w, dtype=kv.k.dtype, device=kv.k.device) for w in (Dk, Dv))
    if rows:
        es = kv.k.element_size()
        _call("mx_gather_means", kv.k_mean.data_ptr(), kv.v_mean.data_ptr(), tables.data_ptr(), bounds.data_ptr(), k.data_ptr(), v.data_ptr(),
              rows, bounds.shape[0] - 1, H, Dk * es, Dv * es, per, kv.block_size, tables.shape[1], kv.mean_of, _lib.stream())
    return k, v
