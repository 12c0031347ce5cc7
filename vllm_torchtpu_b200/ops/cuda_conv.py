"""Bindings of the convolved-attention kernels (``csrc/conv_cache.cu``)."""
from __future__ import annotations

from ctypes import c_float, c_int, c_longlong, c_void_p

import torch

from . import count_launch
from . import cuda as _c


def _call(p, row, q, kv_cache, ring, meta, R, ring_from, single, only_ring):
    assert row.stride(1) == 1 and ring.is_contiguous() and ring.dtype == p.conv_w.dtype == row.dtype
    nb, bs = (kv_cache.shape[0], kv_cache.shape[3]) if kv_cache is not None else (0, 16)
    inv = p.inv_freq
    _c._check(_c.lib().b200_conv_cache(
        _c._p(row), c_int(row.stride(0)), *(c_int(o) for o in p.offsets), _c._p(p.conv_w), c_int(p.taps), _c._p(ring),
        _c._p(inv), c_int(inv.numel() if inv is not None else 0), c_float(p.rot_mult), _c._p(q),
        _c._p(kv_cache) if p.kv_heads else c_void_p(0), _c._p(meta.slot_mapping), _c._p(meta.query_start_loc),
        _c._p(meta.seq_lens), _c._p(meta.state_slots), c_int(row.shape[0]), c_int(R), c_int(p.heads), c_int(p.kv_heads),
        c_int(p.dim), c_int(p.vdim), c_int(p.maps), c_int(p.width), c_int(bs), c_longlong(nb), c_int(ring_from),
        c_int(int(single)), c_int(int(only_ring)), c_int(_c._mixed(row)), _c._stream()), "conv_cache")


def conv_and_cache(plan, row, kv_cache, ring, meta):
    """See ``ops.short_conv.conv_and_cache``."""
    T, R, nd = row.shape[0], meta.num_reqs, meta.num_decode_reqs
    assert not plan.kv_heads or (kv_cache.dtype == row.dtype and kv_cache.is_contiguous())
    q = torch.empty((T, plan.heads * plan.maps, plan.width), dtype=row.dtype, device=row.device)
    single = nd == R
    R_launch = meta.padded_num_reqs if single and meta.padded_num_reqs is not None else R
    _call(plan, row, q, kv_cache, ring, meta, R_launch, R_launch if single else nd, single, False)
    count_launch(1 if single or plan.taps == 1 else 2)
    return q


def conv_ring_update(plan, row, ring, meta) -> None:
    _call(plan, row, None, None, ring, meta, meta.num_reqs, 0, False, True)
    count_launch()


def combine_heads(a, vdim: int, gate=None, lam=None, diff: float = 0.0, eps: float = 0.0):
    """See ``ops.short_conv.combine_heads``; without ``lam`` in place."""
    T, rows, D = a.shape
    assert a.is_contiguous() and (gate is None or (gate.stride(1) == 1 and gate.dtype == a.dtype))
    heads = rows // 2 if lam is not None else rows
    out = torch.empty((T, heads, D), dtype=a.dtype, device=a.device) if lam is not None else a
    _c._check(_c.lib().b200_combine_heads(
        _c._p(a), _c._p(gate), c_int(gate.stride(0) if gate is not None else 0), _c._p(lam), _c._p(out), c_int(T),
        c_int(heads), c_int(D), c_int(vdim), c_float(diff), c_float(eps), c_int(_c._mixed(a)), _c._stream()),
        "combine_heads")
    count_launch()
    return out
