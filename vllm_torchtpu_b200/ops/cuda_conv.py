"""Bindings of the convolved-attention kernels (``csrc/conv_cache.cu``)."""
from __future__ import annotations

from ctypes import c_float, c_int, c_longlong, c_void_p

import torch

from .. import envs
from . import count_launch
from . import cuda as _c


def _call(p, row, q, kv_cache, ring, meta, R, ring_from, single, only_ring):
    assert row.stride(1) == 1 and ring.is_contiguous() and ring.dtype == p.conv_w.dtype == row.dtype
    nb, bs = (kv_cache.shape[0], kv_cache.shape[3]) if kv_cache is not None else (0, 16)
    inv = p.inv_freq
    _c._check(_c.lib().b200_conv_cache(
        _c._p(row), c_int(row.stride(0)), *(c_int(o) for o in p.offsets), _c._p(p.conv_w), c_int(p.taps), _c._p(ring),
        _c._p(inv), c_int(inv.numel() if inv is not None else 0), c_float(p.rot_mult), _c._p(p.q_scale), _c._p(q),
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


def _finish_args(gate, lam, vdim, diff, eps):
    return (_c._p(lam), _c._p(gate), c_int(gate.stride(0) if gate is not None else 0), c_int(vdim), c_float(1.0 - diff),
            c_float(eps))


def paged_attention_heads(q, kv_cache, meta, scale, window, vdim, gate=None, lam=None, diff=0.0, eps=0.0):
    """See ``ops.paged_attention_heads``.  bf16 heads of 64 or 128: decoded tokens, and prompts where the tcgen05 kernel
    runs, leave the attention kernel finished; other prompts and 32-bit caches are finished by ``combine_heads``."""
    T, Hq, D = q.shape
    nb, _, Hkv, bs, _ = kv_cache.shape
    G, R, nd = Hq // Hkv, meta.num_reqs, meta.num_decode_reqs
    if q.dtype != torch.bfloat16 or D not in (64, 128):
        return combine_heads(_c.paged_attention(q, kv_cache, meta, scale, sliding_window=window), vdim, gate, lam, diff, eps)
    assert gate is None or (gate.stride(1) == 1 and gate.dtype == q.dtype)
    ws, heads = _c.Workspace.get(q.device), Hq // 2 if lam is not None else Hq
    if G > 16:
        nd = 0
    tc = D == 128 and G in (1, 2, 4, 8) and envs.B200_ATTN_PREFILL_IMPL == "tc"
    if nd < R and not tc:
        # the whole batch through the unfinished kernels: two launches of attention at most, one behind them
        return combine_heads(_c.paged_attention(q, kv_cache, meta, scale, sliding_window=window), vdim, gate, lam, diff, eps)
    out = ws.attn_out(T, heads, D)
    pages = (_c._p(meta.block_tables), _c._p(meta.seq_lens), _c._p(meta.query_start_loc))
    sizes = (c_int(meta.block_tables.shape[1]), c_int(bs), c_longlong(nb), c_int(Hq), c_int(Hkv), c_int(D), c_float(scale),
             c_int(int(window or 0)))
    fin = _finish_args(gate, lam, vdim, diff, eps)
    L = _c.lib()
    if nd:
        n = meta.padded_num_reqs if nd == R and meta.padded_num_reqs is not None else nd
        splits = _c.decode_splits(n, Hkv)
        need = L.b200_attn_decode_scratch_bytes(c_int(n), c_int(Hkv), c_int(splits), c_int(D))
        if need > ws.attn_scratch.numel() or n * Hkv > ws.attn_counters.numel():
            splits = 1
        _c._check(L.b200_attn_decode_heads(_c._p(q), _c._p(kv_cache), _c._p(out), *pages, c_int(0), c_int(n), *sizes,
                                           c_int(splits), _c._p(ws.attn_scratch), _c._p(ws.attn_counters), *fin,
                                           _c._stream()), "attn_decode_heads")
        count_launch()
    if nd < R:
        qsl = meta.query_start_loc_cpu
        tiles = int(((qsl[nd + 1:R + 1] - qsl[nd:R] + 63) // 64).sum()) if qsl is not None else (T + 63) // 64 + (R - nd)
        _c._check(L.b200_attn_prefill_tc_heads(
            _c._p(q), _c._p(kv_cache), _c._p(out), *pages, c_int(nd), c_int(R), c_int(tiles), c_int(T), *sizes, *fin,
            _c._p(ws.status), _c._stream()), "attn_prefill_tc_heads")
        count_launch()
    return out


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
