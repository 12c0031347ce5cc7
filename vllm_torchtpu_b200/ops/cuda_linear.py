"""Bindings of the carried-state linear-attention kernels (``csrc/linear_attention.cu``)."""
from __future__ import annotations

from ctypes import c_float, c_int, c_void_p

import torch

from . import count_launch
from . import cuda as _c
from .linear_attention import RULES

STEP, CHUNKS, RING, SCAN, FINISH = 0, 1, 2, 3, 4
CHUNK = 16
SCRATCH_BYTES = 64 << 20                 # of one slab of chunks: two of them about fill the L2
_side: dict = {}                         # device index -> stream of the scans


def slabs(lens, heads: int, chunk_bytes: int, budget: int = SCRATCH_BYTES) -> list:
    """Launches that cover prompts of ``lens`` tokens: [(first request, end request, first chunk, chunks)], each with
    (requests * chunks * heads) units of scratch within the budget (at least one chunk of one request)."""
    out, i = [], 0
    need = [-(-n // CHUNK) for n in lens]
    per = max(1, budget // (heads * chunk_bytes))             # chunks that fit over all heads
    while i < len(need):
        j, most = i + 1, need[i]
        while j < len(need) and (j - i + 1) * min(max(most, need[j]), 8) <= per:
            most = max(most, need[j])
            j += 1
        n = max(1, min(most, per // (j - i)))
        out += [(i, j, c, min(n, most - c)) for c in range(0, most, n)]
        i = j
    return out


def _side_stream(device):
    i = torch.device(device).index or 0
    if i not in _side:
        _side[i] = torch.cuda.Stream(device)
    return _side[i]


def carried_state_attention(plan, row, decay_in, gate, meta, cache, out=None):
    """See ``ops.linear_attention``: rows [T, ...] of the packed projection -> y [T, heads * vdim] (``out``, whose rows may
    be strided; rows that belong to no request are left as they are in a step with prompts)."""
    elem = _c._mixed(row)
    p = plan
    T = row.shape[0]
    for t in (row, gate, decay_in):
        assert t is None or (t.stride(1) == 1 and t.dtype == row.dtype)
    ring, state = cache if p.taps else (None, cache[0])
    R, nd = meta.num_reqs, meta.num_decode_reqs
    decode_only = nd == R
    n_dec = (meta.padded_num_reqs if meta.padded_num_reqs is not None else R) if decode_only else nd
    lens = None
    if not decode_only:
        qsl = meta.query_start_loc_cpu if meta.query_start_loc_cpu is not None else meta.query_start_loc.cpu()
        lens = (qsl[nd + 1:R + 1] - qsl[nd:R]).tolist()
    whole = decode_only or int(qsl[R]) == T                   # every row belongs to a request
    y = out if out is not None else (torch.empty if whole else torch.zeros)((T, p.heads * p.vdim), dtype=row.dtype,
                                                                            device=row.device)
    assert y.stride(1) == 1 and y.dtype == row.dtype and y.shape[0] == T and y.shape[1] >= p.heads * p.vdim
    rule = RULES.index(p.rule)
    L = _c.lib()

    def call(mode, lo, hi, scratch=None, chunk=0, slab=0, stream=None):
        _c._check(L.b200_linear_attention(
            c_int(mode), c_int(rule), _c._p(row), c_int(row.stride(0)), *(c_int(o) for o in p.offsets),
            c_int(p.beta_offset), c_int(p.rate_offset), _c._p(decay_in), c_int(decay_in.stride(0) if decay_in is not None else 0), _c._p(gate),
            c_int(gate.stride(0)), _c._p(p.conv_w), _c._p(ring), c_int(p.taps), _c._p(p.inv_freq),
            c_int(p.inv_freq.numel() if p.inv_freq is not None else 0), _c._p(p.decay), _c._p(p.A_log),
            _c._p(p.dt_bias), _c._p(p.rate_bias), c_float(p.tau), _c._p(p.norm_w), c_int(p.norm_stride), _c._p(state),
            _c._p(y), c_int(y.stride(0)), _c._p(meta.query_start_loc), _c._p(meta.seq_lens), _c._p(meta.state_slots), c_int(lo), c_int(hi), c_int(T), c_int(p.heads),
            c_int(p.k_heads), c_int(p.dim), c_int(p.vdim), c_int(int(p.unit_norm)), c_int(int(p.gate_act == "silu")),
            c_float(p.eps), c_float(p.q_mult), c_float(p.k_mult), c_int(int(decode_only)), _c._p(scratch),
            c_int(chunk), c_int(slab), c_int(elem),
            _c._stream() if stream is None else c_void_p(stream.cuda_stream)), "linear_attention")
        count_launch()

    if n_dec:
        call(STEP, 0, n_dec)
    if lens:
        if elem == 2 and p.dim <= 256 and p.taps <= 8:
            per = int(L.b200_linear_attention_chunk_bytes(c_int(p.dim), c_int(p.vdim), c_int(rule)))
            parts = slabs(lens, p.heads, per)
            room = max((j - i) * n for i, j, _, n in parts) * p.heads * per
            scratch = torch.empty((min(2, len(parts)), room), dtype=torch.uint8, device=row.device)
            main = torch.cuda.current_stream()
            side = main if len(parts) == 1 else _side_stream(row.device)
            last = None                   # slab whose scan is on its way: (arguments, event)
            for x, (i, j, c, n) in enumerate(parts):
                args = (nd + i, nd + j, scratch[x & 1], c, n)
                call(CHUNKS, *args)
                if side is not main:
                    side.wait_event(main.record_event())
                call(SCAN, *args, side)   # a chain over the chunks with few CTAs: beside the next slab's products
                if last is not None:
                    main.wait_event(last[1])
                    call(FINISH, *last[0])
                last = (args, side.record_event() if side is not main else None)
            if last[1] is not None:
                main.wait_event(last[1])
            call(FINISH, *last[0])
        else:
            call(STEP, nd, R)
        if p.taps:
            # portions of one token that open a sequence enter here too when they ran as a chunk
            call(RING, nd, R)
    return y
