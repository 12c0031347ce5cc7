"""Token shift: what a sublayer reads is moved towards what it would have read at the token before.

    r = residual (+ y),   h = r / rms(r) * (offset + w),   out_t = h_t + (h_(t-1) - h_t) * shift

with zeros in front of a sequence.  ``state`` [slots, width] fp32 holds the h of every request's last token (not rounded,
not shifted), indexed by its batch slot; a portion that starts at position 0 does not read it, so nothing has to be cleared.

Plain-PyTorch statement (oracle of ``csrc/token_shift.cu`` and the CPU path)."""
from __future__ import annotations

import torch

from .short_conv import portions_of


def shift_rows(h, shift, state, meta):
    """h [T, width] fp32 -> shifted rows; advances ``state``."""
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    for a, b, start, slot in portions_of(meta):
        before[a] = state[slot] if start > 0 and slot >= 0 else 0
    advance(h, state, meta)
    return h + (before - h) * shift.float()


def advance(h, state, meta) -> None:
    for a, b, start, slot in portions_of(meta):
        if slot >= 0:
            state[slot] = h[b - 1]


def add_rms_norm_shift(y, residual, weight, eps, offset, shift, state, meta, post=None, mult: float = 1.0,
                       keep: bool = False):
    """Arguments as in ``ops.add_rms_norm``.  Returns (shifted rows in the weight's dtype, r fp32, h fp32 or None); the
    residual is not updated in place."""
    from .reference import add_rms_norm
    h, r = add_rms_norm(y, residual, weight.float(), eps, offset, True, post, mult)
    return shift_rows(h, shift, state, meta).to(weight.dtype), r, (h if keep else None)
