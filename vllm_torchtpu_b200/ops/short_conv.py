"""Short causal convolutions over projected channels, with the inputs of earlier steps in a ring per request, and what
stands behind them in attention layers (``ConvAttentionPlan``): plain-PyTorch statement (oracle of
``csrc/conv_cache.cu`` and the CPU path).

    y_t = sum_j w[:, j] u_(t - taps + 1 + j)           per channel, zeros in front of the sequence

``ring`` [slots, taps, channels] holds the input of position p in row p % taps, so that the row a decoded token writes is
none of those it reads; a portion that starts at position 0 reads none of it, so nothing has to be cleared.

Attention layers: q, k and v channels of one packed projection ``row`` pass the convolution, then q and k turn (the first
``2 * pairs`` dimensions of a head, interleaved pairs, cos and sin times ``rot_mult``), q is multiplied by one number per
head where the plan has them, k and v go to the token's page.
Heads are stored in ``width`` columns, zeros behind them.  With two maps per head, a key row is both maps side by side,
and the query of a head becomes two rows, each with its map's columns and zeros in the other's place: scores against the
whole key row are then the scores of that map, and the values are shared.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch
import torch.nn.functional as F


def conv_with_ring(x, w, ring, start: int):
    """x [L, C] of one request from position ``start`` on, w [C, taps]; ring [taps, C] is read and updated.  fp32."""
    K = w.shape[1]
    hist = [ring[p % K] if p >= 0 else torch.zeros_like(x[0]) for p in range(start - K + 1, start)]
    full = torch.cat([torch.stack(hist), x], 0) if hist else x
    out = sum(full[j:j + x.shape[0]].float() * w[:, j].float() for j in range(K))
    advance_ring(x, ring, start)
    return out


def advance_ring(x, ring, start: int) -> None:
    K = ring.shape[0]
    for p in range(max(start, start + x.shape[0] - K), start + x.shape[0]):
        ring[p % K] = x[p - start]


@dataclass
class ConvAttentionPlan:
    heads: int
    kv_heads: int                        # 0: the layer reads another layer's keys and values
    dim: int                             # of one map
    vdim: int
    maps: int
    width: int                           # columns of a stored head
    offsets: tuple                       # first columns of q, k, v in the row
    taps: int
    conv_w: Optional[torch.Tensor] = None       # [taps, channels] in the model dtype, channels = q | k | v
    inv_freq: Optional[torch.Tensor] = None     # [pairs] fp32, None: no rotation
    rot_mult: float = 1.0
    q_scale: Optional[torch.Tensor] = None      # [heads] fp32, None: 1

    @property
    def sizes(self) -> tuple:
        """Channels of q, k, v."""
        return self.heads * self.maps * self.dim, self.kv_heads * self.maps * self.dim, self.kv_heads * self.vdim

    @property
    def channels(self) -> int:
        return sum(self.sizes)

    def ring_shape(self, slots: int) -> tuple:
        return (slots, self.taps, self.channels)

    def split(self, row: torch.Tensor) -> torch.Tensor:
        """The q | k | v columns of the packed row, [T, channels]."""
        return torch.cat([row[:, o:o + n] for o, n in zip(self.offsets, self.sizes) if n], -1)


def portions_of(meta):
    """(first row, end row, position of the first, slot) of every request with rows and a slot."""
    qsl, sl, slots = meta.query_start_loc.tolist(), meta.seq_lens.tolist(), meta.state_slots.tolist()
    for r in range(meta.num_reqs):
        a, b = qsl[r], qsl[r + 1]
        if b > a:
            yield a, b, sl[r] - (b - a), slots[r]


def conv_and_cache(plan: ConvAttentionPlan, row, kv_cache, ring, meta):
    """Returns q [T, heads * maps, width]; writes the pages of ``meta.slot_mapping`` (unless the layer shares) and the
    rings of ``meta.state_slots``."""
    from .reference import rope_scaled, write_kv_cache
    p, T = plan, row.shape[0]
    x, y = plan.split(row), torch.zeros(T, plan.channels, device=row.device)
    for a, b, start, slot in portions_of(meta):
        mine = ring[slot] if slot >= 0 else torch.zeros_like(ring[0])
        y[a:b] = conv_with_ring(x[a:b], p.conv_w.t(), mine, start)
    q, k, v = y.split(p.sizes, -1)
    q, k = q.reshape(T, p.heads * p.maps, p.dim), k.reshape(T, p.kv_heads * p.maps, p.dim)
    if p.inv_freq is not None:
        q, k = (rope_scaled(t, meta.positions, p.inv_freq, p.rot_mult, True) for t in (q, k))
    if p.q_scale is not None:
        q = q.reshape(T, p.heads, -1) * p.q_scale[:, None]
    wide = torch.zeros(T, p.heads, p.maps, p.width, device=row.device)
    for m in range(p.maps):
        wide[:, :, m, m * p.dim:(m + 1) * p.dim] = q.reshape(T, p.heads, p.maps, p.dim)[:, :, m]
    if p.kv_heads:
        pad = lambda t: F.pad(t, (0, p.width - t.shape[-1])).to(row.dtype)              # noqa: E731
        write_kv_cache(kv_cache, pad(k.reshape(T, p.kv_heads, -1)), pad(v.reshape(T, p.kv_heads, -1)), meta.slot_mapping)
    return wide.reshape(T, p.heads * p.maps, p.width).to(row.dtype)


def ring_update(plan: ConvAttentionPlan, row, ring, meta) -> None:
    """Only the rings advance over the rows (replay of accepted rows after rejected drafts)."""
    x = plan.split(row)
    for a, b, start, slot in portions_of(meta):
        if slot >= 0:
            advance_ring(x[a:b], ring[slot], start)


def combine_heads(a, vdim: int, gate=None, lam=None, diff: float = 0.0, eps: float = 0.0):
    """What follows the softmax of such a layer.  ``lam`` [1]: rows 2h and 2h + 1 of a [T, 2 H, width] are the maps of
    head h, o = a1 - lam * a2, o / rms(o) * (1 - diff); ``gate`` [T, H * vdim]: times its sigmoid.  [T, H, width], the
    columns behind ``vdim`` as they are (zeros)."""
    T, width = a.shape[0], a.shape[2]
    o = a.float()
    if lam is not None:
        o = o.reshape(T, -1, 2, width)
        o = o[:, :, 0] - lam.float() * o[:, :, 1]
        o = o * torch.rsqrt(o[..., :vdim].pow(2).mean(-1, keepdim=True) + eps) * (1.0 - diff)
    if gate is not None:
        o = torch.cat([o[..., :vdim] * torch.sigmoid(gate.float().reshape(T, -1, vdim)), o[..., vdim:]], -1)
    return o.to(a.dtype)
