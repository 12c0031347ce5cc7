"""Linear attention with a state that is carried from token to token: what a layer asks for (``LinearAttentionPlan``)
and the plain-PyTorch statement (oracle of ``csrc/linear_attention.cu`` and the CPU path).

Per head, with S the [dim, vdim] state (fp32), q and k prepared as the plan says and one of two rules:

    fixed decay per head:            S <- decay_h S + k v^T
    delta rule, decay per channel:   S <- g S (rows);  u = beta (v - S^T k);  S <- S + k u^T

    o = S^T q;   y = o / rms(o) [* norm] * act(gate)

q, k, v come from columns of one packed projection ``row`` [T, >= ...]; preparation is, in this order: the causal
short convolution with silu over all q, k, v channels (``taps`` > 0), rotation of the first dimensions in half-split
pairs (``inv_freq``), unit length (``unit_norm``), multipliers.

State pools are indexed by the request's slot (``meta.state_slots``): ``state`` [slots, heads, dim, vdim] fp32 and, with
convolutions, ``ring`` [slots, taps, channels]: the input of position p in row p % taps, so that the row a decoded
token writes is none of those it reads.  A request whose first token of the step has position 0 starts from zeros;
nothing has to be cleared.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch
import torch.nn.functional as F

from .short_conv import conv_with_ring

UNIT_EPS = 1e-6


@dataclass
class LinearAttentionPlan:
    heads: int
    k_heads: int                         # q / k heads; each serves heads / k_heads value heads
    dim: int
    vdim: int
    offsets: tuple                       # first columns of q, k, v in the row
    gate_act: str                        # silu | sigmoid
    eps: float
    q_mult: float = 1.0
    k_mult: float = 1.0
    unit_norm: bool = False
    norm_w: Optional[torch.Tensor] = None       # [vdim] fp32
    inv_freq: Optional[torch.Tensor] = None     # [rotated pairs] fp32
    decay: Optional[torch.Tensor] = None        # [heads] fp32: fixed decay; None: delta rule
    taps: int = 0
    conv_w: Optional[torch.Tensor] = None       # [channels, taps] in the model dtype, channels = q | k | v
    beta_offset: int = 0                 # delta rule: first column of the step sizes (before the sigmoid) in the row
    A_log: Optional[torch.Tensor] = None        # [heads] fp32
    dt_bias: Optional[torch.Tensor] = None      # [heads * dim] fp32

    @property
    def delta(self) -> bool:
        return self.decay is None

    @property
    def channels(self) -> int:
        return 2 * self.k_heads * self.dim + self.heads * self.vdim

    def state_shape(self, slots: int) -> tuple:
        return (slots, self.heads, self.dim, self.vdim)

    def ring_shape(self, slots: int) -> tuple:
        return (slots, self.taps, self.channels)


def split_qkv(plan: LinearAttentionPlan, row: torch.Tensor) -> torch.Tensor:
    """The q | k | v columns of the packed row, [T, channels]."""
    n = plan.k_heads * plan.dim
    q, k, v = plan.offsets
    return torch.cat([row[:, q:q + n], row[:, k:k + n], row[:, v:v + plan.heads * plan.vdim]], -1)


def rotate_half_split(x: torch.Tensor, positions: torch.Tensor, inv_freq: torch.Tensor) -> torch.Tensor:
    """x [T, H, d] fp32: dimension i < P turns with dimension i + P (P pairs); the rest pass."""
    P = inv_freq.numel()
    a = positions.float()[:, None] * inv_freq[None]
    c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
    u, v = x[..., :P], x[..., P:2 * P]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * P:]], -1)


def linear_attention_reference(plan: LinearAttentionPlan, row, decay_in, gate, meta, cache):
    T, H, G, d, dv = row.shape[0], plan.heads, plan.k_heads, plan.dim, plan.vdim
    y = torch.zeros(T, H * dv, dtype=row.dtype, device=row.device)
    ring, state = cache if plan.taps else (None, cache[0])
    qsl, sl, slots = meta.query_start_loc.tolist(), meta.seq_lens.tolist(), meta.state_slots.tolist()
    for r in range(meta.num_reqs):
        a, b = qsl[r], qsl[r + 1]
        if b <= a or slots[r] < 0:
            continue
        start, S = sl[r] - (b - a), state[slots[r]]
        x = split_qkv(plan, row[a:b])
        x = F.silu(conv_with_ring(x, plan.conv_w, ring[slots[r]], start)) if plan.taps else x.float()
        q, k, v = x.split([G * d, G * d, H * dv], -1)
        q, k, v = q.reshape(-1, G, d), k.reshape(-1, G, d), v.reshape(-1, H, dv)
        if plan.inv_freq is not None:
            pos = torch.arange(start, start + b - a, device=row.device)
            q, k = (rotate_half_split(t, pos, plan.inv_freq) for t in (q, k))
        if plan.unit_norm:
            q, k = (t * torch.rsqrt(t.pow(2).sum(-1, keepdim=True) + UNIT_EPS) for t in (q, k))
        q = (q * plan.q_mult).repeat_interleave(H // G, 1)
        k = (k * plan.k_mult).repeat_interleave(H // G, 1)
        if start == 0:
            S.zero_()
        if plan.delta:
            z = F.softplus(decay_in[a:b].float() + plan.dt_bias).reshape(-1, H, d)
            g = torch.exp(-torch.exp(plan.A_log)[None, :, None] * z)
            beta = torch.sigmoid(row[a:b, plan.beta_offset:plan.beta_offset + H].float())
        o = torch.empty(b - a, H, dv, device=row.device)
        for t in range(b - a):
            if plan.delta:
                S.mul_(g[t][:, :, None])
                u = (v[t] - torch.einsum("hkv,hk->hv", S, k[t])) * beta[t][:, None]
            else:
                S.mul_(plan.decay[:, None, None])
                u = v[t]
            S.add_(k[t][:, :, None] * u[:, None, :])
            o[t] = torch.einsum("hkv,hk->hv", S, q[t])
        o = o * torch.rsqrt(o.pow(2).mean(-1, keepdim=True) + plan.eps)
        if plan.norm_w is not None:
            o = o * plan.norm_w
        gt = gate[a:b].float().reshape(-1, H, dv)
        o = o * (F.silu(gt) if plan.gate_act == "silu" else torch.sigmoid(gt))
        y[a:b] = o.reshape(-1, H * dv).to(y.dtype)
    return y
