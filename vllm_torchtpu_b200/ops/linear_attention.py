"""Linear attention with a state that is carried from token to token: what a layer asks for (``LinearAttentionPlan``)
and the plain-PyTorch statement (oracle of ``csrc/linear_attention.cu`` and the CPU path).

Per head, with S the [dim, vdim] state (fp32), q and k prepared as the plan says and one of four rules:

    fixed     decay per head:      S <- decay_h S + k v^T
    channel   decay per channel:   S <- g S (rows) + k v^T
    delta     decay per channel:   S <- g S (rows);  u = beta (v - S^T k);  S <- S + k u^T
    removal   decay and rate per channel, both on the old state:  S <- g S - (a * n) (S^T n)^T + k v^T,  n = k / |k|

    o = S^T q;   y = o / rms(o) [* norm] * act(gate)

The decays per channel, from z = decay_in + dt_bias:

    delta     g = exp(-exp(A_log) softplus(z))
    channel   g = sigmoid(z)^(1 / tau)
    removal   g = exp(-exp(-1/2) sigmoid(z)),   a = sigmoid(row[rate_offset ..] + rate_bias)

q, k, v come from columns of one packed projection ``row`` [T, >= ...]; preparation is, in this order: the causal
short convolution with silu over all q, k, v channels (``taps`` > 0), rotation of the first dimensions in half-split
pairs (``inv_freq``), unit length (``unit_norm``), multipliers.

State pools are indexed by the request's slot (``meta.state_slots``): ``state`` [slots, heads, dim, vdim] fp32 and, with
convolutions, ``ring`` [slots, taps, channels]: the input of position p in row p % taps, so that the row a decoded
token writes is none of those it reads.  A request whose first token of the step has position 0 starts from zeros;
nothing has to be cleared.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Optional

import torch
import torch.nn.functional as F

from .short_conv import conv_with_ring

RULES = ("fixed", "delta", "channel", "removal")

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
    norm_w: Optional[torch.Tensor] = None       # [vdim], or [heads * vdim], fp32
    inv_freq: Optional[torch.Tensor] = None     # [rotated pairs] fp32
    decay: Optional[torch.Tensor] = None        # [heads] fp32: fixed decay; None: delta rule
    taps: int = 0
    conv_w: Optional[torch.Tensor] = None       # [channels, taps] in the model dtype, channels = q | k | v
    beta_offset: int = 0                 # delta rule: first column of the step sizes (before the sigmoid) in the row
    A_log: Optional[torch.Tensor] = None        # [heads] fp32
    dt_bias: Optional[torch.Tensor] = None      # [heads * dim] fp32
    rule: str = ""                       # one of RULES; not given: fixed with a decay, otherwise delta
    tau: float = 1.0
    rate_offset: int = 0                 # removal: first column of the rates (before bias and sigmoid) in the row
    rate_bias: Optional[torch.Tensor] = None    # [heads * dim] fp32

    def __post_init__(self):
        self.rule = self.rule or ("delta" if self.decay is None else "fixed")
        if self.rule not in RULES:
            raise ValueError(f"unknown rule {self.rule!r}; known: {RULES}")

    @property
    def norm_stride(self) -> int:
        """Elements between the norm weights of neighbouring heads."""
        return self.vdim if self.norm_w is not None and self.norm_w.numel() != self.vdim else 0

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


def channel_decay(plan: LinearAttentionPlan, decay_in: torch.Tensor) -> torch.Tensor:
    """Factors [T, heads, dim] of the rules that have one per channel."""
    z = (decay_in.float() + plan.dt_bias).reshape(-1, plan.heads, plan.dim)
    if plan.rule == "delta":
        return torch.exp(-torch.exp(plan.A_log)[None, :, None] * F.softplus(z))
    if plan.rule == "channel":
        return torch.exp(F.logsigmoid(z) / plan.tau)
    return torch.exp(-math.exp(-0.5) * torch.sigmoid(z))


def linear_attention_reference(plan: LinearAttentionPlan, row, decay_in, gate, meta, cache, out=None):
    T, H, G, d, dv = row.shape[0], plan.heads, plan.k_heads, plan.dim, plan.vdim
    y = torch.zeros(T, H * dv, dtype=row.dtype, device=row.device) if out is None else out.zero_()
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
        if plan.rule != "fixed":
            g = channel_decay(plan, decay_in[a:b])
        if plan.rule == "delta":
            beta = torch.sigmoid(row[a:b, plan.beta_offset:plan.beta_offset + H].float())
        if plan.rule == "removal":
            rate = row[a:b, plan.rate_offset:plan.rate_offset + H * d].float() + plan.rate_bias
            unit = k * torch.rsqrt(k.pow(2).sum(-1, keepdim=True) + UNIT_EPS)
            taken = torch.sigmoid(rate).reshape(-1, H, d) * unit
        o = torch.empty(b - a, H, dv, device=row.device)
        for t in range(b - a):
            u = v[t]
            if plan.rule == "removal":
                m = torch.einsum("hkv,hk->hv", S, unit[t])
            S.mul_(plan.decay[:, None, None] if plan.rule == "fixed" else g[t][:, :, None])
            if plan.rule == "delta":
                u = (v[t] - torch.einsum("hkv,hk->hv", S, k[t])) * beta[t][:, None]
            if plan.rule == "removal":
                S.sub_(taken[t][:, :, None] * m[:, None, :])
            S.add_(k[t][:, :, None] * u[:, None, :])
            o[t] = torch.einsum("hkv,hk->hv", S, q[t])
        o = o * torch.rsqrt(o.pow(2).mean(-1, keepdim=True) + plan.eps)
        if plan.norm_w is not None:
            o = o * (plan.norm_w.reshape(H, dv) if plan.norm_stride else plan.norm_w)
        gt = gate[a:b].float().reshape(-1, H, dv)
        o = o * (F.silu(gt) if plan.gate_act == "silu" else torch.sigmoid(gt))
        y[a:b] = o.reshape(-1, H * dv).to(y.dtype)
    return y
