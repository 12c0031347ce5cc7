"""Grouped-query attention behind short convolutions (``layer_specs.GroupedMixerSpec`` with ``conv``): a sliding window,
optionally rotated q and k with an output gate, or two softmax maps per head (differential attention); or chunks of the
sequence instead of the window, a factor on the scores of every head and a sink of 0.

    row  = [W_q ‖ W_k ‖ W_v ‖ W_g] x + b                              one packed GEMM
    q, cache <- conv(row_q), conv(row_k), conv(row_v), rotated        one launch (``conv_and_cache``)
    o    = softmax over the window (q . k * scale) v                  the paged attention of the other models
    y    = W_o (sigmoid(row_g) o) + b_o

    two maps:   lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + diff,   o = o1 - lambda o2,   o / rms(o) * (1 - diff)

Differential heads need no attention kernel of their own: a cached key row is both maps side by side, and the query of a
head is two query heads of the same group with zeros in the other map's columns (``ops.short_conv``), so that a page's keys
and values are read once for both maps and all heads of the group.  A layer with ``kv_from`` has no keys and values of its
own and reads the pages of the layer it names.

A cache is (ring, pages): the last projected values of every request, indexed by its batch slot, and the paged keys and
values.
"""
from __future__ import annotations

import torch

from .. import ops
from ..config import ModelConfig
from ..layer_specs import GroupedMixerSpec
from ..ops.short_conv import ConvAttentionPlan
from ..parallel.state import get_state
from .grouped_attention import GroupedAttention
from .linear import seeded_normal


class ConvAttention(GroupedAttention):
    def __init__(self, name: str, spec: GroupedMixerSpec, cfg: ModelConfig, device, quant=None, more=(), output=True):
        super().__init__(name, spec, cfg, device, quant, more, output)
        s, at = spec, self.inp.offset
        inv = ops.ref.rope_inv_freq(s.rot.dims, s.rot.base, s.rot.rope_scaling).to(device) if s.rot else None
        mult = ops.ref.rope_attention_factor(s.rot.rope_scaling) if s.rot else 1.0
        self.plan = ConvAttentionPlan(self.Hq, self.Hkv if s.kv_from is None else 0, s.dim, s.vdim, s.maps, self.D,
                                      (at["q"], at.get("k", 0), at.get("v", 0)), s.conv, inv_freq=inv, rot_mult=mult)
        if s.head_temp:
            self.plan.q_scale = torch.ones(self.Hq, dtype=torch.float32, device=device)
        self.lam = torch.zeros(1, dtype=torch.float32, device=device) if s.maps == 2 else None

    # ---- weights ---------------------------------------------------------------
    def _own(self, full, heads: int):
        """This rank's heads of a tensor with rows by heads (fewer heads than ranks are replicated)."""
        st = get_state().tp
        n = full.shape[0] // min(heads, st.size)
        i = st.rank_in_group // max(1, st.size // heads)
        return full[i * n:(i + 1) * n]

    def load_conv(self, q, k=None, v=None) -> None:
        s = self.spec
        parts = [self._own(q, s.heads)] + [self._own(t, s.kv_heads) for t in (k, v) if t is not None]
        self.plan.conv_w = torch.cat(parts, 0).t().to(device=self.device, dtype=self.cfg.dtype).contiguous()

    def load_bias(self, q, k=None, v=None) -> None:
        self.inp.load_bias(**{n: t for n, t in (("q", q), ("k", k), ("v", v)) if t is not None})

    def load_temp(self, full) -> None:
        """Factors on the scores of the heads; they go onto the queries, in 32-bit."""
        self.plan.q_scale.copy_(self._own(full, self.spec.heads))

    def load_out_bias(self, b) -> None:
        self.o.bias = b.to(device=self.device, dtype=self.cfg.dtype).contiguous()

    def load_lambda(self, lq1, lk1, lq2, lk2) -> None:
        a, b = ((x.double() * y.double()).sum() for x, y in ((lq1, lk1), (lq2, lk2)))
        self.lam.fill_(float(torch.exp(a) - torch.exp(b) + self.spec.diff))

    def init_dummy(self, std: float, seed: int) -> None:
        super().init_dummy(std, seed)
        s = self.spec

        def vec(leaf, *shape, scale=0.5):
            return seeded_normal(f"{self.name}.{leaf}", shape, scale, self.cfg.dtype, self.device, seed)
        own = {n: r for n, r in (("q", s.heads * s.maps * s.dim), ("k", s.kv_heads * s.maps * s.dim),
                                 ("v", s.kv_heads * s.vdim)) if n == "q" or s.kv_from is None}
        self.load_conv(**{n: vec(f"{n}_conv", r, s.conv) for n, r in own.items()})
        self.load_bias(**{n: vec(f"{n}_bias", r, scale=0.1) for n, r in own.items()})
        if s.head_temp:
            self.load_temp(1.0 + vec("temp", s.heads, scale=0.2))
        if s.out_bias:
            self.load_out_bias(vec("o_bias", self.cfg.hidden_size, scale=0.1))
        if s.maps == 2:
            self.load_lambda(*(vec(n, s.dim, scale=0.1) for n in ("lq1", "lk1", "lq2", "lk2")))

    # ---- cache -----------------------------------------------------------------
    def allocate_cache(self, num_blocks: int, block_size: int, kv_dtype, device, slots: int, shared=None):
        """``shared``: cache of the layer whose keys and values this one reads."""
        ring = torch.zeros(self.plan.ring_shape(slots), dtype=self.cfg.dtype, device=device)
        if self.spec.kv_from is not None:
            return ring, shared[1]
        return ring, super().allocate_cache(num_blocks, block_size, kv_dtype, device, slots)

    def bytes_per_block(self, block_size: int, elem: int) -> int:
        return super().bytes_per_block(block_size, elem) if self.spec.kv_from is None else 0

    # ---- forward ---------------------------------------------------------------
    def recur(self, inputs, meta, cache) -> None:
        """The stateful part beside the pages: the rings advance over the rows ``meta`` describes."""
        ops.conv_ring_update(self.plan, inputs[0], cache[0], meta)

    def forward(self, x, cache, meta):
        T, row = x.shape[0], self.inp(x)
        q = self.queries(row, cache, meta)
        return self.o(self.attend(q, row, cache[1], meta).reshape(T, self.Hq * self.D))

    def queries(self, row, cache, meta):
        """Convolved and rotated queries of the projected rows; keys and values go to their pages."""
        ring, pages = cache
        rb = getattr(meta, "state_rollback", None)
        if rb is not None:
            rb.capture(self, (ring,), (row,))      # verification step: rejected drafts are rolled back later
        return ops.conv_and_cache(self.plan, row, pages, ring, meta)

    def attend(self, q, row, pages, meta, out=None):
        """Softmax over the visible keys and what follows it: [T, heads, D], or the rows ``out``."""
        s, gate = self.spec, None
        if s.output_gate:
            at = self.inp.offset["g"]
            gate = row[:, at:at + self.Hq * s.vdim]
        if gate is None and s.maps == 1:
            return ops.paged_attention(q, pages, meta, s.scale, sliding_window=s.mask, sinks=self.sinks, out=out)
        return ops.paged_attention_heads(q, pages, meta, s.scale, s.mask, s.vdim, gate, self.lam, s.diff, self.eps)
