"""Latent attention whose sizes, rotation, scale and cache are set per layer (``config.LatentMixerSpec``).

Beside DeepSeek's MLA layer it has a query latent of its own rank, a gate on the concatenated heads, YaRN
applied to the rotated parts only (cos and sin carry the multiplier, the score scale is the configured one), and
``kv_from``: a layer may read the latent and the rotated key that an earlier layer has cached and then owns no
latent projection.

A step of one layer, absorbed form for prompts and decoding alike:

    row  = [W_dq ‖ W_dkv ‖ W_g] x                 one packed GEMM (no W_dkv when the cache is shared)
    c_q  = rms(row_q); cache <- rms(row_c) ‖ rope(row_k)                       one launch (``latent_prep``)
    q    = W_uq c_q;  ql = W_uk^T q_nope (per head)  ‖  rope(q_rot)
    o    = softmax(ql . cache * scale) cache_c                                 paged latent attention
    y    = W_o ( (W_uv o per head) * sigmoid(row_g) )                          gate in the head GEMM's epilogue

A cache row is latent ‖ rotated key, zero-padded to a multiple of 16.  Query heads (W_uq, W_uk, W_uv, W_g, W_o)
are sharded over TP; the latents and the cache are replicated.
"""
from __future__ import annotations

import torch

from .. import ops
from ..config import LatentMixerSpec, ModelConfig
from ..parallel.state import get_state
from .linear import ColumnParallelLinear, RowParallelLinear, seeded_normal


def cache_row_width(spec: LatentMixerSpec) -> int:
    """Elements of a cached row: the attention kernel contracts in steps of 16."""
    return (spec.kv_rank + spec.rot_dim + 15) // 16 * 16


class LatentInputLinear(ColumnParallelLinear):
    """Query latent (replicated), cached latent and shared key (replicated, absent when shared), gate (by heads)."""

    def __init__(self, name, hidden, spec: LatentMixerSpec, **kw):
        self.latent_rows = spec.q_rank + (spec.kv_rank + spec.rot_dim if spec.kv_from is None else 0)
        gate = spec.heads * spec.vdim if spec.output_gate else 0
        super().__init__(name, hidden, [self.latent_rows, gate], **kw)
        self.shard_sizes = [self.latent_rows, gate // self.tp_size]
        self.out_features = sum(self.shard_sizes)

    def shard_of(self, full_weight):
        g = self.shard_sizes[1]
        lo = self.latent_rows + self.tp_rank * g
        return torch.cat([full_weight[:self.latent_rows], full_weight[lo:lo + g]], 0)


class LatentAttention:
    def __init__(self, name: str, spec: LatentMixerSpec, cfg: ModelConfig, device, quant=None):
        st = get_state()
        if spec.heads % st.tp.size:
            raise ValueError(f"{name}: {spec.heads} heads do not divide over tp={st.tp.size}")
        self.name, self.spec, self.cfg, self.device = name, spec, cfg, device
        self.H = spec.heads // st.tp.size
        self.eps = cfg.rms_norm_eps
        kw = dict(dtype=cfg.dtype, device=device, quant_config=quant)
        self.inp = LatentInputLinear(f"{name}.in_proj", cfg.hidden_size, spec, **kw)
        self.uq = ColumnParallelLinear(f"{name}.uq_proj", spec.q_rank, spec.heads * (spec.dim + spec.rot_dim), **kw)
        self.o = RowParallelLinear(f"{name}.o_proj", spec.heads * spec.vdim, cfg.hidden_size, **kw)
        self.dq_norm = torch.ones(spec.q_rank, dtype=cfg.dtype, device=device)
        self.dkv_norm = None
        if spec.kv_from is None:
            self.dkv_norm = torch.ones(spec.kv_rank, dtype=cfg.dtype, device=device)
        self.w_uk = None            # [H, kv_rank, dim]   (K-major for the head GEMM)
        self.w_uv = None            # [H, vdim, kv_rank]
        scaling = spec.rot.rope_scaling
        self.inv_freq = ops.ref.rope_inv_freq(spec.rot.dims, spec.rot.base, scaling).to(device)
        self.rope_mult = ops.ref.rope_attention_factor(scaling)
        self.row_width = cache_row_width(spec)

    def linears(self):
        return [self.inp, self.uq, self.o]

    def load_uk(self, full: torch.Tensor) -> None:
        """Key expansion [heads * dim, kv_rank] -> this rank's heads, transposed per head."""
        s, lo = self.spec, get_state().tp.rank_in_group * self.H
        w = full.view(s.heads, s.dim, s.kv_rank)[lo:lo + self.H]
        self.w_uk = w.transpose(1, 2).to(device=self.device, dtype=self.cfg.dtype).contiguous()

    def load_uv(self, full: torch.Tensor) -> None:
        s, lo = self.spec, get_state().tp.rank_in_group * self.H
        w = full.view(s.heads, s.vdim, s.kv_rank)[lo:lo + self.H]
        self.w_uv = w.to(device=self.device, dtype=self.cfg.dtype).contiguous()

    def init_dummy(self, std: float, seed: int) -> None:
        for lin in self.linears():
            lin.init_dummy(std, seed)
        s = self.spec
        for leaf, rows, load in (("uk_proj", s.heads * s.dim, self.load_uk), ("uv_proj", s.heads * s.vdim, self.load_uv)):
            load(seeded_normal(f"{self.name}.{leaf}", (rows, s.kv_rank), std, self.cfg.dtype, self.device, seed))

    def weight_bytes(self) -> int:
        return sum(l.weight_bytes() for l in self.linears()) + sum(t.numel() * t.element_size()
                                                                   for t in (self.w_uk, self.w_uv))

    def forward(self, x, cache, meta):
        """x [T, hidden] in the model's dtype; ``cache`` [blocks, block_size, row_width] is this layer's or, for a
        layer that shares one, the cache the owner has already written this step."""
        s, T = self.spec, x.shape[0]
        row = self.inp(x)
        cq = ops.latent_prep(row, self.dq_norm, self.dkv_norm, cache, meta.slot_mapping, meta.positions, self.inv_freq,
                             self.rope_mult, self.eps, s.kv_rank, s.rot_dim)
        q = self.uq(cq).view(T, self.H, s.dim + s.rot_dim)
        ql = torch.empty((T, self.H, self.row_width), dtype=x.dtype, device=x.device)
        ops.gemm_heads(q, self.w_uk, out=ql)
        ops.rope_heads_into(q, ql, s.dim, s.rot_dim, s.kv_rank, meta.positions, self.inv_freq, self.rope_mult)
        o = ops.mla_paged_attention(ql, cache, meta, s.scale, s.kv_rank)
        gate = row[:, self.inp.latent_rows:] if s.output_gate else None
        return self.o(ops.gemm_heads(o, self.w_uv, gate=gate).view(T, self.H * s.vdim))
