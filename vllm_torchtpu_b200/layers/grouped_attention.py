"""Grouped-query attention whose sizes are set per layer (``config.GroupedMixerSpec``).

Beside ``layers/attention.py`` it has its own value size, RMS norms over the whole q and k projections (not per head),
no rotation, a query temperature that grows with the position and a sink logit per head:

    row  = [W_q ‖ W_k ‖ W_v] x                                       one packed GEMM
    q, cache <- rms(row_q) * temperature(p);  rms(row_k), row_v       one launch (``norm_and_cache``)
    o    = softmax with sinks (q . k * scale) v                       the paged attention of the other models
    y    = W_o o

Heads are padded with zeros to a size the attention kernels are built for (``cache_head_dim``); the columns of W_o
carry the same padding.  Query heads are sharded over TP; the norms' squared sums are then added up over the ranks.
"""
from __future__ import annotations

import torch
import torch.nn.functional as F

from .. import ops
from ..config import ModelConfig
from ..layer_specs import GroupedMixerSpec
from ..parallel.communicator import get_tp_comm
from ..parallel.state import get_state
from .linear import RowParallelLinear, seeded_normal
from .packed import PackedLinear, Part


def cache_head_dim(dim: int, vdim: int, dtype: torch.dtype) -> int:
    """Head size of the cache: 64 or 128 for the bf16 tensor-core kernels, otherwise the next multiple of 4."""
    d = max(dim, vdim)
    if dtype == torch.bfloat16 and d <= 128:
        return 64 if d <= 64 else 128
    return (d + 3) // 4 * 4


class HeadPaddedRowLinear(RowParallelLinear):
    """Output projection whose input heads are padded from ``size`` to ``padded`` elements."""

    def __init__(self, name, heads: int, size: int, padded: int, out_features: int, **kw):
        self.heads, self.size, self.padded = heads, size, padded
        super().__init__(name, heads * padded, out_features, **kw)
        self.full_in = heads * size

    def shard_of(self, full_weight):
        w = full_weight.reshape(full_weight.shape[0], self.heads, self.size)
        return super().shard_of(F.pad(w, (0, self.padded - self.size)).reshape(full_weight.shape[0], -1))


class GroupedAttention:
    def __init__(self, name: str, spec: GroupedMixerSpec, cfg: ModelConfig, device, quant=None, more=(), output=True):
        """``more``: parts of other mixers that the packed projection of the input computes too; without ``output`` the
        owner applies the output projection."""
        st = get_state()
        tp = st.tp.size
        if spec.heads % tp:
            raise ValueError(f"{name}: {spec.heads} heads do not divide over tp={tp}")
        self.name, self.spec, self.cfg, self.device = name, spec, cfg, device
        self.Hq, self.Hkv = spec.heads // tp, max(1, spec.kv_heads // tp)
        self.D = cache_head_dim(spec.maps * spec.dim, spec.vdim, cfg.dtype)
        self.eps = cfg.rms_norm_eps
        kw = dict(dtype=cfg.dtype, device=device, quant_config=quant)
        self.inp = PackedLinear(f"{name}.qkv_proj", cfg.hidden_size, self.parts(spec) + list(more), bias=spec.bias,
                                **kw)
        self.o = HeadPaddedRowLinear(f"{name}.o_proj", spec.heads, spec.vdim, self.D, cfg.hidden_size,
                                     bias=spec.out_bias, **kw) if output else None
        ones = lambda n: torch.ones(n, dtype=cfg.dtype, device=device)                  # noqa: E731
        self.q_norm = ones(self.Hq * spec.dim) if spec.projection_norm else None
        self.k_norm = ones(self.Hkv * spec.dim) if spec.projection_norm else None
        self.sinks = torch.zeros(self.Hq, dtype=torch.float32, device=device) if spec.sinks or spec.zero_sink \
            else None
        self.kv_replicas = max(1, tp // spec.kv_heads)
        # sharded norms: the squared sums of all ranks, each replicated key head counted once
        self.norm_sizes = (spec.heads * spec.dim, spec.kv_heads * spec.dim)

    @staticmethod
    def parts(spec: GroupedMixerSpec) -> list:
        """Projections of the layer's input, packed into one GEMM."""
        qk, parts = spec.maps * spec.dim, [Part("q", spec.heads * spec.maps * spec.dim, spec.heads)]
        if spec.kv_from is None:
            parts += [Part("k", spec.kv_heads * qk, spec.kv_heads), Part("v", spec.kv_heads * spec.vdim, spec.kv_heads)]
        return parts + ([Part("g", spec.heads * spec.vdim, spec.heads)] if spec.output_gate else [])

    def linears(self):
        return [self.inp] + ([self.o] if self.o is not None else [])

    def init_dummy(self, std: float, seed: int) -> None:
        for lin in self.linears():
            lin.init_dummy(std, seed)
        if self.spec.sinks:
            self.load_sinks(seeded_normal(f"{self.name}.sinks", (self.spec.heads,), 1.0, torch.float32, self.device, seed))

    def load_sinks(self, full) -> None:
        r = get_state().tp.rank_in_group
        self.sinks.copy_(full[r * self.Hq:(r + 1) * self.Hq])

    def load_norm(self, which: str, full) -> None:
        """Weights over the full projection -> those of this rank's heads."""
        t, r = (self.q_norm, self.k_norm)[which == "k"], get_state().tp.rank_in_group
        i = r // self.kv_replicas if which == "k" else r
        t.copy_(full[i * t.numel():(i + 1) * t.numel()])

    def weight_bytes(self) -> int:
        return sum(l.weight_bytes() for l in self.linears())

    # ---- cache -----------------------------------------------------------------
    def cache_shape(self, num_blocks: int, block_size: int) -> tuple:
        return (num_blocks, 2, self.Hkv, block_size, self.D)

    def allocate_cache(self, num_blocks: int, block_size: int, kv_dtype, device, slots: int):
        if kv_dtype != self.cfg.dtype:
            raise ValueError(f"{self.name}: a {kv_dtype} KV cache is not built for this attention")
        return torch.zeros(self.cache_shape(num_blocks, block_size), dtype=kv_dtype, device=device)

    def bytes_per_block(self, block_size: int, elem: int) -> int:
        return 2 * self.Hkv * block_size * self.D * elem

    def _split_sums(self, row):
        """Squared sums of q and k over all ranks ([T], [T]); None, None on one rank."""
        comm = get_tp_comm()
        if self.q_norm is None or comm.size == 1:
            return None, None
        nq, nk = self.q_norm.numel(), self.k_norm.numel()
        k0 = self.inp.offset["k"]
        q, k = row[:, :nq].float(), row[:, k0:k0 + nk].float()
        s = comm.all_reduce(torch.stack([q.pow(2).sum(-1), k.pow(2).sum(-1) / self.kv_replicas], 1))
        return s[:, 0].contiguous(), s[:, 1].contiguous()

    def forward(self, x, cache, meta):
        s, T = self.spec, x.shape[0]
        row = self.inp(x)
        ssq, ssk = self._split_sums(row)
        t = (s.q_temp.coef, s.q_temp.every) if s.q_temp else None
        q = ops.norm_and_cache(row, meta.positions, cache, meta.slot_mapping, self.Hq, self.Hkv, s.dim, s.vdim,
                               self.q_norm, self.k_norm, self.eps, t, ssq, ssk, self.norm_sizes,
                               (self.inp.offset["k"], self.inp.offset["v"]))
        o = ops.paged_attention(q, cache, meta, s.scale, sinks=self.sinks)
        return self.o(o.reshape(T, self.Hq * self.D))
