"""Several projections of one input as one GEMM, with head-wise and replicated parts."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Sequence

import torch
import torch.nn.functional as F

from .linear import ColumnParallelLinear

ALIGN = 8                                # 16 bytes of bf16: parts start where a TMA map can


@dataclass
class Part:
    """``rows`` rows of the packed weight in ``units`` equal heads; 0 units: replicated over the TP ranks.  Fewer
    units than ranks: each unit lives on ranks / units of them."""
    name: str
    rows: int
    units: int = 0


class PackedLinear(ColumnParallelLinear):
    """Rows of the parts one after another, each padded with zero rows to a multiple of 8 on every rank, so that a
    part of the output can be the operand of another GEMM.  ``offset[name]``: first output column of a part."""

    def __init__(self, name, hidden, parts: Sequence[Part], **kw):
        self.parts = list(parts)
        super().__init__(name, hidden, [p.rows for p in parts], **kw)
        self.layout()

    def layout(self) -> None:
        self.shard_sizes, self.offset, at = [], {}, 0
        for p in self.parts:
            if p.units and p.units % self.tp_size and self.tp_size % p.units:
                raise ValueError(f"{self.name}: {p.units} heads of {p.name} do not divide over tp={self.tp_size}")
            n = p.rows // min(p.units, self.tp_size) if p.units else p.rows
            self.offset[p.name] = at
            self.shard_sizes.append(n)
            at += (n + ALIGN - 1) // ALIGN * ALIGN
        self.output_sizes = [p.rows for p in self.parts]
        self.full_out, self.out_features = sum(self.output_sizes), at

    def resize(self, **rows: int) -> None:
        """Sizes that the checkpoint's tensors give (called in front of ``load_weight``)."""
        for p in self.parts:
            p.rows = rows.get(p.name, p.rows)
        self.layout()

    def load_bias(self, **full: torch.Tensor) -> None:
        """Bias vectors of some parts; the others get none."""
        if self.bias is None:
            self.bias = torch.zeros(self.out_features, dtype=self.dtype, device=self.device)
        for p, n in zip(self.parts, self.shard_sizes):
            if p.name in full:
                i = self.tp_rank // max(1, self.tp_size // p.units) if p.units else 0
                at = self.offset[p.name]
                self.bias[at:at + n] = full[p.name][i * n:(i + 1) * n].to(self.bias.device, self.dtype)

    def shard_of(self, full_weight):
        out, at = [], 0
        for p, n in zip(self.parts, self.shard_sizes):
            w = full_weight[at:at + p.rows]
            at += p.rows
            if p.units:
                i = self.tp_rank // max(1, self.tp_size // p.units)
                w = w[i * n:(i + 1) * n]
            out.append(F.pad(w, (0, 0, 0, -n % ALIGN)))
        return torch.cat(out, 0)


class PaddedColumnLinear(ColumnParallelLinear):
    """Column-parallel layer whose input carries the zero padding of a ``PackedLinear`` part."""

    @property
    def padded_in(self) -> int:
        return (self.full_in + ALIGN - 1) // ALIGN * ALIGN

    def shard_of(self, full_weight):
        w = super().shard_of(full_weight)
        return F.pad(w, (0, -w.shape[1] % ALIGN))
