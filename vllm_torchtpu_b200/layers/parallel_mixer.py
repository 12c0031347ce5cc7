"""Two mixers side by side over the same input (``layer_specs.ParallelMixerSpec``): softmax attention behind short
convolutions (left) and a delta rule with a carried state (right).

    row  = [W_q ‖ W_k ‖ W_v ‖ W_r ‖ ... ‖ W_w1] x              one packed GEMM for both
    z    = [attention heads ‖ right heads]                      each mixer writes its columns
    y    = left_scale W_oL z_L + right_scale W_oR z_R           one GEMM

The scales leave the weights alone: the right heads' norm weights carry right_scale / left_scale (32-bit), and the sum
with the residual stream takes y times ``mult`` = left_scale.  A cache is (ring, pages, state): the convolutions' inputs and
the state are indexed by the request's batch slot.
"""
from __future__ import annotations

import torch
import torch.nn.functional as F

from .. import ops
from ..config import ModelConfig
from ..layer_specs import ParallelMixerSpec
from ..parallel.state import get_state
from .conv_attention import ConvAttention
from .linear import RowParallelLinear
from .linear_attention import RemovalDelta
from .packed import ALIGN


class JoinedRowLinear(RowParallelLinear):
    """Output projections of several mixers as one: columns of (heads, size, padded size) each, side by side, and zero
    columns up to a multiple of 8."""

    def __init__(self, name, sides: list, out_features: int, **kw):
        self.sides = sides
        tp = get_state().tp.size
        width = sum(h * padded for h, _, padded in sides) // tp
        super().__init__(name, (width + ALIGN - 1) // ALIGN * ALIGN * tp, out_features, **kw)
        self.full_in = sum(h * size for h, size, _ in sides)

    def shard_of(self, full_weight):
        out, at = [], 0
        for heads, size, padded in self.sides:
            w = full_weight[:, at:at + heads * size].reshape(full_weight.shape[0], heads, size)
            at += heads * size
            n = heads // self.tp_size
            w = F.pad(w[:, self.tp_rank * n:(self.tp_rank + 1) * n], (0, padded - size))
            out.append(w.reshape(full_weight.shape[0], n * padded))
        w = torch.cat(out, 1)
        return F.pad(w, (0, self.in_features - w.shape[1]))


class ParallelMixer:
    def __init__(self, name: str, spec: ParallelMixerSpec, cfg: ModelConfig, device, quant=None):
        self.name, self.spec, self.cfg, self.device = name, spec, cfg, device
        self.left = ConvAttention(f"{name}.left", spec.left, cfg, device, quant, RemovalDelta.parts(spec.right), False)
        self.inp = self.left.inp
        self.right = RemovalDelta(f"{name}.right", spec.right, cfg, device, self.inp, quant)
        l, r = spec.left, spec.right
        self.o = JoinedRowLinear(f"{name}.o_proj", [(l.heads, l.vdim, self.left.D), (r.heads, r.dim, r.dim)],
                                 cfg.hidden_size, dtype=cfg.dtype, device=device, quant_config=quant)
        # y / mult = left + ratio * right; without a left side its columns are zero
        self.drop_left = spec.left_scale == 0.0
        self.mult = spec.right_scale if self.drop_left else spec.left_scale
        self.ratio = 1.0 if self.drop_left else spec.right_scale / spec.left_scale

    def linears(self):
        return [self.inp, self.right.w2, self.o]

    # ---- weights ---------------------------------------------------------------
    def load_projections(self, q, k, v, r, rk, rv, g, a, w1, w2, *qkv_bias) -> None:
        """The rank of the decay projection comes with its tensors; its part is the last one."""
        self.inp.resize(**{"right.w1": w1.shape[0]})
        self.right.w2.full_in = w1.shape[0]
        self.inp.load_weight(torch.cat([q, k, v, r, rk, rv, g, a, w1], 0))
        self.right.w2.load_weight(w2)
        self.left.load_bias(*qkv_bias)

    def load_output(self, left, right) -> None:
        self.o.load_weight(torch.cat([torch.zeros_like(left) if self.drop_left else left, right], 1))

    def load_vectors(self, w0, rate_bias, norm) -> None:
        self.right.load_vectors(w0, rate_bias, norm, self.ratio)

    def init_dummy(self, std: float, seed: int) -> None:
        self.left.init_dummy(std, seed)
        self.right.w2.init_dummy(std, seed)
        self.right.init_vectors(seed, self.ratio)
        self.o.init_dummy(std, seed)

    def weight_bytes(self) -> int:
        return sum(l.weight_bytes() for l in self.linears())

    # ---- cache -----------------------------------------------------------------
    def cache_shape(self, num_blocks: int, block_size: int) -> tuple:
        return self.left.cache_shape(num_blocks, block_size)

    def allocate_cache(self, num_blocks: int, block_size: int, kv_dtype, device, slots: int):
        return self.left.allocate_cache(num_blocks, block_size, kv_dtype, device, slots) + \
            self.right.allocate_cache(num_blocks, block_size, kv_dtype, device, slots)

    def bytes_per_block(self, block_size: int, elem: int) -> int:
        return self.left.bytes_per_block(block_size, elem)

    # ---- forward ---------------------------------------------------------------
    def forward(self, x, cache, meta):
        """y / ``mult``."""
        ring, pages, state = cache
        row = self.inp(x)
        n, m = self.left.Hq * self.left.D, self.right.H * self.right.spec.dim
        z = ops.mixer_rows(x, self.o.in_features)
        q = self.left.queries(row, (ring, pages), meta)
        self.left.attend(q, row, pages, meta, out=z[:, :n])
        self.right.advance((row, self.right.decays(row)), (state,), meta, out=z[:, n:n + m])
        return self.o(z)
