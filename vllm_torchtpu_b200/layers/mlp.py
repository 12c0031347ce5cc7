"""Feed-forward without a gate projection: down(act(up(x)))."""
from __future__ import annotations

import torch.nn.functional as F

from .. import ops
from ..config import ModelConfig
from ..quantization.unquantized import UnquantizedLinearMethod
from .linear import ColumnParallelLinear, RowParallelLinear


class DenseMLP:
    """``act``: "gelu" (erf form), applied in the epilogue of the up projection."""

    def __init__(self, name: str, cfg: ModelConfig, intermediate_size: int, device, quant=None, act: str = "gelu"):
        if act != "gelu":
            raise ValueError(f"{name}: ungated activation {act!r} is not built (gelu)")
        kw = dict(dtype=cfg.dtype, device=device, quant_config=quant)
        self.up = ColumnParallelLinear(f"{name}.up_proj", cfg.hidden_size, [intermediate_size], **kw)
        self.down = RowParallelLinear(f"{name}.down_proj", intermediate_size, cfg.hidden_size, **kw)

    def linears(self):
        return [self.up, self.down]

    def init_dummy(self, std: float, seed: int) -> None:
        for lin in self.linears():
            lin.init_dummy(std, seed)

    def weight_bytes(self) -> int:
        return sum(lin.weight_bytes() for lin in self.linears())

    def forward(self, x):
        from ..lora import wiring
        if type(self.up.method) is UnquantizedLinearMethod and not (self.up.lora_targets and wiring.active()):
            return self.down(ops.gemm_gelu(x, self.up.weight))
        return self.down(F.gelu(self.up(x)))
