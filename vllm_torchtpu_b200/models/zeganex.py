"""Zeganex: decoder configured layer by layer with two mixers (differential attention; rotated attention with an output
gate), both behind short convolutions and with a sliding window, and dense or expert feed-forwards.

    x = embed[token] + bigram[previous token, token]
    x <- x + m * norm1b(mixer(norm1(x)));   x <- x + m * norm2b(ff(norm2(x)))      (the second absent without an MLP)

Sublayer inputs and outputs pass RMS norms.  The residual stream is 32-bit from the embedding on: a sublayer's output is
handed on as it is, and the kernel that prepares the next sublayer's input normalises it, scales it, adds it to the stream
and normalises the sum.  Layers with ``kv_from`` read the pages of an earlier layer.  The head is the embedding table.
"""
from __future__ import annotations

from dataclasses import replace
from typing import Optional

import torch

from .. import ops
from ..config import ModelConfig
from ..layers.conv_attention import ConvAttention
from ..layers.linear import seeded_normal
from .layer_list import LayerListForCausalLM, NoMLP, packed_loader, vector_loader
from .llama import LlamaMLP
from .qwen3_moe import MoEBlock


class ZeganexDecoderLayer:
    def __init__(self, idx: int, cfg: ModelConfig, device, quant):
        spec = cfg.layer_specs[idx]
        name = f"model.layers.{idx}"
        self.idx, self.eps, self.mult, self.spec = idx, cfg.rms_norm_eps, cfg.residual_mult, spec
        self.self_attn = ConvAttention(f"{name}.self_attn", spec.mixer, cfg, device, quant)
        ones = lambda: torch.ones(cfg.hidden_size, dtype=cfg.dtype, device=device)      # noqa: E731
        self.norm1, self.norm1b = ones(), ones()
        self.norm2: Optional[torch.Tensor] = None
        self.norm2b: Optional[torch.Tensor] = None
        self.mlp = NoMLP()
        if spec.ff or spec.experts:
            self.norm2, self.norm2b = ones(), ones()
        if spec.experts:
            e = spec.experts
            self.mlp = MoEBlock(f"{name}.mlp", replace(cfg, num_experts=e.experts, num_experts_per_tok=e.top,
                                                       moe_intermediate_size=e.ff, hidden_act=e.act), device, quant)
        elif spec.ff:
            self.mlp = LlamaMLP(f"{name}.mlp", cfg, spec.ff, device, quant)

    @property
    def last_norm(self) -> torch.Tensor:
        """Weight of the norm that the layer's output still has to pass."""
        return self.norm1b if self.norm2b is None else self.norm2b

    def forward(self, y, post, residual, cache, meta):
        """y: output of the sublayer before (None in front of the first layer), whose norm ``post`` and sum with
        ``residual`` are still to come."""
        h, residual = ops.add_rms_norm(y, residual, self.norm1, self.eps, post=post, mult=self.mult)
        y = self.self_attn.forward(h, cache, meta)
        if self.norm2 is not None:
            h, residual = ops.add_rms_norm(y, residual, self.norm2, self.eps, post=self.norm1b, mult=self.mult)
            y = self.mlp.forward(h)
        return y, self.last_norm, residual


class ZeganexForCausalLM(LayerListForCausalLM):
    layer_cls = ZeganexDecoderLayer
    fusion_reason = "short convolutions and normalised sublayer outputs"

    def __init__(self, cfg: ModelConfig, device="cpu", layer_range=None):
        super().__init__(cfg, device, layer_range)
        self.bigram: Optional[torch.Tensor] = None

    # ---- weights -------------------------------------------------------------
    def init_dummy(self) -> None:
        super().init_dummy()
        cfg = self.cfg
        if cfg.bigram:
            self.bigram = seeded_normal("model.bigram", (cfg.bigram[0] + 1, cfg.hidden_size), cfg.init_std, cfg.dtype,
                                        self.device, cfg.seed)

    def weight_bytes(self) -> int:
        n = super().weight_bytes()
        return n + (self.bigram.numel() * self.bigram.element_size() if self.bigram is not None else 0)

    def embedding_groups(self) -> list:
        def pairs(t):
            if t.shape[0] != self.cfg.bigram[0] + 1:
                raise ValueError(f"bigram: {t.shape[0]} rows for {self.cfg.bigram[0]} buckets and the first token's")
            self.bigram = t.to(device=self.device, dtype=self.cfg.dtype).contiguous()
        return super().embedding_groups() + ([(("bigram",), pairs)] if self.cfg.bigram else [])

    def checkpoint_groups(self) -> list:
        groups = self.embedding_groups()
        for l in self.layers:
            a, s, p = l.self_attn, l.spec.mixer, f"l{l.idx}."
            m = p + "mix."
            qkv = [m + n for n in ("q", "k", "v") if n == "q" or s.kv_from is None]
            groups += [((p + n,), vector_loader(getattr(l, n))) for n in ("norm1", "norm1b")]
            groups += [(tuple(qkv) + ((m + "g",) if s.output_gate else ()), packed_loader(a.inp)),
                       (tuple(n + ".b" for n in qkv), a.load_bias), (tuple(n + ".conv" for n in qkv), a.load_conv),
                       ((m + "o",), packed_loader(a.o))]
            if s.out_bias:
                groups.append(((m + "o.b",), a.load_out_bias))
            if s.maps == 2:
                groups.append((tuple(m + n for n in ("lq1", "lk1", "lq2", "lk2")), a.load_lambda))
            if l.norm2 is None:
                continue
            groups += [((p + n,), vector_loader(getattr(l, n))) for n in ("norm2", "norm2b")]
            if l.spec.experts:
                moe = l.mlp.experts
                groups.append(((p + "mlp.router",), packed_loader(moe.gate)))
                lo, hi = moe.expert_range
                groups += [((f"{p}mlp.e{e}.up", f"{p}mlp.e{e}.down"), lambda up, down, moe=moe, e=e - lo: moe.load_ungated(
                    e, up, down) if 0 <= e < moe.num_local_experts else None) for e in range(moe.num_experts)]
            else:
                groups += [((p + "mlp.gate", p + "mlp.up"), packed_loader(l.mlp.gate_up)),
                           ((p + "mlp.down",), packed_loader(l.mlp.down))]
        return groups

    # ---- forward -------------------------------------------------------------
    def forward(self, input_ids, meta, kv_caches, *, hidden=None, residual=None):
        """``hidden``: the embeddings, fp32.  Returns (output of the last sublayer, 32-bit residual stream its norm is
        still to be added to)."""
        if hidden is None:
            if self.cfg.bigram:
                raise ValueError("the embedding of a bigram model needs the previous tokens: pass hidden")
            hidden = ops.embedding(input_ids, self.embed)
        y, post, residual = None, None, hidden
        for layer, cache in zip(self.layers, kv_caches):
            y, post, residual = layer.forward(y, post, residual, cache, meta)
        return ops.materialize(y), residual

    def finalize(self, hidden, residual):
        last = self.layers[-1]
        return ops.add_rms_norm(hidden, residual, self.norm, self.cfg.rms_norm_eps, update=False, post=last.last_norm,
                                mult=last.mult)[0]

    # ---- caches ----------------------------------------------------------------
    def allocate_kv_caches(self, num_blocks: int, block_size: int, kv_dtype, device, max_reqs: int = 256):
        caches: list = []
        for l in self.layers:
            src = l.spec.mixer.kv_from
            caches.append(l.self_attn.allocate_cache(num_blocks, block_size, kv_dtype, device, max_reqs + 1,
                                                     shared=None if src is None else caches[src]))
        return caches

    def kv_bytes_per_block(self, block_size: int, kv_dtype: torch.dtype) -> int:
        elem = torch.empty((), dtype=kv_dtype).element_size()
        return sum(l.self_attn.bytes_per_block(block_size, elem) for l in self.layers)

    def kv_cache_shape(self, num_blocks: int, block_size: int) -> tuple:
        shapes = {l.self_attn.cache_shape(num_blocks, block_size) for l in self.layers}
        if len(shapes) != 1:
            raise ValueError("the layers' caches differ in shape: use allocate_kv_caches")
        return shapes.pop()
