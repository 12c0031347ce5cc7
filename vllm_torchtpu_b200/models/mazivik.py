"""Mazivik: latent-attention decoder configured layer by layer.

A layer normalises the OUTPUT of its sublayers (layer norm, weight only) and adds it to the residual stream, which
the sublayers read as it is:

    x <- x + LN1(mixer(x));   x <- x + LN2(down(gelu(up(x))))        (the second line is absent without an MLP)

The residual stream is 32-bit; every norm kernel also stores it rounded to the model dtype as the next
projection's input.  Mixers are ``layers/latent_attention.py`` with per-layer sizes; a layer with ``kv_from`` is
handed the cache tensor of the layer it names, so the latents of a token are stored once per owning layer.  The
logits are soft-capped with tanh.
"""
from __future__ import annotations

from typing import Optional

import torch

from .. import ops
from ..config import ModelConfig
from ..layers.latent_attention import LatentAttention
from ..layers.mlp import DenseMLP
from .layer_list import LayerListForCausalLM, NoMLP, packed_loader, vector_loader


class MazivikDecoderLayer:
    def __init__(self, idx: int, cfg: ModelConfig, device, quant):
        spec = cfg.layer_specs[idx]
        name = f"model.layers.{idx}"
        self.idx, self.eps, self.spec = idx, cfg.rms_norm_eps, spec
        self.self_attn = LatentAttention(f"{name}.self_attn", spec.mixer, cfg, device, quant)
        self.norm1 = torch.ones(cfg.hidden_size, dtype=cfg.dtype, device=device)
        self.norm2: Optional[torch.Tensor] = None
        self.mlp = NoMLP()
        if spec.ff:
            self.norm2 = torch.ones(cfg.hidden_size, dtype=cfg.dtype, device=device)
            self.mlp = DenseMLP(f"{name}.mlp", cfg, spec.ff, device, quant, act=spec.act)

    def forward(self, hidden, residual, kv_cache, meta):
        """hidden: the stream rounded to the model dtype; residual: the stream itself (None in front of the first
        layer, where the embedding rows are exact in the model dtype)."""
        y = self.self_attn.forward(hidden, kv_cache, meta)
        hidden, residual = ops.layer_norm_add(y, hidden if residual is None else residual, self.norm1, self.eps)
        if self.norm2 is not None:
            hidden, residual = ops.layer_norm_add(self.mlp.forward(hidden), residual, self.norm2, self.eps)
        return hidden, residual


class MazivikForCausalLM(LayerListForCausalLM):
    layer_cls = MazivikDecoderLayer
    fusion_reason = "latent attention with normalised sublayer outputs"

    # ---- weights -------------------------------------------------------------
    def checkpoint_groups(self) -> list:
        """[(checkpoint tensors that make up one parameter, loader of these tensors)] for ``models/loader.py``."""
        groups = self.embedding_groups()
        for l in self.layers:
            a, p = l.self_attn, f"l{l.idx}."
            m = p + "mix."
            own = a.dkv_norm is not None
            groups += [((m + "dq",) + ((m + "dkv",) if own else ()) + (m + "g",), packed_loader(a.inp)),
                       ((m + "uq",), packed_loader(a.uq)), ((m + "o",), packed_loader(a.o)), ((m + "uk",), a.load_uk),
                       ((m + "uv",), a.load_uv), ((m + "dq.norm",), vector_loader(a.dq_norm)),
                       ((p + "norm1",), vector_loader(l.norm1))]
            if own:
                groups.append(((m + "dkv.norm",), vector_loader(a.dkv_norm)))
            if l.norm2 is not None:
                groups += [((p + "norm2",), vector_loader(l.norm2)), ((p + "mlp.up",), packed_loader(l.mlp.up)),
                           ((p + "mlp.down",), packed_loader(l.mlp.down))]
        return groups

    # ---- forward -------------------------------------------------------------
    def forward(self, input_ids, meta, kv_caches, *, hidden=None, residual=None):
        """Returns (32-bit residual stream, None)."""
        if hidden is None:
            hidden = ops.embedding(input_ids, self.embed)
        for layer, cache in zip(self.layers, kv_caches):
            hidden, residual = layer.forward(hidden, residual, cache, meta)
        return residual, None

    def finalize(self, hidden, residual):
        return ops.layer_norm(hidden, self.norm, self.cfg.rms_norm_eps)

    # ---- KV geometry -----------------------------------------------------------
    def _cache_owners(self) -> list:
        return [l for l in self.layers if l.spec.mixer.kv_from is None]

    def allocate_kv_caches(self, num_blocks: int, block_size: int, kv_dtype, device, max_reqs: int = 256):
        caches: list = []
        for l in self.layers:
            src = l.spec.mixer.kv_from
            caches.append(caches[src] if src is not None else torch.zeros(
                (num_blocks, block_size, l.self_attn.row_width), dtype=kv_dtype, device=device))
        return caches

    def kv_bytes_per_block(self, block_size: int, kv_dtype: torch.dtype) -> int:
        width = sum(l.self_attn.row_width for l in self._cache_owners())
        return width * block_size * torch.empty((), dtype=kv_dtype).element_size()

    def kv_cache_shape(self, num_blocks: int, block_size: int) -> tuple:
        widths = {l.self_attn.row_width for l in self._cache_owners()}
        if len(widths) > 1:
            raise ValueError("the layers' cache rows differ in width: use allocate_kv_caches")
        return (num_blocks, block_size, widths.pop())
