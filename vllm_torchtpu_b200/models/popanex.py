"""Popanex: decoder configured layer by layer with three mixers (softmax attention with projection norms, query
temperature and sinks; retention; a gated delta rule with one decay per key channel).

    x <- x + mixer(norm1(x));   x <- x + down(gelu_tanh(gate) * up)(norm2(x))      (the second absent without an MLP)

The norms are RMS norms whose weights are stored around zero.  The residual stream is 32-bit: a sublayer's output is
added to it by the kernel that normalises it for the next sublayer.  A layer with ``weights_of`` runs the weights of
the layer it names on a cache or state of its own.
"""
from __future__ import annotations

from typing import Optional

import torch

from .. import ops
from ..config import ModelConfig
from ..layer_specs import DeltaMixerSpec, GroupedMixerSpec, RetentionMixerSpec
from ..layers.grouped_attention import GroupedAttention
from ..layers.linear_attention import ChannelDelta, Retention
from .layer_list import LayerListForCausalLM, NoMLP, packed_loader, vector_loader
from .llama import LlamaMLP

NORM_OFFSET = 1.0                        # x / rms(x) * (1 + w)
MIXERS = {GroupedMixerSpec: ("self_attn", GroupedAttention), RetentionMixerSpec: ("retention", Retention),
          DeltaMixerSpec: ("delta", ChannelDelta)}


class PopanexDecoderLayer:
    def __init__(self, idx: int, cfg: ModelConfig, device, quant):
        spec = cfg.layer_specs[idx]
        name = f"model.layers.{idx}"
        self.idx, self.eps, self.spec = idx, cfg.rms_norm_eps, spec
        leaf, mixer = MIXERS[type(spec.mixer)]
        self.self_attn = mixer(f"{name}.{leaf}", spec.mixer, cfg, device, quant)
        self.norm1 = torch.zeros(cfg.hidden_size, dtype=cfg.dtype, device=device)
        self.norm2: Optional[torch.Tensor] = None
        self.mlp = NoMLP()
        if spec.ff:
            self.norm2 = torch.zeros(cfg.hidden_size, dtype=cfg.dtype, device=device)
            self.mlp = LlamaMLP(f"{name}.mlp", cfg, spec.ff, device, quant)

    def run_weights_of(self, owner: "PopanexDecoderLayer") -> None:
        self.self_attn, self.mlp = owner.self_attn, owner.mlp
        self.norm1, self.norm2 = owner.norm1, owner.norm2

    def forward(self, y, residual, cache, meta):
        """y: output of the sublayer before (None in front of the first layer), not yet added to ``residual``."""
        h, residual = ops.add_rms_norm(y, residual, self.norm1, self.eps, NORM_OFFSET)
        y = self.self_attn.forward(h, cache, meta)
        if self.norm2 is not None:
            h, residual = ops.add_rms_norm(y, residual, self.norm2, self.eps, NORM_OFFSET)
            y = self.mlp.forward(h)
        return y, residual


class PopanexForCausalLM(LayerListForCausalLM):
    layer_cls = PopanexDecoderLayer
    fusion_reason = "mixers of several kinds on a 32-bit residual stream"

    def __init__(self, cfg: ModelConfig, device="cpu", layer_range=None):
        super().__init__(cfg, device, layer_range)
        self.norm.zero_()
        for l in self.layers:
            if l.spec.weights_of is not None:
                l.run_weights_of(self.layers[l.spec.weights_of])

    def weight_owners(self) -> list:
        return [l for l in self.layers if l.spec.weights_of is None]

    def checkpoint_groups(self) -> list:
        groups = self.embedding_groups()
        for l in self.weight_owners():
            a, p = l.self_attn, f"l{l.idx}."
            m = p + "mix."
            groups += [((p + "norm1",), vector_loader(l.norm1)), ((m + "o",), packed_loader(a.o))]
            if isinstance(a, GroupedAttention):
                groups += [((m + "q", m + "k", m + "v"), packed_loader(a.inp)), ((m + "sink",), a.load_sinks)]
                groups += [((m + w + ".norm",), lambda t, a=a, w=w: a.load_norm(w, t)) for w in "qk"]
            elif isinstance(a, Retention):
                groups.append((tuple(m + w for w in ("q", "k", "v", "g")), packed_loader(a.inp)))
            else:
                # the low-rank second factors go in behind the first ones, whose rows give the ranks
                groups += [(tuple(m + w for w in ("q", "k", "v", "a1", "g1", "b", "a2", "g2")), a.load_projections),
                           (tuple(m + w + ".conv" for w in "qkv"), a.load_conv),
                           ((m + "A_log", m + "dt_bias", m + "norm"), a.load_vectors)]
            if l.norm2 is not None:
                groups += [((p + "norm2",), vector_loader(l.norm2)), ((p + "mlp.down",), packed_loader(l.mlp.down)),
                           ((p + "mlp.gate", p + "mlp.up"), packed_loader(l.mlp.gate_up))]
        return groups

    # ---- forward -------------------------------------------------------------
    def forward(self, input_ids, meta, kv_caches, *, hidden=None, residual=None):
        """Returns (output of the last sublayer, 32-bit residual stream it is still to be added to)."""
        if hidden is None:
            hidden = ops.embedding(input_ids, self.embed)
        y, residual = None, hidden
        for layer, cache in zip(self.layers, kv_caches):
            y, residual = layer.forward(y, residual, cache, meta)
        return ops.materialize(y), residual

    def finalize(self, hidden, residual):
        return ops.add_rms_norm(hidden, residual, self.norm, self.cfg.rms_norm_eps, NORM_OFFSET, update=False)[0]

    # ---- caches ----------------------------------------------------------------
    def allocate_kv_caches(self, num_blocks: int, block_size: int, kv_dtype, device, max_reqs: int = 256):
        return [l.self_attn.allocate_cache(num_blocks, block_size, kv_dtype, device, max_reqs + 1) for l in self.layers]

    def kv_bytes_per_block(self, block_size: int, kv_dtype: torch.dtype) -> int:
        elem = torch.empty((), dtype=kv_dtype).element_size()
        return sum(l.self_attn.bytes_per_block(block_size, elem) for l in self.layers)

    def kv_cache_shape(self, num_blocks: int, block_size: int) -> tuple:
        shapes = {l.self_attn.cache_shape(num_blocks, block_size) for l in self.layers if not l.spec.mixer.recurrent}
        if len(shapes) != 1:
            raise ValueError("the layers' caches differ in shape: use allocate_kv_caches")
        return shapes.pop()
