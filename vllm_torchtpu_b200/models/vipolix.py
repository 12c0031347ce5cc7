"""Vipolix: decoder configured layer by layer with two mixers (gated linear attention; chunked attention and a generalised
delta rule side by side), clamped experts with a shared one, a token shift in front of every mixer and a token input of its
own behind every layer.

    h = norm1(x);  h_t <- h_t + (h_(t-1) - h_t) * shift;   x <- x + mixer(h)
    x <- x + experts(norm2(x))                                                  (absent without an MLP)
    x <- x + norm(proj (gelu_tanh(gate x) * side[token]))

norm1, norm2 and the final norm are RMS norms whose weights are stored around zero.  The residual stream is 32-bit.  The
kernel in front of a mixer adds the token input of the layer before (norm included), normalises the sum and shifts it; the
last kernel of the experts adds them to the stream and leaves it rounded for the token input's gate.
"""
from __future__ import annotations

from dataclasses import replace
from typing import Optional

import torch

from .. import ops
from ..config import ModelConfig
from ..layer_specs import GlaMixerSpec, ParallelMixerSpec
from ..layers.linear import ReplicatedLinear, seeded_normal
from ..layers.linear_attention import GatedLinear
from ..layers.parallel_mixer import ParallelMixer
from ..ops import token_shift
from .layer_list import LayerListForCausalLM, NoMLP, packed_loader, vector_loader
from .qwen3_moe import MoEBlock

NORM_OFFSET = 1.0                        # x / rms(x) * (1 + w)
MIXERS = {GlaMixerSpec: ("linear_attn", GatedLinear), ParallelMixerSpec: ("self_attn", ParallelMixer)}


class TokenShift:
    """Mix weights of a layer's token shift; its state is the previous token's normalised row of every request."""

    def __init__(self, cfg: ModelConfig, device):
        self.weight = torch.zeros(cfg.hidden_size, dtype=cfg.dtype, device=device)

    def allocate_state(self, device, slots: int) -> torch.Tensor:
        return torch.zeros(slots, self.weight.numel(), dtype=torch.float32, device=device)

    def recur(self, inputs, meta, cache) -> None:
        """Accepted rows after rejected drafts."""
        token_shift.advance(inputs[0], cache[0], meta)


class TokenInput:
    """A layer's part of the second token embedding, behind a gate that the stream drives."""

    def __init__(self, name: str, layer: int, dim: int, cfg: ModelConfig, device):
        kw = dict(dtype=cfg.dtype, device=device, quant_config=None)
        self.first = layer * dim
        self.gate = ReplicatedLinear(f"{name}.gate", cfg.hidden_size, dim, **kw)
        self.proj = ReplicatedLinear(f"{name}.proj", dim, cfg.hidden_size, **kw)
        self.norm = torch.ones(cfg.hidden_size, dtype=cfg.dtype, device=device)

    def linears(self):
        return [self.gate, self.proj]

    def forward(self, x, table, ids):
        """Before the norm, which the next norm kernel applies."""
        return self.proj(ops.gemm_token_gate(x, self.gate.weight, table, self.first, ids))


class VipolixDecoderLayer:
    def __init__(self, idx: int, cfg: ModelConfig, device, quant):
        spec = cfg.layer_specs[idx]
        name = f"model.layers.{idx}"
        self.idx, self.eps, self.spec = idx, cfg.rms_norm_eps, spec
        leaf, mixer = MIXERS[type(spec.mixer)]
        self.self_attn = mixer(f"{name}.{leaf}", spec.mixer, cfg, device, quant)
        self.mult = getattr(self.self_attn, "mult", 1.0)
        self.shift = TokenShift(cfg, device)
        zeros = lambda: torch.zeros(cfg.hidden_size, dtype=cfg.dtype, device=device)      # noqa: E731
        self.norm1 = zeros()
        self.norm2: Optional[torch.Tensor] = None
        self.mlp = NoMLP()
        self.side = TokenInput(f"{name}.side", idx, spec.side_dim, cfg, device) if spec.side_dim else None
        if spec.experts:
            e = spec.experts
            self.norm2 = zeros()
            self.mlp = MoEBlock(f"{name}.mlp", replace(
                cfg, num_experts=e.experts, num_experts_per_tok=e.top, moe_intermediate_size=e.ff, hidden_act=e.act,
                moe_n_group=e.groups, moe_topk_group=e.keep, moe_renormalize=True, moe_routed_scaling=e.scale,
                num_shared_experts=int(e.shared_ff > 0), shared_expert_intermediate_size=e.shared_ff,
                shared_expert_gate=e.shared_ff > 0, shared_expert_act=e.shared_act), device, quant)

    def forward(self, y, post, residual, cache, meta, table, ids):
        """y: token input of the layer before (None in front of the first), whose norm ``post`` and sum with ``residual``
        are still to come."""
        state, rb = cache[0], getattr(meta, "state_rollback", None)
        before = rb.snapshot((state,)) if rb is not None else None
        h, residual, rows = ops.add_rms_norm_shift(y, residual, self.norm1, self.eps, NORM_OFFSET, self.shift.weight, state,
                                                   meta, post, keep=rb is not None)
        if rb is not None:
            rb.capture(self.shift, (state,), (rows,), before)      # verification step: rejected drafts are rolled back
        y = self.self_attn.forward(h, cache[1], meta)
        if self.norm2 is not None:
            h, residual = ops.add_rms_norm(y, residual, self.norm2, self.eps, NORM_OFFSET, mult=self.mult)
            x, residual = self.mlp.forward_add(h, residual)
        else:
            x, residual = ops.residual_add(y, residual, self.mult)
        if self.side is None:
            return None, None, residual
        return self.side.forward(x, table, ids), self.side.norm, residual


class VipolixForCausalLM(LayerListForCausalLM):
    layer_cls = VipolixDecoderLayer
    fusion_reason = "mixers of several kinds behind a token shift on a 32-bit residual stream"

    def __init__(self, cfg: ModelConfig, device="cpu", layer_range=None):
        super().__init__(cfg, device, layer_range)
        self.norm.zero_()
        self.side_embed: Optional[torch.Tensor] = None

    # ---- weights -------------------------------------------------------------
    def named_linears(self):
        yield from super().named_linears()
        for l in self.layers:
            yield from l.side.linears() if l.side else []

    def init_dummy(self) -> None:
        super().init_dummy()
        cfg = self.cfg

        def vec(name, *shape, std=cfg.init_std):
            return seeded_normal(name, shape, std, cfg.dtype, self.device, cfg.seed)
        if cfg.token_side_dim:
            self.side_embed = vec("model.side_embed", cfg.vocab_size, cfg.num_layers * cfg.token_side_dim)
        for l in self.layers:
            l.shift.weight.copy_(vec(f"model.layers.{l.idx}.shift", cfg.hidden_size, std=0.3))
            for lin in l.side.linears() if l.side else []:
                lin.init_dummy(cfg.init_std, cfg.seed)

    def weight_bytes(self) -> int:
        n = super().weight_bytes() + sum(lin.weight_bytes() for l in self.layers if l.side for lin in l.side.linears())
        return n + (self.side_embed.numel() * self.side_embed.element_size() if self.side_embed is not None else 0)

    def embedding_groups(self) -> list:
        def side(t):
            cfg = self.cfg
            if t.shape[1] != cfg.num_layers * cfg.token_side_dim:
                raise ValueError(f"side.embed: {t.shape[1]} columns for {cfg.num_layers} layers of {cfg.token_side_dim}")
            self.side_embed = t.to(device=self.device, dtype=cfg.dtype).contiguous()
        return super().embedding_groups() + ([(("side.embed",), side)] if self.cfg.token_side_dim else [])

    def checkpoint_groups(self) -> list:
        groups = self.embedding_groups()
        for l in self.layers:
            a, p = l.self_attn, f"l{l.idx}."
            m = p + "mix."
            groups += [((p + "norm1",), vector_loader(l.norm1)), ((p + "shift",), vector_loader(l.shift.weight))]
            if isinstance(a, GatedLinear):
                groups += [(tuple(m + n for n in ("q", "k", "v", "g", "a1", "a2")), a.load_projections),
                           ((m + "a2.b", m + "norm"), a.load_vectors), ((m + "o",), packed_loader(a.o))]
            else:
                ml, mr = m + "left.", m + "right."
                groups += [(tuple(ml + n for n in "qkv") + tuple(mr + n for n in ("r", "k", "v", "g", "a", "w1", "w2"))
                            + tuple(ml + n + ".b" for n in "qkv"), a.load_projections),
                           (tuple(ml + n + ".conv" for n in "qkv"), a.left.load_conv), ((ml + "temp",), a.left.load_temp),
                           ((mr + "w0", mr + "a.b", mr + "norm"), a.load_vectors), ((ml + "o", mr + "o"), a.load_output)]
            if l.side:
                groups += [((p + "side.gate",), packed_loader(l.side.gate)), ((p + "side.proj",), packed_loader(l.side.proj)),
                           ((p + "side.norm",), vector_loader(l.side.norm))]
            if l.norm2 is not None:
                groups += [((p + "norm2",), vector_loader(l.norm2))] + self._expert_groups(p + "mlp.", l.mlp)
        return groups

    @staticmethod
    def _expert_groups(p: str, block: MoEBlock) -> list:
        moe = block.experts
        lo, hi = moe.expert_range
        shared = [p + "shared.sg"] if block.shared is not None else []
        groups = [((p + "router", *shared), packed_loader(moe.gate)), ((p + "correction",), vector_loader(moe.score_bias))]
        if block.shared is not None:
            groups += [((p + "shared.gate", p + "shared.up"), packed_loader(block.shared.gate_up)),
                       ((p + "shared.down",), packed_loader(block.shared.down))]
        return groups + [(tuple(f"{p}e{e}.{n}" for n in ("gate", "up", "down")),
                          lambda gate, up, down, e=e - lo: moe.load_gated(e, gate, up, down)
                          if 0 <= e < moe.num_local_experts else None) for e in range(moe.num_experts)]

    # ---- forward -------------------------------------------------------------
    def forward(self, input_ids, meta, kv_caches, *, hidden=None, residual=None):
        """``input_ids``: the tokens themselves, also where they come from the device.  Returns (token input of the last
        layer, 32-bit residual stream its norm is still to be added to)."""
        if hidden is None:
            hidden = ops.embedding(input_ids, self.embed)
        y, post, residual = None, None, hidden
        for layer, cache in zip(self.layers, kv_caches):
            y, post, residual = layer.forward(y, post, residual, cache, meta, self.side_embed, input_ids)
        return (residual if y is None else ops.materialize(y)), residual

    def finalize(self, hidden, residual):
        side = self.layers[-1].side
        return ops.add_rms_norm(hidden if side else None, residual, self.norm, self.cfg.rms_norm_eps, NORM_OFFSET,
                                update=False, post=side.norm if side else None)[0]

    # ---- caches ----------------------------------------------------------------
    def allocate_kv_caches(self, num_blocks: int, block_size: int, kv_dtype, device, max_reqs: int = 256):
        """Per layer: (state of the token shift, cache of the mixer)."""
        return [(l.shift.allocate_state(device, max_reqs + 1),
                 l.self_attn.allocate_cache(num_blocks, block_size, kv_dtype, device, max_reqs + 1)) for l in self.layers]

    def kv_bytes_per_block(self, block_size: int, kv_dtype: torch.dtype) -> int:
        elem = torch.empty((), dtype=kv_dtype).element_size()
        return sum(l.self_attn.bytes_per_block(block_size, elem) for l in self.layers)

    def kv_cache_shape(self, num_blocks: int, block_size: int) -> tuple:
        shapes = {l.self_attn.cache_shape(num_blocks, block_size) for l in self.layers if not l.spec.mixer.recurrent}
        if len(shapes) != 1:
            raise ValueError("the layers' caches differ in shape: use allocate_kv_caches")
        return shapes.pop()
