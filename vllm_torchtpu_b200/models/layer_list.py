"""Base of the models whose configuration lists its layers one by one (``config.LayerSpec``): a 32-bit residual
stream, ops with 32-bit kernels throughout, checkpoint tensors that the model lists itself, fp32 logits with a factor
and an optional tanh soft cap."""
from __future__ import annotations

import torch

from .. import ops
from ..layers.linear import seeded_normal
from ..parallel.communicator import get_tp_comm
from .llama import LlamaForCausalLM


class NoMLP:
    """Stands for the feed-forward of a layer that has none."""

    def linears(self):
        return []

    def init_dummy(self, std, seed):
        pass

    def weight_bytes(self):
        return 0


def vector_loader(t: torch.Tensor):
    return lambda src: t.copy_(src.to(device=t.device, dtype=t.dtype))


def packed_loader(lin):
    return lambda *parts: lin.load_weight(torch.cat(parts, 0) if len(parts) > 1 else parts[0])


class LayerListForCausalLM(LlamaForCausalLM):
    float32_kernels = True              # every op of these models has a 32-bit CUDA kernel
    fusion_reason = "layers configured one by one"

    def weight_owners(self) -> list:
        """Layers that hold weights (one that runs with another's is not among them)."""
        return self.layers

    def named_linears(self):
        for l in self.weight_owners():
            yield from l.self_attn.linears()
            yield from l.mlp.linears()

    def init_dummy(self) -> None:
        cfg = self.cfg
        std, seed = cfg.init_std, cfg.seed
        self.embed = seeded_normal("model.embed_tokens", (cfg.vocab_size, cfg.hidden_size), std, cfg.dtype, self.device,
                                   seed)
        self.lm_head = self._shard_vocab(self.embed if cfg.tie_word_embeddings else seeded_normal(
            "lm_head", (cfg.vocab_size, cfg.hidden_size), std, cfg.dtype, self.device, seed))
        for l in self.weight_owners():
            l.self_attn.init_dummy(std, seed)
            l.mlp.init_dummy(std, seed)

    def weight_bytes(self) -> int:
        n = sum(t.numel() * t.element_size() for t in {id(t): t for t in (self.embed, self.lm_head)}.values() if t is not None)
        return n + sum(l.self_attn.weight_bytes() + l.mlp.weight_bytes() for l in self.weight_owners())

    def embedding_groups(self) -> list:
        """[(checkpoint tensors that make up one parameter, loader of these tensors)] of what is outside the layers."""
        def embed(t):
            self.embed = t.to(device=self.device, dtype=self.cfg.dtype).contiguous()
            if self.cfg.tie_word_embeddings:
                self.lm_head = self._shard_vocab(self.embed)

        def head(t):
            self.lm_head = self._shard_vocab(t.to(device=self.device, dtype=self.cfg.dtype).contiguous())
        groups = [(("embed",), embed), (("final.norm",), vector_loader(self.norm))]
        return groups if self.cfg.tie_word_embeddings else groups + [(("head",), head)]

    def setup_decode_fusion(self, kv_caches) -> None:
        self.decode_mega, self.decode_mega_reason = None, self.fusion_reason

    def compute_logits(self, hidden_rows):
        """fp32, scaled and soft-capped."""
        cap, scale = self.cfg.final_logit_softcap or 0.0, self.cfg.logit_scale
        if getattr(self, "dp_vocab", None) is not None:
            logits = self.dp_vocab.logits(hidden_rows, self.lm_head)
            logits = logits * scale if scale != 1.0 else logits
            return ops.softcap(logits, cap) if cap else logits
        logits = self.local_logits(hidden_rows)
        comm = get_tp_comm()
        return comm.all_gather(logits, dim=-1) if comm.size > 1 and self.vocab_shard is not None else logits

    def local_logits(self, hidden_rows):
        return ops.gemm_softcap(hidden_rows, self.lm_head, self.cfg.final_logit_softcap or 0.0, self.cfg.logit_scale)
