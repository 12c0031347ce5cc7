"""Op entry points used by layers.

CUDA tensors go to the hand-written sm_100a kernels (``ops.cuda``, loaded from
the in-tree shared library; a missing library on a GPU box is an error, never a
silent fallback).  CPU tensors go to the plain-PyTorch statements in
``ops.reference`` so the whole engine also runs in CPU unit tests.
"""
from __future__ import annotations

import torch

from . import reference as ref

_cuda = None


def cuda_ops():
    global _cuda
    if _cuda is None:
        from . import cuda as _c
        _cuda = _c
    return _cuda


def _on_gpu(t: torch.Tensor) -> bool:
    return t.is_cuda


def rms_norm(x, weight, eps):
    return cuda_ops().rms_norm(x, weight, eps) if _on_gpu(x) else ref.rms_norm(x, weight, eps)


def layer_norm(x, weight, eps):
    return cuda_ops().layer_norm(x, weight, eps) if _on_gpu(x) else ref.layer_norm(x, weight, eps)


def layer_norm_add(y, residual, weight, eps):
    """(rounded r', fp32 r') of r' = residual + LN(y) * weight; an fp32 residual is updated in place on a GPU."""
    return cuda_ops().layer_norm_add(y, residual, weight, eps) if _on_gpu(y) else \
        ref.layer_norm_add(y, residual, weight, eps)


def add_rms_norm(y, residual, weight, eps, offset=0.0, update=True, post=None, mult=1.0):
    """(h, fp32 r) of r = residual (+ mult * y), h = RMS norm of r times (offset + weight); an fp32 residual is updated in
    place on a GPU.  ``y`` None: r = residual.  ``post``: the RMS norm of y with this weight, times ``mult``, is added
    instead of y.  Without ``update`` the stream is only read and r is None."""
    y = materialize(y)
    return cuda_ops().add_rms_norm(y, residual, weight, eps, offset, update, post, mult) if _on_gpu(residual) else \
        ref.add_rms_norm(y, residual, weight, eps, offset, update, post, mult)


def add_rms_norm_shift(y, residual, weight, eps, offset, shift, state, meta, post=None, mult=1.0, keep=False):
    """Residual sum and norm of ``add_rms_norm`` with a token shift behind them; see ``ops.token_shift``."""
    if _on_gpu(residual):
        return cuda_ops().add_rms_norm_shift(materialize(y), residual, weight, eps, offset, shift, state, meta, post, mult,
                                             keep)
    from .token_shift import add_rms_norm_shift as f
    return f(materialize(y), residual, weight, eps, offset, shift, state, meta, post, mult, keep)


def add_gated(y, z, gate):
    """y + sigmoid(gate)[:, None] * z, gate fp32 [T] (rows may be strided)."""
    if _on_gpu(y):
        return cuda_ops().add_gated(y, z, gate)
    return (y.float() + torch.sigmoid(gate.float())[:, None] * z.float()).to(y.dtype)


def residual_add(y, residual, mult=1.0, dtype=None):
    """(r rounded to ``dtype``, fp32 r) of r = residual + mult * y; r may be the residual's storage."""
    y = materialize(y)
    return cuda_ops().residual_add(y, residual, mult, dtype) if _on_gpu(y) else ref.residual_add(y, residual, mult, dtype)


def gemm_token_gate(x, w, table, first, ids):
    """gelu_tanh(x @ w.T) * table[ids, first : first + N], in the GEMM's epilogue on a GPU."""
    f = cuda_ops().gemm_token_gate if _on_gpu(x) else ref.gemm_token_gate
    return f(x, w, table, first, ids)


def resolve_tokens(ids, token_src, last_tokens):
    """Token ids of a step's rows: those still on the device (token_src >= 0) are last_tokens[token_src]."""
    if _on_gpu(ids):
        return cuda_ops().resolve_tokens(ids, token_src, last_tokens)
    return torch.where(token_src >= 0, last_tokens[token_src.clamp_min(0).long()], ids)


def softcap(x, cap):
    return cuda_ops().softcap(x, cap) if _on_gpu(x) else ref.softcap(x, cap)


def materialize(x):
    """A row-parallel output whose cross-rank sum is still pending becomes a tensor."""
    return x.materialize() if hasattr(x, "materialize") else x


def fused_add_rms_norm(x, residual, weight, eps):
    if hasattr(x, "add_rms_norm"):          # pushed partials: the sum rides in this kernel
        return x.add_rms_norm(residual, weight, eps)
    if _on_gpu(x):
        return cuda_ops().fused_add_rms_norm(x, residual, weight, eps)
    return ref.fused_add_rms_norm(x, residual, weight, eps)


def gated_act_and_mul(x, spec: str = "silu"):
    if spec == "silu":
        return silu_and_mul(x)
    return cuda_ops().gated_act_and_mul(x, spec) if _on_gpu(x) else ref.gated_act_and_mul(x, spec)


def silu_and_mul(x):
    return cuda_ops().silu_and_mul(x) if _on_gpu(x) else ref.silu_and_mul(x)


def gemm(x, w, bias=None, out=None):
    return cuda_ops().gemm(x, w, bias, out=out) if _on_gpu(x) else ref.gemm(x, w, bias)


def gemm_gelu(x, w):
    """gelu(x @ w.T) with gelu in its erf form, in the GEMM's epilogue on a GPU."""
    return cuda_ops().gemm_gelu(x, w) if _on_gpu(x) else ref.gemm_gelu(x, w)


def gemm_softcap(x, w, cap=0.0, scale=1.0):
    """fp32 logits with a factor and the tanh soft cap in the GEMM's epilogue on a GPU; see
    ``ops.reference.gemm_softcap``."""
    return cuda_ops().gemm_softcap(x, w, cap, scale) if _on_gpu(x) else ref.gemm_softcap(x, w, cap, scale)


def gemm_gated(x, w, act):
    """act(x @ w[:I].T, x @ w[I:].T), in the GEMM's epilogue where it has the activation (silu, gelu_tanh)."""
    return cuda_ops().gemm_gated(x, w, act) if _on_gpu(x) else ref.gated_act_and_mul(ref.gemm(x, w), act)


def carried_state_attention(plan, row, decay_in, gate, meta, cache, out=None):
    """Linear attention with a carried state; see ``ops.linear_attention``.  ``out``: [T, heads * vdim], rows may be
    strided."""
    if _on_gpu(row):
        return cuda_ops().carried_state_attention(plan, row, decay_in, gate, meta, cache, out)
    from .linear_attention import linear_attention_reference
    return linear_attention_reference(plan, row, decay_in, gate, meta, cache, out)


def mixer_rows(x, width: int):
    """[T, width] rows that mixers write into; rows of padding stay finite."""
    if _on_gpu(x) and x.dtype == torch.bfloat16:
        return cuda_ops().Workspace.get(x.device).attn_out(x.shape[0], 1, width)[:, 0]
    return torch.zeros(x.shape[0], width, dtype=x.dtype, device=x.device)


def tanh_(x):
    """In place, fp32 inside; rows may be strided."""
    return cuda_ops().tanh_(x) if _on_gpu(x) else x.copy_(torch.tanh(x.float()))


def gemm_heads(x, w, gate=None, out=None):
    """Per-head product x [T, H, >= K] with w [H, N, K] -> [T, H, N]; see ``ops.reference.gemm_heads``."""
    return cuda_ops().gemm_heads(x, w, gate, out) if _on_gpu(x) else ref.gemm_heads(x, w, gate, out)


def latent_prep(*a, **kw):
    return cuda_ops().latent_prep(*a, **kw) if _on_gpu(a[0]) else ref.latent_prep(*a, **kw)


def rope_heads_into(q, out, *a, **kw):
    return cuda_ops().rope_heads_into(q, out, *a, **kw) if _on_gpu(q) else ref.rope_heads_into(q, out, *a, **kw)


def embedding_pairs(ids, prev, table, pairs, bigram, token_src, last_tokens, last_inputs):
    """fp32 sum of token and bigram embeddings; see ``ops.reference.embedding_pairs``."""
    f = cuda_ops().embedding_pairs if _on_gpu(table) else ref.embedding_pairs
    return f(ids, prev, table, pairs, bigram, token_src, last_tokens, last_inputs)


def conv_and_cache(plan, row, kv_cache, ring, meta):
    """Short convolutions, rotation and cache write of an attention layer; see ``ops.short_conv``."""
    if _on_gpu(row):
        return cuda_ops().conv_and_cache(plan, row, kv_cache, ring, meta)
    from .short_conv import conv_and_cache as f
    return f(plan, row, kv_cache, ring, meta)


def conv_ring_update(plan, row, ring, meta):
    if _on_gpu(row):
        return cuda_ops().conv_ring_update(plan, row, ring, meta)
    from .short_conv import ring_update as f
    return f(plan, row, ring, meta)


def paged_attention_heads(q, kv_cache, meta, scale, window, vdim, gate=None, lam=None, diff=0.0, eps=0.0):
    """Paged attention over a window and ``combine_heads`` behind it, in the attention kernels' epilogue where they have
    it: [T, heads, width]."""
    if _on_gpu(q):
        return cuda_ops().paged_attention_heads(q, kv_cache, meta, scale, window, vdim, gate, lam, diff, eps)
    return combine_heads(paged_attention(q, kv_cache, meta, scale, sliding_window=window), vdim, gate, lam, diff, eps)


def combine_heads(a, vdim, gate=None, lam=None, diff=0.0, eps=0.0):
    """Difference of two softmax maps with its norm, output gate; see ``ops.short_conv``."""
    if _on_gpu(a):
        return cuda_ops().combine_heads(a, vdim, gate, lam, diff, eps)
    from .short_conv import combine_heads as f
    return f(a, vdim, gate, lam, diff, eps)


def embedding(ids, table):
    return cuda_ops().embedding(ids, table) if _on_gpu(table) else ref.embedding(ids, table)


def rope_and_cache(qkv, positions, inv_freq, kv_cache, slot_mapping, num_q_heads, num_kv_heads,
                   head_dim, interleaved=False, q_norm_w=None, k_norm_w=None, eps=1e-6,
                   k_scale=1.0, v_scale=1.0):
    f = cuda_ops().rope_and_cache if _on_gpu(qkv) else ref.rope_and_cache
    return f(qkv, positions, inv_freq, kv_cache, slot_mapping, num_q_heads, num_kv_heads, head_dim,
             interleaved, q_norm_w, k_norm_w, eps, k_scale, v_scale)


def norm_and_cache(qkv, positions, kv_cache, slot_mapping, *a, **kw):
    f = cuda_ops().norm_and_cache if _on_gpu(qkv) else ref.norm_and_cache
    return f(qkv, positions, kv_cache, slot_mapping, *a, **kw)


def paged_attention(q, kv_cache, meta, scale, *, sliding_window=None, softcap=None, sinks=None,
                    k_scale=1.0, v_scale=1.0, return_lse=False, out=None):
    """``sliding_window`` n > 0: a query sees the last n keys; n < 0: the keys of its own chunk of -n positions.  ``out``:
    [T, >= heads * dim] rows, which may be strided, for the heads side by side."""
    if _on_gpu(q):
        return cuda_ops().paged_attention(q, kv_cache, meta, scale, sliding_window=sliding_window,
                                          softcap=softcap, sinks=sinks, k_scale=k_scale,
                                          v_scale=v_scale, return_lse=return_lse, out=out)
    if out is not None:
        o = paged_attention(q, kv_cache, meta, scale, sliding_window=sliding_window, softcap=softcap, sinks=sinks)
        return out[:, :o.shape[1] * o.shape[2]].copy_(o.reshape(o.shape[0], -1))
    return ref.paged_attention(q, kv_cache, meta.block_tables, meta.seq_lens, meta.query_start_loc,
                               scale, num_reqs=meta.num_reqs, sliding_window=sliding_window,
                               softcap=softcap, sinks=sinks, k_scale=k_scale, v_scale=v_scale,
                               return_lse=return_lse, global_seq_lens=meta.global_seq_lens,
                               dcp_size=meta.dcp_size, dcp_rank=meta.dcp_rank,
                               dcp_interleave=meta.dcp_interleave)


def mla_write_cache(cache, kv_c, k_pe, slot_mapping):
    if _on_gpu(cache):
        return cuda_ops().mla_write_cache(cache, kv_c, k_pe, slot_mapping)
    return ref.mla_write_cache(cache, kv_c, k_pe, slot_mapping)


def mla_paged_attention(q_latent, cache, meta, scale, kv_lora_rank, *, topk_indices=None, return_lse=False):
    if _on_gpu(q_latent):
        return cuda_ops().mla_paged_attention(q_latent, cache, meta, scale, kv_lora_rank,
                                              topk_indices=topk_indices, return_lse=return_lse)
    return ref.mla_paged_attention(q_latent, cache, meta.block_tables, meta.seq_lens, meta.query_start_loc,
                                   scale, kv_lora_rank, num_reqs=meta.num_reqs, topk_indices=topk_indices,
                                   return_lse=return_lse)


def sample(logits, temperature, top_k, top_p, uniform=None, all_greedy=False):
    if _on_gpu(logits):
        return cuda_ops().sample(logits, temperature, top_k, top_p, uniform, all_greedy)
    return ref.sample(logits, temperature, top_k, top_p, None if all_greedy else uniform)


def moe_route(router_logits, top_k, **kw):
    if _on_gpu(router_logits):
        return cuda_ops().moe_route(router_logits, top_k, **kw)
    return ref.moe_route(router_logits, top_k, **kw)


# ---- launch accounting ---------------------------------------------------------
_launches = 0


def count_launch(n: int = 1) -> None:
    """Every wrapper of a hand-written kernel calls this once per launch."""
    global _launches
    _launches += n


def launch_count() -> int:
    return _launches
