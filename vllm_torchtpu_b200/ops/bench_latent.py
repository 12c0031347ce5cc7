"""Layer throughput of Mazivik beside DeepSeek's latent attention at equal size, and the kernels of both.

    python bench.py --layer-bench mazivik [--layer-size 2048x16,4096x32]

Random weights; a model of a few layers without embedding and head runs one prefill batch (four prompts of 2048
tokens) and one decode batch (64 requests with 2048 cached tokens) through ``model.forward``, as one CUDA graph.
The neighbour is the DeepSeek-V3 layer class with a dense SwiGLU MLP of the same parameter count, the same latent
and head sizes.  CUDA events, L2 flushed before every timed launch, median; fractions are of the measured peaks.
"""
from __future__ import annotations

import torch

from ..config import ModelConfig
from ..runner.attn_metadata import AttentionMetadata
from .bench_kernels import peaks, time_fn

LATENT = dict(dim=128, rot_dim=64, vdim=128, kv_rank=512)
BS = 16


def mazivik_config(width: int, heads: int, layers: int, q_rank: int, ff: int, share: bool) -> ModelConfig:
    rot = {"base": 50000.0, "dims": LATENT["rot_dim"],
           "scaling": {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}}
    mix = dict(LATENT, heads=heads, q_rank=q_rank, scale=(LATENT["dim"] + LATENT["rot_dim"]) ** -0.5, rot=rot)
    entries = [{"type": "latent_attention", "mixer": dict(mix, kv_from=i - 1) if share and i % 2 else mix,
                "mlp": {"kind": "dense", "ff": ff}} for i in range(layers)]
    mc = ModelConfig.from_layer_list({"architecture": "Mazivik", "width": width, "vocab": 1024, "norm": {"eps": 1e-6},
                                      "logit_softcap": 30.0, "layers": entries}, "mazivik-bench")
    return mc


def deepseek_config(width: int, heads: int, layers: int, q_rank: int, ff: int) -> ModelConfig:
    return ModelConfig(name="deepseek-bench", architecture="deepseek_v3", num_layers=layers, hidden_size=width,
                       num_q_heads=heads, num_kv_heads=heads, head_dim=LATENT["dim"] + LATENT["rot_dim"],
                       intermediate_size=ff, vocab_size=1024, q_lora_rank=q_rank, kv_lora_rank=LATENT["kv_rank"],
                       qk_nope_head_dim=LATENT["dim"], qk_rope_head_dim=LATENT["rot_dim"], v_head_dim=LATENT["vdim"],
                       rope_interleaved=True, rope_theta=50000.0)


def step_meta(q_len: int, ctx: int, reqs: int, device="cuda"):
    """(metadata, number of blocks) of ``reqs`` requests that run ``q_len`` tokens behind ``ctx`` cached ones."""
    n = q_len + ctx
    nblk = -(-n // BS)
    g = torch.Generator().manual_seed(0)
    bt = (torch.randperm(reqs * nblk, generator=g) + 1).to(torch.int32).view(reqs, nblk)
    pos = torch.arange(ctx, n).repeat(reqs)
    slots = bt[torch.arange(reqs).repeat_interleave(q_len), pos // BS].long() * BS + pos % BS
    qsl = torch.arange(reqs + 1) * q_len
    dec = reqs if q_len == 1 else 0
    T = reqs * q_len
    to = lambda t: t.to(torch.int32).to(device)
    return AttentionMetadata(to(pos), to(slots), to(bt), to(torch.full((reqs,), n)), to(qsl), reqs, T,
                             num_decode_reqs=dec, max_query_len=q_len, max_seq_len=n, padded_num_reqs=reqs,
                             padded_num_tokens=T, query_start_loc_cpu=qsl, state_slots=to(torch.arange(reqs))), \
        reqs * nblk + 1


def build(cfg: ModelConfig):
    from ..models.registry import get_model_class
    cfg.dtype = torch.bfloat16
    model = get_model_class(cfg)(cfg, "cuda")
    model.init_dummy()
    return model


def caches_of(model, blocks: int):
    if hasattr(model, "allocate_kv_caches"):
        caches = model.allocate_kv_caches(blocks, BS, torch.bfloat16, "cuda")
    else:
        caches = [torch.zeros(model.kv_cache_shape(blocks, BS), dtype=torch.bfloat16, device="cuda")
                  for _ in model.layers]
    for c in {id(c): c for c in caches}.values():
        c.normal_(0, 0.3)
    return caches


STEPS = {"prefill": (2048, 0, 4), "decode": (1, 2047, 64)}


def bench_layers(width: int, heads: int, layers: int = 4, iters: int = 10) -> list:
    """Milliseconds and tokens per second of ``layers`` layers of both models."""
    q_rank, ff = width * 3 // 8, 4 * width
    swiglu = ff * 2 // 3 // 128 * 128
    rows = []
    for name, cfg in (("mazivik", mazivik_config(width, heads, layers, q_rank, ff, False)),
                      ("mazivik, every second layer shares its latent", mazivik_config(width, heads, layers, q_rank, ff, True)),
                      ("deepseek_v3 layer, dense", deepseek_config(width, heads, layers, q_rank, swiglu))):
        cfg.first_dense_layers = layers
        model = build(cfg)
        for step, (q_len, ctx, reqs) in STEPS.items():
            meta, blocks = step_meta(q_len, ctx, reqs)
            caches = caches_of(model, blocks)
            x = torch.randn(reqs * q_len, width, device="cuda").bfloat16()
            ms = time_fn(lambda: model.forward(None, meta, caches, hidden=x), iters)
            rows.append({"op": "layers", "model": name, "width": width, "heads": heads, "layers": layers, "step": step,
                         "tokens": reqs * q_len, "context": q_len + ctx, "ms": round(ms, 4),
                         "tok_s_per_layer": round(reqs * q_len * layers / ms * 1e3),
                         "weight_mb": round((model.weight_bytes() - 4 * 1024 * width) / 1e6, 1)})
            del caches
        del model
        torch.cuda.empty_cache()
    return rows


def _pairs(width: int, heads: int, step: str):
    """(what, step kernel of Mazivik, its flops, bytes; like kernel of the DeepSeek layer, flops, bytes)."""
    from . import cuda, ref
    q_len, ctx, reqs = STEPS[step]
    T, H = q_len * reqs, heads
    dn, R, v, L = LATENT["dim"], LATENT["rot_dim"], LATENT["vdim"], LATENT["kv_rank"]
    Q, ff = width * 3 // 8, 4 * width
    I = ff * 2 // 3 // 128 * 128
    Dq, eps = L + R, 1e-6
    rnd = lambda *s: (torch.randn(*s, device="cuda") * 0.1).bfloat16()
    meta, blocks = step_meta(q_len, ctx, reqs)
    cache = rnd(blocks, BS, Dq)
    inv = ref.rope_inv_freq(R, 50000.0, None).cuda()
    x, n_in = rnd(T, width), Q + L + R + H * v
    w_in, w_q, w_kv, w_uq = rnd(n_in, width), rnd(Q, width), rnd(L + R, width), rnd(H * (dn + R), Q)
    row, cq, kv = rnd(T, n_in), rnd(T, Q), rnd(T, L + R)
    nq, nc, nw = rnd(Q), rnd(L), rnd(width)
    q, ql = rnd(T, H, dn + R), rnd(T, H, Dq)
    uk, uv, o_lat = rnd(H, L, dn), rnd(H, v, L), rnd(T, H, L)
    w_o, heads_out, res = rnd(width, H * v), rnd(T, H * v), torch.randn(T, width, device="cuda")
    w_up, w_dn, h_ff = rnd(ff, width), rnd(width, ff), rnd(T, ff)
    w_gu, w_dn2, h_i, res16 = rnd(2 * I, width), rnd(width, I), rnd(T, I), rnd(T, width)
    gemm_fb = lambda n, k: (2.0 * T * n * k, 2.0 * (n * k + T * k + T * n))
    keys = reqs * (q_len * ctx + q_len * (q_len + 1) / 2)               # visible (query, key) pairs
    attn = (2.0 * keys * H * (Dq + L), 2.0 * (reqs * (q_len + ctx) * Dq + T * H * (Dq + L)))

    def absorb():
        cuda.gemm_heads(q, uk, out=ql)
        cuda.rope_heads_into(q, ql, dn, R, L, meta.positions, inv, 1.2)

    def ds_prep():
        cuda.rms_norm(cq, nq, eps)
        kv_c = cuda.rms_norm(kv[:, :L].contiguous(), nc, eps)
        cuda.mla_write_cache(cache, kv_c, kv[:, L:], meta.slot_mapping)

    def ds_in():
        cuda.gemm(x, w_q)
        cuda.gemm(x, w_kv)
    prep_b = 2.0 * T * (2 * Q + 2 * (L + R))
    head_in = (2.0 * T * H * dn * L, 2.0 * (H * L * dn + T * H * (dn + R + Dq)))
    head_out = (2.0 * T * H * v * L, 2.0 * (H * L * v + T * H * (L + v)))
    yield ("input projection (query latent, latent, gate)", lambda: cuda.gemm(x, w_in), *gemm_fb(n_in, width),
           ds_in, *[a + b for a, b in zip(gemm_fb(Q, width), gemm_fb(L + R, width))])
    yield ("latent norms, key rotation, cache write",
           lambda: cuda.latent_prep(row, nq, nc, cache, meta.slot_mapping, meta.positions, inv, 1.2, eps, L, R), 0.0, prep_b,
           ds_prep, 0.0, prep_b)
    yield ("query expansion", lambda: cuda.gemm(cq, w_uq), *gemm_fb(H * (dn + R), Q),
           lambda: cuda.gemm(cq, w_uq), *gemm_fb(H * (dn + R), Q))
    yield ("W_uk per head, query rotation", absorb, *head_in,
           lambda: cuda.mla_absorb(q, kv, meta.positions, inv, uk, dn, R, L, True), *head_in)
    yield ("latent attention", lambda: cuda.mla_paged_attention(ql, cache, meta, 0.07, L), *attn,
           lambda: cuda.mla_paged_attention(ql, cache, meta, 0.07, L), *attn)
    yield ("W_uv per head (with gate)", lambda: cuda.gemm_heads(o_lat, uv, gate=row[:, Q + L + R:]), head_out[0],
           head_out[1] + 2.0 * T * H * v, lambda: cuda.mla_unabsorb(o_lat, uv), *head_out)
    yield ("output projection", lambda: cuda.gemm(heads_out, w_o), *gemm_fb(width, H * v),
           lambda: cuda.gemm(heads_out, w_o), *gemm_fb(width, H * v))
    yield ("norm and residual", lambda: cuda.layer_norm_add(x, res, nw, eps), 0.0, T * width * (2.0 + 4 + 4 + 2),
           lambda: cuda.fused_add_rms_norm(x, res16, nw, eps), 0.0, T * width * 8.0)
    yield ("up projection with activation", lambda: cuda.gemm_gelu(x, w_up), *gemm_fb(ff, width),
           lambda: cuda.gemm_swiglu(x, w_gu), 4.0 * T * I * width, 2.0 * (2 * I * width + T * width + T * I))
    yield ("down projection", lambda: cuda.gemm(h_ff, w_dn), *gemm_fb(width, ff),
           lambda: cuda.gemm(h_i, w_dn2), *gemm_fb(width, I))
    if step == "decode":
        V = 128256
        w_head = rnd(V, width)
        yield ("logits (128256, soft cap, fp32)", lambda: cuda.gemm_softcap(x, w_head, 30.0), 2.0 * T * V * width,
               2.0 * (V * width + T * width) + 4.0 * T * V, lambda: cuda.gemm(x, w_head), *gemm_fb(V, width))


def bench_steps(width: int, heads: int, iters: int = 10) -> list:
    """Every kernel step of a layer beside the like step of the DeepSeek layer, with roofline fractions."""
    pk, tag = peaks()

    def frac(ms, flops, nbytes):
        floor = max(flops / pk["bf16_tflops"] / 1e9, nbytes / pk["hbm_gbs"] / 1e6)
        return floor / ms
    rows = []
    for step in STEPS:
        for what, fn, fl, by, fn2, fl2, by2 in _pairs(width, heads, step):
            ms, ms2 = time_fn(fn, iters), time_fn(fn2, iters)
            f, f2 = frac(ms, fl, by), frac(ms2, fl2, by2)
            rows.append({"op": what, "width": width, "heads": heads, "step": step, "us": round(ms * 1e3, 1),
                         "roofline_frac": round(f, 3), "neighbour_us": round(ms2 * 1e3, 1),
                         "neighbour_frac": round(f2, 3), "distance_ratio": round(f2 / f, 2), "peaks": tag})
        torch.cuda.empty_cache()
    return rows


def run(sizes: str, what: str = "layers,steps", iters: int = 10) -> list:
    from . import cuda
    rows = []
    for size in sizes.split(","):
        width, heads = (int(n) for n in size.split("x"))
        if "layers" in what:
            rows += bench_layers(width, heads, iters=iters)
        if "steps" in what:
            rows += bench_steps(width, heads, iters=iters)
    status = cuda.check_status()
    if status:
        raise RuntimeError(f"device status {status}")
    return rows
