"""Layer throughput of Zeganex beside a sliding-window mixture-of-experts decoder (the Qwen3-MoE classes) at equal size,
and the kernels of both.

    python bench.py --layer-bench zeganex [--layer-size 2048x16,4096x32]

Random weights; four layers (a window of 1024 tokens, four query heads per key head, 128-wide values, 32 experts of which a
token uses 4) without embedding and head run one prefill batch (four prompts of 2048 tokens) and one decode batch (64
requests behind 2047 tokens) through ``model.forward``, as one CUDA graph.  Differential layers have two 64-wide maps per
head, so that projections and cache are as large as the neighbour's; rotated layers have the output gate on top.  Experts
have as many parameters as the neighbour's gated ones.  CUDA events, L2 flushed before every timed launch, median; fractions
are of the measured peaks.
"""
from __future__ import annotations

import torch

from ..config import ModelConfig
from .bench_kernels import peaks, time_fn
from .bench_latent import BS, STEPS, build, step_meta
from .bench_linear import fill

D, TAPS, WINDOW = 128, 4, 1024
EXPERTS, TOP, FF, GATED_FF = 32, 4, 1152, 768


def zeganex_config(width: int, heads: int, kind: str, layers: int = 4) -> ModelConfig:
    mix = {"heads": heads, "kv_heads": heads // 4, "vdim": D, "conv": TAPS, "mask": {"size": WINDOW}}
    mixer = {"attention": dict(mix, dim=D // 2, scale=(D // 2) ** -0.5, diff=0.4),
             "attention_2": dict(mix, dim=D, scale=D ** -0.5, rot={"base": 10000.0, "dims": D // 2, "scaling": {
                 "factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}})}[kind]
    mlp = {"kind": "moe", "router": {"experts": EXPERTS, "top": TOP}, "expert": {"ff": FF}}
    return ModelConfig.from_layer_list({
        "architecture": "Zeganex", "width": width, "vocab": 1024, "norm": {"eps": 1e-6}, "residual_mult": 0.5,
        "embedding": {"bigram": {"buckets": 4099, "mul_prev": 29, "mul_cur": 13}},
        "layers": [{"type": kind, "mixer": mixer, "mlp": mlp}] * layers}, "zeganex-bench")


def neighbour_config(width: int, heads: int, layers: int = 4) -> ModelConfig:
    return ModelConfig(name="qwen3-moe-bench", architecture="qwen3_moe", num_layers=layers, hidden_size=width, num_q_heads=heads,
                       num_kv_heads=heads // 4, head_dim=D, sliding_window=WINDOW, num_experts=EXPERTS,
                       num_experts_per_tok=TOP, moe_intermediate_size=GATED_FF, vocab_size=1024, rms_norm_eps=1e-6)


def caches_of(model, blocks: int, reqs: int):
    if hasattr(model, "allocate_kv_caches"):
        caches = model.allocate_kv_caches(blocks, BS, torch.bfloat16, "cuda", reqs)
    else:
        caches = [torch.zeros(model.kv_cache_shape(blocks, BS), dtype=torch.bfloat16, device="cuda") for _ in model.layers]
    fill(caches)
    return caches


def bench_layers(width: int, heads: int, iters: int = 10) -> list:
    """Milliseconds and tokens per second of four layers of each model."""
    rows = []
    for name, cfg in (("zeganex: differential attention", zeganex_config(width, heads, "attention")),
                      ("zeganex: rotated attention with gate", zeganex_config(width, heads, "attention_2")),
                      ("qwen3_moe with a window", neighbour_config(width, heads))):
        model = build(cfg)
        for step, (q_len, ctx, reqs) in STEPS.items():
            meta, blocks = step_meta(q_len, ctx, reqs)
            caches = caches_of(model, blocks, reqs)
            x = torch.randn(reqs * q_len, width, device="cuda")
            x = x if cfg.architecture == "zeganex" else x.bfloat16()
            ms = time_fn(lambda: model.forward(None, meta, caches, hidden=x), iters)
            rows.append({"op": "layers", "model": name, "width": width, "heads": heads, "layers": 4, "step": step,
                         "tokens": reqs * q_len, "context": q_len + ctx, "ms": round(ms, 4),
                         "tok_s_per_layer": round(reqs * q_len * 4 / ms * 1e3),
                         "weight_mb": round(sum(l.mlp.weight_bytes() + sum(x.weight_bytes() for x in l.self_attn.linears())
                                                for l in model.layers) / 1e6, 1)})
            del caches
        del model
        torch.cuda.empty_cache()
    return rows


def _pairs(width: int, heads: int, step: str):
    """(what, step kernel of Zeganex, its flops, bytes; like kernel of the neighbour, flops, bytes)."""
    from . import cuda
    q_len, ctx, reqs = STEPS[step]
    T, H, G, eps = q_len * reqs, heads, heads // 4, 1e-6
    rnd = lambda *s: (torch.randn(*s, device="cuda") * 0.1).bfloat16()                  # noqa: E731
    meta, blocks = step_meta(q_len, ctx, reqs)
    dm, gm, nm = (build(c) for c in (zeganex_config(width, H, "attention", 1), zeganex_config(width, H, "attention_2", 1),
                                     neighbour_config(width, H, 1)))
    caches = [caches_of(m, blocks, reqs)[0] for m in (dm, gm, nm)]
    da, ga, na = dm.layers[0].self_attn, gm.layers[0].self_attn, nm.layers[0].self_attn
    x = rnd(T, width)
    gemm_fb = lambda n, k: (2.0 * T * n * k, 2.0 * (n * k + T * k + T * n))             # noqa: E731
    n_qkv = (H + 2 * G) * D
    yield "differential: projection", lambda: da.inp(x), *gemm_fb(n_qkv, width), lambda: na.qkv(x), *gemm_fb(n_qkv, width)
    yield "gated: projection", lambda: ga.inp(x), *gemm_fb(n_qkv + H * D, width), lambda: na.qkv(x), *gemm_fb(n_qkv, width)
    # ---- between projection and attention
    d_row, g_row, n_row = da.inp(x), ga.inp(x), na.qkv(x)
    ring = 2.0 * reqs * TAPS * n_qkv * (2 if q_len == 1 else 1)
    prep = 2.0 * T * 2 * n_qkv
    rope = lambda: cuda.rope_and_cache(n_row, meta.positions, na.attn.inv_freq, caches[2], meta.slot_mapping, H, G, D)  # noqa: E731
    yield "differential: convolutions, cache write (neighbour: rotation)", lambda: cuda.conv_and_cache(
        da.plan, d_row, caches[0][1], caches[0][0], meta), 0.0, prep + ring, rope, 0.0, prep
    yield "gated: convolutions, rotation, cache write (neighbour: rotation)", lambda: cuda.conv_and_cache(
        ga.plan, g_row, caches[1][1], caches[1][0], meta), 0.0, prep + ring, rope, 0.0, prep
    # ---- attention with what follows the softmax
    seen = [min(p + 1, WINDOW) for p in range(ctx, ctx + q_len)]
    keys, kv_rows = reqs * float(sum(seen)), reqs * min(q_len + ctx, WINDOW + q_len - 1)
    kv = 2.0 * kv_rows * 2 * G * D
    qd, qg = cuda.conv_and_cache(da.plan, d_row, caches[0][1], caches[0][0], meta), rnd(T, H, D)
    yield "differential: attention, difference of the maps, norm", lambda: da.attend(qd, d_row, caches[0][1], meta), \
        keys * H * 2 * (2 * 64 + 2 * D), kv + 2.0 * 2 * T * H * D, lambda: cuda.paged_attention(
            qg, caches[2], meta, D ** -0.5, sliding_window=WINDOW), keys * H * 4 * D, kv + 2.0 * 2 * T * H * D
    yield "gated: attention, gate", lambda: ga.attend(qg, g_row, caches[1][1], meta), keys * H * 4 * D, \
        kv + 2.0 * 3 * T * H * D, lambda: cuda.paged_attention(
            qg, caches[2], meta, D ** -0.5, sliding_window=WINDOW), keys * H * 4 * D, kv + 2.0 * 2 * T * H * D
    y = rnd(T, H * D)
    yield "output projection", lambda: ga.o(y), *gemm_fb(width, H * D), lambda: na.o(y), *gemm_fb(width, H * D)
    # ---- around the sublayers
    res, res16, nw = torch.randn(T, width, device="cuda"), rnd(T, width), rnd(width)
    yield "both norms and residual (32-bit stream)", lambda: cuda.add_rms_norm(x, res, nw, eps, post=nw, mult=0.5), 0.0, \
        T * width * 12.0, lambda: cuda.fused_add_rms_norm(x, res16, nw, eps), 0.0, T * width * 8.0
    dx, nx = dm.layers[0].mlp.experts, nm.layers[0].mlp.experts
    route = (2.0 * T * EXPERTS * width, 2.0 * (EXPERTS * width + T * width))
    yield "router", lambda: dx.route(x), *route, lambda: nx.route(x), *route
    ids, wt = dx.route(x)
    used = min(EXPERTS, T * TOP)
    fl = 4.0 * T * TOP * FF * width
    by = 2.0 * (used * 2 * FF * width + 2 * T * width)
    yield "experts", lambda: cuda.moe_experts(x, dx.w13, dx.w2, ids, wt, act="relu2"), fl, by, \
        lambda: cuda.moe_experts(x, nx.w13, nx.w2, ids, wt), fl, by
    table, pairs = rnd(8192, width), rnd(4100, width)
    tok = torch.randint(0, 8192, (T,), device="cuda", dtype=torch.int32)
    src, last = torch.full((T,), -1, dtype=torch.int32, device="cuda"), torch.zeros(reqs, dtype=torch.int32, device="cuda")
    yield "embedding", lambda: cuda.embedding_pairs(tok, tok, table, pairs, (4099, 29, 13), src, last, last.clone()), 0.0, \
        T * width * 8.0, lambda: cuda.embedding(tok, table), 0.0, T * width * 4.0
    if step == "decode":
        V = 128256
        w_head = rnd(V, width)
        yield "logits (128256, fp32)", lambda: cuda.gemm_softcap(x, w_head), 2.0 * T * V * width, \
            2.0 * (V * width + T * width) + 4.0 * T * V, lambda: cuda.gemm(x, w_head), *gemm_fb(V, width)


def bench_steps(width: int, heads: int, iters: int = 10) -> list:
    """Every kernel step of a layer beside the like step of the neighbour, with roofline fractions."""
    pk, tag = peaks()

    def frac(ms, flops, nbytes):
        return max(flops / pk["bf16_tflops"] / 1e9, nbytes / pk["hbm_gbs"] / 1e6) / ms
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
            rows += bench_layers(width, heads, iters)
        if "steps" in what:
            rows += bench_steps(width, heads, iters)
    status = cuda.check_status()
    if status:
        raise RuntimeError(f"device status {status}")
    return rows
