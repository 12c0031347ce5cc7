"""Layer throughput of Popanex beside the Kimi-Linear hybrid at equal size, and the kernels of both.

    python bench.py --layer-bench popanex [--layer-size 2048x16,4096x32]

Random weights; four layers (three with a carried state, one of softmax attention; 128-wide heads, gated feed-forward of
8/3 x width) without embedding and head run one prefill batch (four prompts of 2048 tokens) and one decode batch (64
requests behind 2047 tokens) through ``model.forward``, as one CUDA graph.  The neighbour's layers are Kimi Delta
Attention and grouped-query attention.  CUDA events, L2 flushed before every timed launch, median; fractions are of the
measured peaks.
"""
from __future__ import annotations

import torch

from ..config import ModelConfig
from .bench_kernels import peaks, time_fn
from .bench_latent import BS, STEPS, build, step_meta

D = 128
TAPS = 4


def feed_forward(width: int) -> int:
    return width * 8 // 3 // 128 * 128


def popanex_config(width: int, heads: int, kind: str) -> ModelConfig:
    att = {"heads": heads, "kv_heads": heads // 4, "dim": D, "vdim": D, "scale": D ** -0.5,
           "q_temp": {"coef": 0.1, "every": 1024}}
    rec = {"channel_delta": {"heads": heads, "kv_heads": heads, "dim": D, "vdim": D, "conv": TAPS},
           "retention": {"heads": heads, "dim": D, "vdim": D, "rot": {"base": 10000.0, "dims": D},
                         "decay": [1.0 - 2.0 ** (-5 - 4 * h / heads) for h in range(heads)]}}[kind]
    mlp = {"kind": "dense", "ff": feed_forward(width)}
    layers = [{"type": kind, "mixer": rec, "mlp": mlp}] * 3 + [{"type": "attention", "mixer": att, "mlp": mlp}]
    return ModelConfig.from_layer_list({"architecture": "Popanex", "width": width, "vocab": 1024, "norm": {"eps": 1e-6},
                                        "logit_scale": 0.5, "layers": layers}, "popanex-bench")


def kimi_config(width: int, heads: int) -> ModelConfig:
    return ModelConfig(name="kimi-bench", architecture="kimi_linear", num_layers=4, full_attention_interval=4,
                       hidden_size=width, num_q_heads=heads, num_kv_heads=heads // 4, head_dim=D,
                       intermediate_size=feed_forward(width), vocab_size=1024, gdn_num_k_heads=heads,
                       gdn_num_v_heads=heads, gdn_head_k_dim=D, gdn_head_v_dim=D, gdn_conv_kernel=TAPS, kda_gate_rank=D)


def fill(caches) -> None:
    for c in caches:
        for t in c if isinstance(c, tuple) else (c,):
            t.normal_(0, 0.3)


def bench_layers(width: int, heads: int, iters: int = 10) -> list:
    """Milliseconds and tokens per second of four layers of each model."""
    rows = []
    for name, cfg in (("popanex: 3 channel delta, 1 attention", popanex_config(width, heads, "channel_delta")),
                      ("popanex: 3 retention, 1 attention", popanex_config(width, heads, "retention")),
                      ("kimi_linear: 3 KDA, 1 attention", kimi_config(width, heads))):
        model = build(cfg)
        for step, (q_len, ctx, reqs) in STEPS.items():
            meta, blocks = step_meta(q_len, ctx, reqs)
            caches = model.allocate_kv_caches(blocks, BS, torch.bfloat16, "cuda", reqs)
            fill(caches)
            x = torch.randn(reqs * q_len, width, device="cuda").bfloat16()
            ms = time_fn(lambda: model.forward(None, meta, caches, hidden=x), iters)
            rows.append({"op": "layers", "model": name, "width": width, "heads": heads, "layers": 4, "step": step,
                         "tokens": reqs * q_len, "context": q_len + ctx, "ms": round(ms, 4),
                         "tok_s_per_layer": round(reqs * q_len * 4 / ms * 1e3),
                         "weight_mb": round((model.weight_bytes() - 4 * 1024 * width) / 1e6, 1)})
            del caches
        del model
        torch.cuda.empty_cache()
    return rows


def _pairs(width: int, heads: int, step: str):
    """(what, step kernel of Popanex, its flops, bytes; like kernel of the neighbour, flops, bytes)."""
    from . import cuda, ref
    q_len, ctx, reqs = STEPS[step]
    T, H, eps = q_len * reqs, heads, 1e-6
    rnd = lambda *s: (torch.randn(*s, device="cuda") * 0.1).bfloat16()                  # noqa: E731
    meta, blocks = step_meta(q_len, ctx, reqs)
    pop, ret, kimi = (build(c) for c in (popanex_config(width, H, "channel_delta"), popanex_config(width, H, "retention"),
                                         kimi_config(width, H)))
    caches = [m.allocate_kv_caches(blocks, BS, torch.bfloat16, "cuda", reqs) for m in (pop, ret, kimi)]
    for c in caches:
        fill(c)
    dl, rt, kd = pop.layers[0].self_attn, ret.layers[0].self_attn, kimi.layers[0].self_attn
    at, ka = pop.layers[3].self_attn, kimi.layers[3].self_attn
    x = rnd(T, width)
    gemm_fb = lambda n, k: (2.0 * T * n * k, 2.0 * (n * k + T * k + T * n))             # noqa: E731
    add = lambda *p: tuple(sum(v) for v in zip(*p))                                     # noqa: E731

    # ---- projections of the recurrent layers
    kda_in = lambda: (kd.in_qkv(x), kd.f_b(kd.f_a(x)), kd.b_proj(x), kd.g_b(kd.g_a(x)))  # noqa: E731
    fb_delta = add(gemm_fb(3 * H * D + 2 * D + H, width), gemm_fb(H * D, D), gemm_fb(H * D, D))
    fb_kda = add(gemm_fb(3 * H * D, width), gemm_fb(D, width), gemm_fb(D, width), gemm_fb(H, width), gemm_fb(H * D, D),
                 gemm_fb(H * D, D))
    yield "channel delta: projections", lambda: dl.project(x), *fb_delta, kda_in, *fb_kda
    yield "retention: projections", lambda: rt.project(x), *gemm_fb(4 * H * D, width), kda_in, *fb_kda
    # ---- convolution to output gate
    d_in, r_in = dl.project(x), rt.project(x)
    mixed, a, b, gate = kd.in_qkv(x), kd.f_b(kd.f_a(x)).reshape(T, H, D), kd.b_proj(x), kd.g_b(kd.g_a(x)).reshape(T, H, D)
    state = 2.0 * 4 * reqs * H * D * D
    rec_fl = 6.0 * T * H * D * D                      # S^T k, the update and S^T q
    delta_by = 2.0 * T * (6 * H * D + H) + state      # q, k, v, decays, gate, output
    ret_by = 2.0 * T * 5 * H * D + state

    def kda():
        o = kd.recur((mixed, a, b), meta, caches[2][0])
        o = cuda.rms_norm(o.reshape(T * H, D), kd.norm_w, eps).reshape(T, H, D)
        return (o.float() * torch.sigmoid(gate.float())).to(x.dtype)
    yield "channel delta: convolution, recurrence, norm, gate", lambda: dl.recur(d_in, meta, caches[0][0]), rec_fl, \
        delta_by, kda, rec_fl, delta_by
    yield "retention: rotation, recurrence, norm, gate", lambda: rt.recur(r_in, meta, caches[1][0]), rec_fl * 2 / 3, \
        ret_by, kda, rec_fl, delta_by
    y = rnd(T, H * D)
    yield "recurrent layers: output projection", lambda: dl.o(y), *gemm_fb(width, H * D), lambda: kd.out(y), \
        *gemm_fb(width, H * D)
    # ---- attention
    kv = H // 4
    n_qkv = (H + 2 * kv) * D
    yield "attention: projection", lambda: at.inp(x), *gemm_fb(n_qkv, width), lambda: ka.qkv(x), *gemm_fb(n_qkv, width)
    row, s = at.inp(x), at.spec
    inv = ref.rope_inv_freq(D, 10000.0, None).cuda()
    prep_b = 2.0 * T * 2 * n_qkv
    yield "attention: norms, temperature, cache write (neighbour: rotation)", lambda: cuda.norm_and_cache(
        row, meta.positions, caches[0][3], meta.slot_mapping, H, kv, D, D, at.q_norm, at.k_norm, eps,
        (s.q_temp.coef, s.q_temp.every)), 0.0, prep_b, lambda: cuda.rope_and_cache(
            row, meta.positions, inv, caches[2][3], meta.slot_mapping, H, kv, D), 0.0, prep_b
    q = rnd(T, H, D)
    keys = reqs * (q_len * ctx + q_len * (q_len + 1) / 2)
    attn = (4.0 * keys * H * D, 2.0 * (reqs * (q_len + ctx) * 2 * kv * D + 2 * T * H * D))
    yield "attention: paged attention with sinks", lambda: cuda.paged_attention(
        q, caches[0][3], meta, s.scale, sinks=at.sinks), *attn, lambda: cuda.paged_attention(
            q, caches[2][3], meta, s.scale), *attn
    # ---- around the sublayers
    res, res16, nw = torch.randn(T, width, device="cuda"), rnd(T, width), rnd(width)
    yield "norm and residual (32-bit stream)", lambda: cuda.add_rms_norm(x, res, nw, eps, 1.0), 0.0, T * width * 12.0, \
        lambda: cuda.fused_add_rms_norm(x, res16, nw, eps), 0.0, T * width * 8.0
    ff = feed_forward(width)
    w_gu, w_dn, h_ff = rnd(2 * ff, width), rnd(width, ff), rnd(T, ff)
    gu = (4.0 * T * ff * width, 2.0 * (2 * ff * width + T * width + T * ff))
    yield "gate and up projection with activation", lambda: cuda.gemm_gated(x, w_gu, "gelu_tanh"), *gu, \
        lambda: cuda.gemm_swiglu(x, w_gu), *gu
    yield "down projection", lambda: cuda.gemm(h_ff, w_dn), *gemm_fb(width, ff), lambda: cuda.gemm(h_ff, w_dn), \
        *gemm_fb(width, ff)
    if step == "decode":
        V = 128256
        w_head = rnd(V, width)
        yield "logits (128256, factor, fp32)", lambda: cuda.gemm_softcap(x, w_head, 0.0, 0.5), 2.0 * T * V * width, \
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
