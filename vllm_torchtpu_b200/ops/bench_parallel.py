"""Layer throughput of Vipolix beside the framework's closest layers (Zeganex' convolved attention with experts, Popanex'
channel-wise delta rule) at equal size, and the kernels of all.

    python bench.py --layer-bench vipolix [--layer-size 2048x16,4096x32]

Random weights; four layers without embedding and head run one prefill batch (four prompts of 2048 tokens) and one decode
batch (64 requests behind 2047 tokens) through ``model.forward``, as one CUDA graph.  Parallel layers: H query heads of 128
dimensions, four per key head, chunks of 1024 tokens, beside H / 2 heads of 128 x 128 state; linear layers: H heads of
128 x 128.  32 clamped experts in 8 groups of which a token uses 4, and a shared one of the same width; token input of 256.
Zeganex: a window of 1024, the output gate, 32 ungated experts with as many parameters.  Popanex: H heads of 128 x 128, a
dense feed-forward as wide as the experts a token uses.  CUDA events, L2 flushed before every timed launch, median;
fractions are of the measured peaks.
"""
from __future__ import annotations

import torch

from ..config import ModelConfig
from .bench_kernels import peaks, time_fn
from .bench_latent import BS, STEPS, build, step_meta
from .bench_linear import fill
from .bench_window import zeganex_config

D, TAPS, CHUNK, RANK, SIDE = 128, 4, 1024, 64, 256
EXPERTS, TOP, FF = 32, 4, 768


def vipolix_config(width: int, heads: int, kind: str, layers: int = 4) -> ModelConfig:
    left = {"heads": heads, "kv_heads": heads // 4, "dim": D, "vdim": D, "conv": TAPS, "mask": {"size": CHUNK},
            "scale": D ** -0.5, "rot": {"base": 10000.0, "dims": D // 2}}
    mixer = {"parallel": {"left": left, "right": {"heads": heads // 2, "dim": D, "decay_rank": RANK}, "left_scale": 0.7,
                          "right_scale": 0.7},
             "gla": {"heads": heads, "dim": D, "vdim": D, "tau": 16.0, "decay_rank": RANK}}[kind]
    mlp = {"kind": "moe", "expert": {"ff": FF, "limit": 7.0}, "shared": {"ff": FF, "limit": 7.0},
           "router": {"experts": EXPERTS, "top": TOP, "scale": 2.0, "groups": {"count": 8, "keep": 4}}}
    return ModelConfig.from_layer_list({
        "architecture": "Vipolix", "width": width, "vocab": 1024, "norm": {"eps": 1e-6}, "token_side": {"dim": SIDE},
        "layers": [{"type": kind, "mixer": mixer, "mlp": mlp}] * layers}, "vipolix-bench")


def popanex_config(width: int, heads: int, layers: int = 4) -> ModelConfig:
    mixer = {"heads": heads, "kv_heads": heads, "dim": D, "vdim": D, "conv": TAPS, "gate_rank": RANK}
    mlp = {"kind": "dense", "ff": (TOP + 1) * FF}
    return ModelConfig.from_layer_list({
        "architecture": "Popanex", "width": width, "vocab": 1024, "norm": {"eps": 1e-6},
        "layers": [{"type": "channel_delta", "mixer": mixer, "mlp": mlp}] * layers}, "popanex-bench")


def caches_of(model, blocks: int, reqs: int) -> list:
    caches = model.allocate_kv_caches(blocks, BS, torch.bfloat16, "cuda", reqs)

    def tensors(c):
        return [c] if torch.is_tensor(c) else [t for x in c for t in tensors(x)]
    fill(tensors(caches))
    return caches


def bench_layers(width: int, heads: int, iters: int = 10) -> list:
    """Milliseconds and tokens per second of four layers of each model."""
    rows = []
    for name, cfg in (("vipolix: attention beside a delta rule", vipolix_config(width, heads, "parallel")),
                      ("vipolix: gated linear attention", vipolix_config(width, heads, "gla")),
                      ("zeganex: rotated attention with gate", zeganex_config(width, heads, "attention_2")),
                      ("popanex: channel delta", popanex_config(width, heads))):
        model = build(cfg)
        for step, (q_len, ctx, reqs) in STEPS.items():
            meta, blocks = step_meta(q_len, ctx, reqs)
            caches = caches_of(model, blocks, reqs)
            T = reqs * q_len
            x = torch.randn(T, width, device="cuda")
            ids = torch.randint(0, cfg.vocab_size, (T,), device="cuda", dtype=torch.int32)
            ms = time_fn(lambda: model.forward(ids, meta, caches, hidden=x), iters)
            rows.append({"op": "layers", "model": name, "width": width, "heads": heads, "layers": 4, "step": step,
                         "tokens": T, "context": q_len + ctx, "ms": round(ms, 4), "tok_s_per_layer": round(T * 4 / ms * 1e3),
                         "weight_mb": round(sum(l.mlp.weight_bytes() + l.self_attn.weight_bytes() for l in model.layers) / 1e6, 1)})
            del caches
        del model
        torch.cuda.empty_cache()
    return rows


def _pairs(width: int, heads: int, step: str):
    """(what, step kernel of Vipolix, its flops, bytes; like kernel of a neighbour, flops, bytes)."""
    from . import cuda
    q_len, ctx, reqs = STEPS[step]
    T, H, eps = q_len * reqs, heads, 1e-6
    G, R = H // 4, H // 2
    rnd = lambda *s: (torch.randn(*s, device="cuda") * 0.1).bfloat16()                  # noqa: E731
    meta, blocks = step_meta(q_len, ctx, reqs)
    pm, gm, zm, dm, d2 = (build(c) for c in (vipolix_config(width, H, "parallel", 1), vipolix_config(width, H, "gla", 1),
                                             zeganex_config(width, H, "attention_2", 1), popanex_config(width, H, 1),
                                             popanex_config(width, R, 1)))
    pc, gc, zc, dc, d2c = (caches_of(m, blocks, reqs)[0] for m in (pm, gm, zm, dm, d2))
    pa, ga, za, da, ha = (m.layers[0].self_attn for m in (pm, gm, zm, dm, d2))
    x = rnd(T, width)
    gemm_fb = lambda n, k: (2.0 * T * n * k, 2.0 * (n * k + T * k + T * n))             # noqa: E731
    add = lambda *p: tuple(sum(v) for v in zip(*p))                                     # noqa: E731
    # ---- projections
    n_qkv = (H + 2 * G) * D
    n_par = n_qkv + 5 * R * D + RANK
    yield "parallel: projection of both mixers", lambda: pa.inp(x), *gemm_fb(n_par, width), lambda: za.inp(x), \
        *gemm_fb(n_qkv + H * D, width)
    row, z_row = pa.inp(x), za.inp(x)
    rank_row = rnd(T, RANK)
    yield "parallel: tanh and second decay projection (neighbour: projection alone)", lambda: pa.right.decays(row), \
        *gemm_fb(R * D, RANK), lambda: ha.a2(rank_row), *gemm_fb(R * D, RANK)
    fb_delta = add(gemm_fb(3 * H * D + 2 * RANK + H, width), gemm_fb(H * D, RANK), gemm_fb(H * D, RANK))
    yield "linear: projections", lambda: ga.project(x), *add(gemm_fb(4 * H * D + RANK, width), gemm_fb(H * D, RANK)), \
        lambda: da.project(x), *fb_delta
    # ---- attention
    ring = 2.0 * reqs * TAPS * n_qkv * (2 if q_len == 1 else 1)
    prep = 2.0 * T * 2 * n_qkv
    shift_state, (c_ring, pages, state) = pc
    yield "parallel: convolutions, rotation, cache write", lambda: cuda.conv_and_cache(pa.left.plan, row, pages, c_ring, meta), \
        0.0, prep + ring, lambda: cuda.conv_and_cache(za.plan, z_row, zc[1], zc[0], meta), 0.0, prep + ring
    q = rnd(T, H, D)
    z = torch.zeros(T, pa.o.in_features, dtype=torch.bfloat16, device="cuda")

    def attn(seen, span):
        return reqs * float(sum(seen)) * H * 4 * D, 2.0 * reqs * span * 2 * G * D + 2.0 * 2 * T * H * D
    pos = range(ctx, ctx + q_len)
    a_par = attn([p % CHUNK + 1 for p in pos], q_len + min(ctx, ctx % CHUNK))
    a_win = attn([min(p + 1, CHUNK) for p in pos], min(q_len + ctx, CHUNK + q_len - 1))
    yield "parallel: attention in chunks with sinks (neighbour: window)", lambda: pa.left.attend(q, row, pages, meta, z[:, :H * D]), \
        *a_par, lambda: cuda.paged_attention(q, zc[1], meta, D ** -0.5, sliding_window=CHUNK), *a_win
    # ---- recurrences
    p_in, g_in, d_in, h_in = (row, pa.right.decays(row)), ga.project(x), da.project(x), ha.project(x)

    def rec(h, products, columns):
        return 2.0 * products * T * h * D * D, 2.0 * T * columns * h * D + 2.0 * 4 * reqs * h * D * D
    yield "parallel: removal recurrence, norm, gate", lambda: pa.right.recur(p_in, meta, (state,), z[:, H * D:H * D + R * D]), \
        *rec(R, 4, 7), lambda: ha.recur(h_in, meta, d2c), *rec(R, 3, 6)
    yield "linear: recurrence, norm, gate", lambda: ga.recur(g_in, meta, gc[1]), *rec(H, 2, 6), \
        lambda: da.recur(d_in, meta, dc), *rec(H, 3, 6)
    y, y2 = rnd(T, H * D), rnd(T, pa.o.in_features)
    yield "parallel: output projection of both mixers", lambda: pa.o(y2), *gemm_fb(width, pa.o.in_features), lambda: za.o(y), \
        *gemm_fb(width, H * D)
    # ---- around the sublayers
    res, nw = torch.randn(T, width, device="cuda"), rnd(width)
    layer = pm.layers[0]
    yield "norm of the token input, sum, norm, shift (neighbour: both norms)", lambda: cuda.add_rms_norm_shift(
        x, res, nw, eps, 1.0, nw, shift_state, meta, nw), 0.0, T * width * 12.0 + 2.0 * reqs * width * 4, \
        lambda: cuda.add_rms_norm(x, res, nw, eps, post=nw, mult=0.5), 0.0, T * width * 12.0
    yield "sum and norm", lambda: cuda.add_rms_norm(x, res, nw, eps, 1.0, mult=0.7), 0.0, T * width * 12.0, \
        lambda: cuda.add_rms_norm(x, res, nw, eps, post=nw, mult=0.5), 0.0, T * width * 12.0
    block, zx = layer.mlp, zm.layers[0].mlp.experts
    px = block.experts
    route = (2.0 * T * EXPERTS * width, 2.0 * (EXPERTS * width + T * width))
    yield "router", lambda: px.route(x), *route, lambda: zx.route(x), *route
    ids, wt = px.route(x)
    z_ids, z_wt = zx.route(x)
    used, zff = min(EXPERTS, T * TOP), zx.intermediate_size
    out = 2.0 * 2 * T * width
    yield "experts (neighbour: ungated)", lambda: cuda.moe_experts(x, px.w13, px.w2, ids, wt, act=px.activation), \
        6.0 * T * TOP * FF * width, 2.0 * used * 3 * FF * width + out, lambda: cuda.moe_experts(
            x, zx.w13, zx.w2, z_ids, z_wt, act="relu2"), 4.0 * T * TOP * zff * width, 2.0 * used * 2 * zff * width + out
    yield "experts, shared expert, sum on the stream (neighbour: experts, sum and norm)", lambda: block.forward_add(x, res), \
        6.0 * T * (TOP + 1) * FF * width, 2.0 * (used + 1) * 3 * FF * width + 12.0 * T * width, lambda: cuda.add_rms_norm(
            zx.forward(x), res, nw, eps), 4.0 * T * TOP * zff * width, 2.0 * used * 2 * zff * width + 14.0 * T * width
    table, tok = rnd(1024, SIDE), torch.randint(0, 1024, (T,), device="cuda", dtype=torch.int32)
    side = add(gemm_fb(SIDE, width), gemm_fb(width, SIDE))
    yield "token input (neighbour: two plain products)", lambda: layer.side.forward(x, table, tok), *side, \
        lambda: cuda.gemm(cuda.gemm(x, layer.side.gate.weight), layer.side.proj.weight), *side
    if step == "decode":
        V = 128256
        w_head = rnd(V, width)
        yield "logits (128256, fp32)", lambda: cuda.gemm_softcap(x, w_head), 2.0 * T * V * width, \
            2.0 * (V * width + T * width) + 4.0 * T * V, lambda: cuda.gemm(x, w_head), *gemm_fb(V, width)


def bench_steps(width: int, heads: int, iters: int = 10) -> list:
    """Every kernel step of a layer beside the like step of a neighbour, with roofline fractions."""
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
