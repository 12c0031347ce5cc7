"""Popanex (softmax attention, retention and a channel-wise gated delta rule, chosen per layer) against the plain
statement in ``plain_popanex.py``: every mechanism alone, then the model through the engine's scheduler, caches and
kernels."""
import copy
import json
import math
import os
import subprocess

import numpy as np
import plain_popanex as plain
import pytest
import torch
from test_mazivik import BF16, DEV_DTYPE, DEVS, F32, ROOT, _close, _rand, logit_error, portions, replay_logits, tokens_of

from vllm_torchtpu_b200 import SamplingParams, ops
from vllm_torchtpu_b200.config import CacheConfig, EngineConfig, ModelConfig, ParallelConfig, model_preset
from vllm_torchtpu_b200.entrypoints.trace_replay import make_replay
from vllm_torchtpu_b200.ops import linear_attention as la
from vllm_torchtpu_b200.runner.attn_metadata import AttentionMetadata


LIMIT = {"float32": 2e-5, "bfloat16": 5e-2}


def assert_like(got, want, dtype, what="", factor=1.0):
    """Every position in 32-bit.  In bf16 nine of ten: a head's output is divided by its root mean square, so that where
    q . k happens to vanish (the first tokens above all) rounding decides the direction."""
    d = got.double() - want.double()
    e = (d - d.mean(-1, keepdim=True)).pow(2).mean(-1).sqrt() / want.double().pow(2).mean().sqrt()
    if dtype == "float32":
        assert e.max() < LIMIT[dtype] * factor, (what, e.max())
    else:
        assert e.sort().values[int(0.9 * (len(e) - 1))] < LIMIT[dtype] * factor and e.max() < 0.5, (what, e)


# ------------------------------------------------------------------------------------------------- configurations
def attention(heads=4, kv_heads=2, dim=20, vdim=28, scale=0.3, coef=0.4, every=24):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                                           "q_temp": {"coef": coef, "every": every}}}


def retention(heads=3, dim=24, vdim=40, dims=16, base=700.0, decay=None):
    decay = decay or [1.0 - 0.2 * 0.4 ** i for i in range(heads)]
    return {"type": "retention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "rot": {"base": base, "dims": dims},
                                           "decay": decay}}


def delta(heads=4, kv_heads=2, dim=16, vdim=24, conv=3, rank=12):
    """``rank`` is no entry of the configuration: the tensors' shapes give it."""
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim,
                                               "conv": conv}, "rank": rank}


def config(layers, width=72, vocab=211, eps=3e-6, scale=1.7):
    """layers: (mixer entry, feed-forward width or 0, index of the layer whose weights it uses or None)."""
    out = []
    for layer, ff, src in layers:
        e = dict(copy.deepcopy(layer), mlp={"kind": "dense", "ff": ff} if ff else None)
        if src is not None:
            e["weights_of"] = src
        out.append(e)
    return {"architecture": "Popanex", "width": width, "vocab": vocab, "norm": {"eps": eps}, "logit_scale": scale,
            "layers": out}


MIXED = config([(delta(), 88, None), (attention(), 0, None), (retention(), 56, None), (retention(), 56, 2),
                (delta(heads=3, kv_heads=3, dim=24, vdim=16, conv=4, rank=7), 0, None), (attention(), 0, 1)])
MODELS = {
    "mixed": MIXED,
    "all_sizes_odd": config([(attention(heads=3, kv_heads=1, dim=7, vdim=5), 13, None),
                             (delta(heads=2, kv_heads=1, dim=9, vdim=11, conv=2, rank=3), 0, None),
                             (retention(heads=1, dim=10, vdim=3, dims=6), 9, None)], width=21, vocab=37, scale=0.3),
    "recurrent_only": config([(retention(heads=2, dim=32, vdim=64, dims=32), 0, None),
                              (delta(heads=2, kv_heads=2, dim=40, vdim=72, conv=6, rank=24), 64, None)], width=80),
    "attention_only": config([(attention(heads=8, kv_heads=8, dim=64, vdim=64, scale=0.05, coef=1.5, every=7), 0, None),
                              (attention(heads=18, kv_heads=1, dim=36, vdim=52, scale=0.08, every=1, coef=0.1), 40, None)], width=96),
    "wide": config([(delta(heads=8, kv_heads=4, dim=64, vdim=128, conv=4, rank=32), 320, None),
                    (attention(heads=16, kv_heads=4, dim=128, vdim=128, scale=0.05, every=40), 448, None),
                    (retention(heads=4, dim=128, vdim=128, dims=64), 0, None),
                    (attention(heads=4, kv_heads=2, dim=160, vdim=144, scale=0.05), 0, None)], width=256, vocab=1000),
}


def random_model(cfg, seed=0, gain=1.0):
    """Weights of ``cfg`` (bfloat16), scaled so that activations stay of order one."""
    g = torch.Generator().manual_seed(seed)

    def rnd(*s, scale=1.0, mean=0.0):
        return (mean + torch.randn(*s, generator=g) * scale).bfloat16()

    def mat(o, i):
        return rnd(o, i, scale=gain / math.sqrt(i))
    W = cfg["width"]
    w = {"embed": rnd(cfg["vocab"], W), "final.norm": rnd(W, scale=0.3), "head": mat(cfg["vocab"], W)}
    for i, layer in enumerate(cfg["layers"]):
        if "weights_of" in layer:
            continue
        m, p = layer["mixer"], f"l{i}.mix."
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        G = m.get("kv_heads", H)
        w[f"l{i}.norm1"] = rnd(W, scale=0.3)
        w[p + "q"], w[p + "k"] = mat(H * d if layer["type"] == "attention" else G * d, W), mat(G * d, W)
        w[p + "v"] = mat(G * dv if layer["type"] == "attention" else H * dv, W)
        w[p + "o"] = mat(W, H * dv)
        if layer["type"] == "attention":
            w[p + "q.norm"], w[p + "k.norm"] = rnd(H * d, mean=1.5, scale=0.3), rnd(G * d, mean=1.0, scale=0.3)
            w[p + "sink"] = rnd(H, scale=2.0)
        elif layer["type"] == "retention":
            w[p + "g"] = mat(H * dv, W)
        else:
            r = layer["rank"]
            for n, c in (("q", G * d), ("k", G * d), ("v", H * dv)):
                w[p + n + ".conv"] = rnd(c, m["conv"], scale=0.7)
            w[p + "b"], w[p + "A_log"], w[p + "dt_bias"] = mat(H, W), rnd(H, scale=1.5), rnd(H * d, mean=-2.0, scale=1.5)
            w[p + "a1"], w[p + "a2"], w[p + "g1"], w[p + "g2"] = mat(r, W), mat(H * d, r), mat(r + 1, W), mat(H * dv, r + 1)
            w[p + "norm"] = rnd(dv, mean=1.0, scale=0.3)
        if layer["mlp"]:
            F = layer["mlp"]["ff"]
            w[f"l{i}.norm2"] = rnd(W, scale=0.3)
            w[f"l{i}.mlp.gate"], w[f"l{i}.mlp.up"], w[f"l{i}.mlp.down"] = mat(F, W), mat(F, W), mat(W, F)
    return w


def write_model(path, cfg, seed=0, gain=1.0, edit=None):
    from safetensors.torch import save_file
    w = random_model(cfg, seed, gain)
    if edit:
        edit(w)
    os.makedirs(path, exist_ok=True)
    save_file({k: v.contiguous() for k, v in w.items()}, os.path.join(path, "model.safetensors"))
    shown = copy.deepcopy(cfg)
    for layer in shown["layers"]:
        layer.pop("rank", None)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(shown, f)
    return w


# ------------------------------------------------------------------------------------------------- mechanisms
@pytest.mark.parametrize("dev,dtype", DEV_DTYPE)
@pytest.mark.parametrize("width", [8, 72, 77, 1024, 4104])
def test_residual_add_and_rms_norm_with_offset_weight(dev, dtype, width):
    y, w, eps = _rand(dev, dtype, 5, width), _rand(dev, dtype, width, seed=1) * 0.5, 1e-3
    for res in (_rand(dev, dtype, 5, width, seed=2), _rand(dev, F32, 5, width, seed=3) * 30):
        if dtype == F32 and res.dtype != F32:
            continue
        for add in (True, False):
            want = res.double().cpu() + (y.double().cpu() if add else 0)
            keep = res.clone()
            h, none = ops.add_rms_norm(y if add else None, keep, w, eps, 1.0, update=False)
            assert none is None and torch.equal(keep, res)
            h2, r = ops.add_rms_norm(y if add else None, keep, w, eps, 1.0)
            assert r.dtype == F32 and h.dtype == dtype and torch.equal(h, h2)
            _close(r, want, F32)                          # the stream is 32-bit whatever the model's dtype
            _close(h, plain.model_norm(want, w.double().cpu(), eps), dtype)
    h, _ = ops.add_rms_norm(y, res, w, eps, 0.0, update=False)
    _close(h, plain.rms(res.double().cpu() + y.double().cpu(), eps) * w.double().cpu(), dtype)


@pytest.mark.parametrize("dev,dtype", DEV_DTYPE)
@pytest.mark.parametrize("T,width,ff", [(3, 40, 24), (70, 64, 136), (300, 128, 200), (9, 21, 13), (40, 2048, 64)])
def test_gelu_tanh_gate_and_up_projection(dev, dtype, T, width, ff):
    x, w = _rand(dev, dtype, T, width), _rand(dev, dtype, 2 * ff, width, seed=1) / math.sqrt(width) * 2
    xd, wd = x.double().cpu(), w.double().cpu()
    want = plain.gelu_tanh(xd @ wd[:ff].t()) * (xd @ wd[ff:].t())
    _close(ops.gemm_gated(x, w, "gelu_tanh"), want, dtype)
    got = ops.gemm_gated(x, w, "silu")
    _close(got, plain.silu(xd @ wd[:ff].t()) * (xd @ wd[ff:].t()), dtype)


@pytest.mark.parametrize("dev,dtype", DEV_DTYPE)
def test_logit_scale(dev, dtype):
    for N, K in ((211, 64), (37, 21), (300, 512)):
        x, w = _rand(dev, dtype, 6, K), _rand(dev, dtype, N, K, seed=1)
        got = ops.gemm_softcap(x, w, 0.0, 0.37)
        assert got.dtype == F32
        want = 0.37 * (x.double().cpu() @ w.double().cpu().t())
        _close(got, want, F32, 50)                       # straight from the accumulator, not rounded to bf16
        _close(ops.gemm_softcap(x, w, 3.0, 0.37), 3.0 * torch.tanh(want / 3.0), F32, 50)


@pytest.mark.parametrize("dev,dtype", DEV_DTYPE)
@pytest.mark.parametrize("H,G,d,dv,D", [(4, 2, 20, 28, 64), (6, 1, 128, 96, 128), (3, 3, 7, 5, 64), (2, 2, 16, 24, 64)])
def test_projection_norms_temperature_and_cache_write(dev, dtype, H, G, d, dv, D):
    T, bs, eps = 9, 16, 1e-2
    nq, nk = H * d, G * d
    row = _rand(dev, dtype, T, nq + nk + G * dv + 24) * 2
    qw, kw = _rand(dev, dtype, nq, seed=1), _rand(dev, dtype, nk, seed=2)
    cache = torch.full((4, 2, G, bs, D), 9.0, dtype=dtype, device=dev)
    pos = torch.tensor([0, 5, 6, 7, 8, 22, 23, 24, 1000], dtype=torch.int32, device=dev)
    slots = torch.tensor([3, 17, 15, 16, -1, 40, 63, 0, 31], dtype=torch.int32, device=dev)
    off = (nq + 8, nq + nk + 16)                          # parts may start behind padding
    q = ops.norm_and_cache(row, pos, cache, slots, H, G, d, dv, qw, kw, eps, (0.7, 8), offsets=off)
    r = row.double().cpu()
    want = plain.rms(r[:, :nq], eps) * qw.double().cpu()
    want *= torch.tensor([plain.query_temperature(int(p), {"coef": 0.7, "every": 8}) for p in pos]).double()[:, None]
    _close(q[..., :d], want.reshape(T, H, d), dtype)
    assert (q[..., d:] == 0).all()
    k = (plain.rms(r[:, off[0]:off[0] + nk], eps) * kw.double().cpu()).reshape(T, G, d)
    v = r[:, off[1]:off[1] + G * dv].reshape(T, G, dv)
    flat = cache.permute(0, 3, 1, 2, 4).reshape(4 * bs, 2, G, D).cpu()
    for t, s in enumerate(slots.tolist()):
        if s >= 0:
            _close(flat[s, 0, :, :d], k[t], dtype)
            _close(flat[s, 1, :, :dv], v[t], dtype)
            assert (flat[s, 0, :, d:] == 0).all() and (flat[s, 1, :, dv:] == 0).all()
    used = [s for s in slots.tolist() if s >= 0]
    assert (flat[[i for i in range(4 * bs) if i not in used]] == 9).all()
    # squared sums that come from outside replace the rows' own
    one = torch.ones(T, device=dev)
    q2 = ops.norm_and_cache(row, pos, cache, slots, H, G, d, dv, qw, kw, eps, None, one * nq, one * nk, (nq, nk), off)
    _close(q2[..., :d], (r[:, :nq] / math.sqrt(1 + eps) * qw.double().cpu()).reshape(T, H, d), dtype)


def paged_case(dev, dtype, lens, ctxs, H, G, D, bs=16, seed=0):
    """Queries of a ragged batch, a shuffled paged cache, and the keys and values per request."""
    rng = np.random.RandomState(seed)
    kv, tables, n = [], [], 1
    total = [a + b for a, b in zip(lens, ctxs)]
    blocks = [-(-t // bs) for t in total]
    ids = (rng.permutation(sum(blocks)) + 1).tolist()
    cache = torch.zeros(sum(blocks) + 1, 2, G, bs, D, dtype=dtype, device=dev)
    for r, t in enumerate(total):
        k, v = _rand(dev, dtype, t, G, D, seed=seed + 10 + r), _rand(dev, dtype, t, G, D, seed=seed + 50 + r)
        mine, ids = ids[:blocks[r]], ids[blocks[r]:]
        for p in range(t):
            cache[mine[p // bs], 0, :, p % bs], cache[mine[p // bs], 1, :, p % bs] = k[p], v[p]
        kv.append((k.double().cpu(), v.double().cpu()))
        tables.append(mine)
    n = max(blocks)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)                      # noqa: E731
    qsl = np.concatenate([[0], np.cumsum(lens)]).tolist()
    q = _rand(dev, dtype, qsl[-1], H, D, seed=seed + 99)
    nd = sum(1 for a, b in zip(lens, ctxs) if a == 1 and b > 0)
    meta = AttentionMetadata(i32([0] * qsl[-1]), i32([0] * qsl[-1]), i32([t + [0] * (n - len(t)) for t in tables]),
                             i32(total), i32(qsl), len(lens), qsl[-1], num_decode_reqs=nd, max_query_len=max(lens),
                             max_seq_len=max(total), query_start_loc_cpu=torch.tensor(qsl))
    return q, cache, meta, kv


@pytest.mark.parametrize("dev,dtype", DEV_DTYPE)
@pytest.mark.parametrize("H,G,D", [(4, 2, 64), (8, 2, 128), (6, 1, 128), (3, 3, 36), (2, 1, 160)])
def test_sink_attention_over_pages(dev, dtype, H, G, D):
    """Decoded tokens, portions and prompts in one batch; sinks from negligible to dominant."""
    lens, ctxs = [1, 1, 2, 17, 70, 1], [16, 95, 31, 15, 0, 0]
    q, cache, meta, kv = paged_case(dev, dtype, lens, ctxs, H, G, D)
    sinks = torch.linspace(-9.0, 6.0, H, device=dev)
    got = ops.paged_attention(q, cache, meta, 0.4 if D <= 64 else 0.2, sinks=sinks).double().cpu()
    scale, at = (0.4 if D <= 64 else 0.2), 0
    for n, c, (k, v) in zip(lens, ctxs, kv):
        for i in range(n):
            for h in range(H):
                s = k[:c + i + 1, h // (H // G)] @ q[at + i, h].double().cpu() * scale
                want = plain.sink_softmax(s, sinks[h].double().cpu().reshape(())) @ v[:c + i + 1, h // (H // G)]
                _close(got[at + i, h], want, dtype, 2)
        at += n
    with_sinks = ops.paged_attention(q, cache, meta, scale, sinks=sinks).float()
    without = ops.paged_attention(q, cache, meta, scale).float()
    assert (with_sinks - without).abs().max() > 0.05         # a sink that is left out shows


def _plan(kind, dtype, dev, H, G, d, dv, taps=0, dims=None, decay=None, seed=0, **kw):
    """(plan, first free column) of a row q | k | v | beta with padding between the parts."""
    up = lambda n: (n + 7) // 8 * 8                                                      # noqa: E731
    k0 = up(G * d)
    v0 = k0 + up(G * d)
    b0 = v0 + up(H * dv)
    rnd = lambda *s, scale=1.0: _rand(dev, F32, *s, seed=seed + len(s), scale=scale)     # noqa: E731
    if kind == "retention":
        dims = dims if dims is not None else d // 2 * 2
        p = la.LinearAttentionPlan(H, G, d, dv, (0, k0, v0), "silu", 1e-5, k_mult=d ** -0.5,
                                   inv_freq=ops.ref.rope_inv_freq(dims, 50.0).to(dev) if dims else None,
                                   decay=torch.tensor(decay or [0.9 ** (1 + h) for h in range(H)], dtype=F32, device=dev))
    else:
        p = la.LinearAttentionPlan(H, G, d, dv, (0, k0, v0), "sigmoid", 1e-5, q_mult=d ** -0.5, unit_norm=True, taps=taps,
                                   norm_w=rnd(dv), conv_w=rnd(2 * G * d + H * dv, taps, scale=0.7).to(dtype), beta_offset=b0,
                                   A_log=kw.get("A_log", rnd(H)), dt_bias=rnd(H * d) - 1.0)
    return p, b0 + up(H)


def _carried(kind, p, row, a, gate, n_before=0):
    """Plain result for one request from its first token on (rows fp64 on the CPU)."""
    x = la.split_qkv(p, row)
    H, G, d, dv = p.heads, p.k_heads, p.dim, p.vdim
    c = lambda t: t.double().cpu()                                                       # noqa: E731
    if kind == "retention":
        q, k, v = x.split([G * d, G * d, H * dv], -1)
        rot = {"base": 50.0, "dims": 2 * p.inv_freq.numel() if p.inv_freq is not None else 0}
        q, k = (plain.rotate_halves(t.reshape(-1, G, d), rot) if rot["dims"] else t.reshape(-1, G, d) for t in (q, k))
        o, st = plain.retention_states(q, k * d ** -0.5, v.reshape(-1, H, dv), c(p.decay))
        return (plain.rms(o, p.eps).reshape(-1, H * dv) * plain.silu(gate)), st
    x = plain.short_conv(x, c(p.conv_w))
    q, k, v = x.split([G * d, G * d, H * dv], -1)
    q = (plain.unit(q.reshape(-1, G, d)) * d ** -0.5).repeat_interleave(H // G, 1)
    k = plain.unit(k.reshape(-1, G, d)).repeat_interleave(H // G, 1)
    beta = plain.sigmoid(row[:, p.beta_offset:p.beta_offset + H])
    g = plain.delta_decay(a, c(p.A_log), c(p.dt_bias), H)
    o, st = plain.delta_states(q, k, v.reshape(-1, H, dv), g, beta)
    return (plain.rms(o, p.eps) * c(p.norm_w)).reshape(-1, H * dv) * plain.sigmoid(gate), st


def _state_meta(dev, lens, starts, slots):
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)                       # noqa: E731
    qsl = np.concatenate([[0], np.cumsum(lens)]).tolist()
    nd = 0
    while nd < len(lens) and lens[nd] == 1 and starts[nd] > 0:
        nd += 1
    return AttentionMetadata(i32([0] * qsl[-1]), i32([0] * qsl[-1]), i32([[0]] * len(lens)),
                             i32([a + b for a, b in zip(lens, starts)]), i32(qsl), len(lens), qsl[-1], num_decode_reqs=nd,
                             max_query_len=max(lens), max_seq_len=999, state_slots=i32(slots),
                             query_start_loc_cpu=torch.tensor(qsl))


CARRIED = [("retention", 3, 3, 24, 40, 0, {}), ("retention", 2, 2, 64, 64, 0, {"dims": 32}), ("retention", 1, 1, 10, 3, 0, {"dims": 0}),
           ("retention", 2, 2, 128, 200, 0, {"decay": [1.0, 0.003]}), ("retention", 1, 1, 256, 128, 0, {}),
           ("delta", 4, 2, 32, 64, 4, {}), ("delta", 3, 1, 40, 24, 3, {}), ("delta", 2, 2, 9, 11, 2, {}), ("delta", 2, 1, 16, 16, 1, {}),
           ("delta", 2, 2, 128, 128, 4, {}), ("delta", 1, 1, 200, 72, 7, {}), ("delta", 1, 1, 24, 16, 11, {}),
           ("delta", 1, 1, 264, 12, 4, {})]


@pytest.mark.parametrize("dev,dtype", DEV_DTYPE)
@pytest.mark.parametrize("kind,H,G,d,dv,taps,kw", CARRIED, ids=lambda v: str(v) if not isinstance(v, dict) else "-".join(v))
def test_carried_state_over_portions_batches_and_reused_slots(dev, dtype, kind, H, G, d, dv, taps, kw):
    """Four sequences whose portions meet in ragged batches; slots come back with other sequences' leftovers."""
    p, n = _plan(kind, dtype, dev, H, G, d, dv, taps, **kw)
    slots_n = 4
    state = torch.full(p.state_shape(slots_n), 5.0, device=dev)
    cache = (torch.full(p.ring_shape(slots_n), 5.0, dtype=dtype, device=dev), state) if taps else (state,)
    total = {"a": 61, "b": 19, "c": 3, "e": 40}
    seq = {}
    for i, (k, t) in enumerate(total.items()):
        row, gate = _rand(dev, dtype, t, n, seed=20 + i), _rand(dev, dtype, t, H * dv, seed=40 + i)
        a = _rand(dev, dtype, t, H * d, seed=60 + i) * 2 if kind == "delta" else None
        seq[k] = (row, a, gate)
    got, at = {k: [] for k in seq}, dict.fromkeys(seq, 0)
    steps = [[("a", 1), ("b", 2)], [("b", 1), ("a", 15)], [("a", 1), ("c", 3), ("b", 16)], [("a", 33), ("e", 17)],
             [("a", 1), ("e", 1)], [("e", 22), ("a", 2)], [("a", 8)]]
    slot_of = {"a": 2, "b": 0, "c": 3, "e": 0}            # e takes b's slot
    for step in steps:
        lens = [x for _, x in step]
        parts = [tuple(t[at[k]:at[k] + x] if t is not None else None for t in seq[k]) for k, x in step]
        row, a, gate = (torch.cat(t) if t[0] is not None else None for t in zip(*parts))
        y = ops.carried_state_attention(p, row, a, gate, _state_meta(dev, lens, [at[k] for k, _ in step],
                                                                     [slot_of[k] for k, _ in step]), cache)
        lo = 0
        for k, x in step:
            got[k].append(y[lo:lo + x])
            lo += x
            at[k] += x
    assert at == total
    for k, (row, a, gate) in seq.items():
        want, st = _carried(kind, p, row.double().cpu(), a.double().cpu() if a is not None else None, gate.double().cpu())
        g = torch.cat(got[k]).double().cpu()
        err = ((g - want).norm() / want.norm()).item()
        assert err < (3e-6 if dtype == F32 else 6e-3), (k, err)
        if k != "b":
            es = ((state[slot_of[k]].double().cpu() - st).norm() / st.norm()).item()
            assert es < (3e-6 if dtype == F32 else 2e-5), (k, es)
    assert (state[1] == 5.0).all()                        # a slot that nobody used


@pytest.mark.parametrize("dev,dtype", DEV_DTYPE)
def test_strong_decays_leave_recent_tokens_exact(dev, dtype):
    """Factors from one to nothing within a chunk: what is forgotten must not disturb what is kept."""
    H, d, dv = 2, 32, 32
    p, n = _plan("delta", dtype, dev, H, H, d, dv, 4, A_log=torch.tensor([4.0, -6.0], device=dev))
    T = 50
    row, gate = _rand(dev, dtype, T, n, seed=1), _rand(dev, dtype, T, H * dv, seed=2)
    a = _rand(dev, dtype, T, H * d, seed=3) * 6
    cache = (torch.zeros(p.ring_shape(1), dtype=dtype, device=dev), torch.zeros(p.state_shape(1), device=dev))
    y = ops.carried_state_attention(p, row, a, gate, _state_meta(dev, [T], [0], [0]), cache)
    want, st = _carried("delta", p, row.double().cpu(), a.double().cpu(), gate.double().cpu())
    assert torch.isfinite(y).all()
    assert ((y.double().cpu() - want).norm() / want.norm()).item() < (2e-5 if dtype == F32 else 6e-3)
    assert ((cache[1][0].double().cpu() - st).norm() / st.norm()).item() < 2e-5


@pytest.mark.gpu
def test_decode_rows_of_padded_requests_come_back_as_zeros():
    p, n = _plan("delta", BF16, "cuda", 2, 2, 16, 16, 4)
    cache = (torch.zeros(p.ring_shape(3), dtype=BF16, device="cuda"), torch.zeros(p.state_shape(3), device="cuda"))
    meta = _state_meta("cuda", [1, 1], [4, 9], [0, 2])
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device="cuda")                    # noqa: E731
    meta.query_start_loc, meta.seq_lens, meta.state_slots = i32([0, 1, 2, 2, 2]), i32([5, 10, 0, 0]), i32([0, 2, -1, -1])
    meta.padded_num_reqs, meta.padded_num_tokens = 4, 4
    row = _rand("cuda", BF16, 4, n)
    y = ops.carried_state_attention(p, row, _rand("cuda", BF16, 4, 32), _rand("cuda", BF16, 4, 32), meta, cache)
    assert (y[2:] == 0).all() and (y[:2] != 0).any() and (cache[1][1] == 0).all()


@pytest.mark.gpu
@pytest.mark.parametrize("kind,taps", [("retention", 0), ("delta", 4)])
@pytest.mark.parametrize("chunks", [1, 5])
def test_prompts_in_several_slabs_on_two_streams(monkeypatch, kind, taps, chunks):
    """A scratch of few chunks: states cross slabs in the pool, requests of unequal lengths end in different slabs."""
    from vllm_torchtpu_b200.ops import cuda, cuda_linear
    H, d, dv = 2, 64, 96
    per = cuda.lib().b200_linear_attention_chunk_bytes(d, dv, int(kind == "delta"))
    monkeypatch.setattr(cuda_linear.slabs, "__defaults__", (chunks * H * per,))
    p, n = _plan(kind, BF16, "cuda", H, H, d, dv, taps)
    lens, slots = [1, 150, 33, 2, 97], [4, 2, 0, 3, 1]
    assert len(cuda_linear.slabs(lens[1:], H, per)) > 3
    state = torch.full(p.state_shape(5), 5.0, device="cuda")
    cache = (torch.full(p.ring_shape(5), 5.0, dtype=BF16, device="cuda"), state) if taps else (state,)
    seqs = []
    for i, t in enumerate(lens):
        t += i == 0
        seqs.append((_rand("cuda", BF16, t, n, seed=i), _rand("cuda", BF16, t, H * d, seed=i + 20) if taps else None,
                     _rand("cuda", BF16, t, H * dv, seed=i + 40)))
    first = tuple(t[:1] if t is not None else None for t in seqs[0])
    ops.carried_state_attention(p, *first, _state_meta("cuda", [1], [0], [4]), cache)
    parts = [tuple(t[1:] if t is not None else None for t in seqs[0])] + seqs[1:]
    row, a, gate = (torch.cat(t) if t[0] is not None else None for t in zip(*parts))
    for _ in range(2):                                    # the second time over states that the first one left
        y = ops.carried_state_attention(p, row, a, gate, _state_meta("cuda", lens, [1, 0, 0, 0, 0], slots), cache)
        if _ == 0:
            y0 = y.clone()
    at = 1
    for (r, a_, g), x, slot in list(zip(seqs, lens, slots))[1:]:
        want, st = _carried(kind, p, r.double().cpu(), a_.double().cpu() if taps else None, g.double().cpu())
        for got in (y0, y):
            e = got[at:at + x].double().cpu() - want
            assert (e.norm() / want.norm()).item() < 6e-3
        assert ((state[slot].double().cpu() - st).norm() / st.norm()).item() < 2e-5
        at += x


def test_slabs_cover_every_chunk_once():
    from vllm_torchtpu_b200.ops.cuda_linear import CHUNK, slabs
    for lens in ([1], [16, 17, 1, 400], [5000], [3] * 300 + [2000]):
        for budget in (1 << 16, 1 << 20, 48 << 20):
            seen, per = set(), max(1, budget // (8 * 40000))
            for i, j, c, n in slabs(lens, 8, 40000, budget):
                assert n >= 1 and ((j - i) * n <= per or (j - i) == 1 and n == 1)
                for r in range(i, j):
                    for x in range(c, min(c + n, -(-lens[r] // CHUNK))):
                        assert (r, x) not in seen
                        seen.add((r, x))
            assert seen == {(r, x) for r, t in enumerate(lens) for x in range(-(-t // CHUNK))}


# ------------------------------------------------------------------------------------------------- the model
@pytest.mark.parametrize("dev", DEVS)
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(MODELS))
def test_prompt_portions_and_single_tokens_match_the_plain_model(tmp_path, dev, dtype, name):
    cfg = MODELS[name]
    if name == "wide" and dev == "cpu":
        pytest.skip("sizes for the tensor-core kernels")
    w = write_model(str(tmp_path), cfg, seed=3)
    toks = tokens_of(83, cfg["vocab"], 1)
    want = plain.forward(cfg, w, toks)
    rep = make_replay(str(tmp_path), dtype, 128, dev)
    for cuts in ([83], [50] + [1] * 33, portions(83, [2, 3]), portions(83, [15, 2, 16, 1, 17, 31])):
        got = replay_logits(rep, toks, cuts)
        assert_like(got, want, dtype, cuts)
    if name == "mixed":
        assert_like(replay_logits(rep, toks, [1] * 83), want, dtype)


@pytest.mark.parametrize("dev", DEVS)
def test_residual_stream_after_every_layer(tmp_path, dev):
    """32-bit layer by layer, so that two mistakes cannot make up for each other."""
    w = write_model(str(tmp_path), MIXED, seed=9)
    toks = tokens_of(21, MIXED["vocab"], 4)
    want: list = []
    plain.forward(MIXED, w, toks, layers_out=want)
    rep = make_replay(str(tmp_path), "float32", 64, dev)
    model, got = rep.engine.runner.model, []
    for layer in model.layers:
        fwd = layer.forward

        def spy(*a, fwd=fwd):
            y, r = fwd(*a)
            got.append((r + y).double().cpu())
            return y, r
        layer.forward = spy
    replay_logits(rep, toks, [21])
    assert len(got) == len(want) == 6
    for g, e in zip(got, want):
        assert (g - e).abs().max() < 3e-5 * e.abs().max()


@pytest.mark.parametrize("dev", DEVS)
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_mixed_batches_reused_pages_and_slots_match_each_request_alone(tmp_path, dev, dtype):
    cfg = MIXED
    w = write_model(str(tmp_path), cfg, seed=5)
    rep = make_replay(str(tmp_path), dtype, 176, dev)                # eleven pages for eight requests
    rng = np.random.RandomState(7)
    reqs = {f"r{i}": tokens_of(n, cfg["vocab"], 10 + i) for i, n in enumerate((70, 33, 1, 48, 17, 64, 2, 31))}
    want = {k: plain.forward(cfg, w, v) for k, v in reqs.items()}
    queue, live, at, got = list(reqs), [], {}, {k: [] for k in reqs}
    pool = rep.engine.scheduler.kv.pool
    free0 = pool.num_free_blocks
    while queue or live:
        while queue and len(live) < 4 and sum(-(-len(reqs[k]) // 16) for k in live + queue[:1]) <= 11:
            live.append(queue.pop(0))
            at[live[-1]] = 0
        entries, end = [], []
        for k in live:
            if rng.rand() < 0.2 and len(live) > 1:
                continue                                             # left out of this step
            n = min(int(rng.choice([1, 1, 2, 3, 16, 19, 40])), len(reqs[k]) - at[k])
            entries.append((k, reqs[k][at[k]:at[k] + n], list(range(n))))
            at[k] += n
            if at[k] == len(reqs[k]):
                end.append(k)
        rows = rep.step(entries, end)
        lo = 0
        for k, t, _ in entries:
            got[k].append(rows[lo:lo + len(t)])
            lo += len(t)
        live = [k for k in live if k not in end]
    for k in reqs:
        assert_like(torch.cat(got[k]), want[k], dtype, k)
    assert pool.num_free_blocks == free0


@pytest.mark.parametrize("dev", DEVS)
def test_far_keys_sinks_temperature_states_and_convolution_windows_decide_logits(tmp_path, dev):
    """With pointed weights each mistake that is planted in the plain model moves its logits far; the engine stays with
    the unspoilt model, in prompts and in decoding."""
    cfg = config([(attention(every=10, coef=0.6), 0, None), (retention(decay=[0.999, 0.99, 0.98]), 0, None),
                  (delta(conv=4), 48, None)])

    def edit(w):
        w["l0.mix.q.norm"] = (w["l0.mix.q.norm"].float() * 4).bfloat16()
        w["l2.mix.dt_bias"] = (w["l2.mix.dt_bias"].float() - 4).bfloat16()
    w = write_model(str(tmp_path), cfg, seed=2, edit=edit)
    toks = tokens_of(130, cfg["vocab"], 3)
    want = plain.forward(cfg, w, toks)
    rep = make_replay(str(tmp_path), "float32", 192, dev)
    for cuts in ([97, 2] + [1] * 31, portions(130, [2, 5]), [130]):
        assert logit_error(replay_logits(rep, toks, cuts), want) < LIMIT["float32"] * 5, cuts
    plants = [{0: {"lost_key": k}} for k in (0, 1, 15, 16, 31, 32, 63, 64, 96, 97)]
    plants += [{0: {"no_sink": True}}, {0: {"no_temp": True}}]
    plants += [{1: {"forget_at": p}} for p in (1, 16, 64, 97, 99)]
    plants += [{2: {"conv_cut": p}} for p in (1, 2, 16, 97, 99, 100)]
    for plant in plants:
        wrong = plain.forward(cfg, w, toks, plant=plant)
        assert logit_error(wrong, want) > 100 * LIMIT["float32"], plant


@pytest.mark.parametrize("dev", DEVS)
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_first_tokens_of_a_sequence_after_a_slot_was_used(tmp_path, dev, dtype):
    w = write_model(str(tmp_path), MIXED, seed=1)
    rep = make_replay(str(tmp_path), dtype, 64, dev)
    for n in (1, 2, 3, 5, 1):
        toks = tokens_of(n, MIXED["vocab"], n)
        want = plain.forward(MIXED, w, toks)
        for cuts in ([n], [1] * n):
            assert_like(replay_logits(rep, toks, cuts), want, dtype)


@pytest.mark.parametrize("dev", DEVS)
@pytest.mark.parametrize("kw", [{}, {"async_scheduling": True}, {"enforce_eager": True},
                                {"enable_prefix_caching": True}, {"num_gpu_blocks_override": 12},
                                {"speculative_config": {"method": "ngram", "num_speculative_tokens": 3}}],
                         ids=lambda k: next(iter(k), "default"))
def test_greedy_generation_through_the_engine(tmp_path, dev, kw):
    """``LLM.generate`` in 32-bit: chunked prompts (40-token steps), batches of unequal requests, long decoding, a pool
    small enough to preempt (states start over), rejected drafts (states are rolled back), against the plain model."""
    from vllm_torchtpu_b200.engine.llm import LLM
    cfg = config([(delta(), 64, None), (attention(), 0, None), (retention(), 0, None), (delta(), 64, 0)])
    w = write_model(str(tmp_path), cfg, seed=6)
    prompts = [tokens_of(n, cfg["vocab"], n) for n in (3, 52, 17, 41)]
    if "enable_prefix_caching" in kw or "speculative_config" in kw:
        prompts[3] = prompts[1][:32] + prompts[1][:9]
    llm = LLM(str(tmp_path), device=dev, dtype="float32", max_num_seqs=4, max_num_batched_tokens=40, max_model_len=128,
              init_dist=False, **{"num_gpu_blocks_override": 64, **kw})
    n_out = 48 if not kw else 24
    sp = SamplingParams(temperature=0.0, max_tokens=n_out, ignore_eos=True)
    outs = llm.generate(prompts, sp)
    for p, o in zip(prompts, outs):
        ids = o.outputs[0].token_ids
        assert len(ids) == n_out
        z = plain.forward(cfg, w, list(p) + list(ids[:-1]))[len(p) - 1:]
        top = z.max(-1).values
        assert (top - z[torch.arange(n_out), torch.tensor(ids)] <= 1e-4).all()      # ties aside, the greedy path
    if kw.get("num_gpu_blocks_override") == 12:
        assert llm.engine.scheduler.stats["preemptions"] > 0
    if "speculative_config" in kw:
        assert llm.engine.runner.stats.get("spec_drafted", 0) > 0
    if "enable_prefix_caching" in kw:                     # a prefix has no state to continue from: never reused
        assert llm.generate([prompts[3]], sp)[0].outputs[0].token_ids == outs[3].outputs[0].token_ids
        assert llm.engine.scheduler.stats.get("prefix_hit_tokens", 0) == 0


@pytest.mark.gpu
def test_bf16_decode_graphs_match_eager_steps(tmp_path):
    from vllm_torchtpu_b200.engine.llm import LLM
    from vllm_torchtpu_b200.ops import cuda
    cfg = MODELS["wide"]
    write_model(str(tmp_path), cfg, seed=8)
    prompts = [tokens_of(n, cfg["vocab"], n) for n in (5, 33, 90)]
    sp = SamplingParams(temperature=0.0, max_tokens=12, ignore_eos=True)
    got = []
    for eager in (True, False):
        llm = LLM(str(tmp_path), device="cuda", max_num_seqs=8, max_num_batched_tokens=64, num_gpu_blocks_override=64,
                  enforce_eager=eager, init_dist=False)
        got.append([o.outputs[0].token_ids for o in llm.generate(prompts, sp)])
        assert eager or llm.engine.runner.stats["graph_steps"] > 0
    assert got[0] == got[1]
    assert cuda.check_status() == 0


@pytest.mark.gpu
def test_pool_size_and_long_bf16_decoding_with_default_settings(tmp_path):
    """HBM budget with state pools, graphs of several buckets, 300 decoded tokens."""
    from vllm_torchtpu_b200.engine.llm import LLM
    w = write_model(str(tmp_path), MIXED, seed=4)
    llm = LLM(str(tmp_path), device="cuda", max_num_seqs=4, max_model_len=512, gpu_memory_utilization=0.05, init_dist=False)
    p = tokens_of(20, MIXED["vocab"], 1)
    ids = llm.generate([p], SamplingParams(temperature=0.0, max_tokens=300, ignore_eos=True))[0].outputs[0].token_ids
    z = plain.forward(MIXED, w, p + list(ids[:-1]))[len(p) - 1:]
    short = z.max(-1).values - z[torch.arange(300), torch.tensor(ids)]
    assert (short < 0.1 * z.std()).all()                 # the arg-max up to bf16 rounding


# ------------------------------------------------------------------------------------------------- surroundings
def test_configuration_reads_every_size_and_refuses_what_is_not_built():
    mc = ModelConfig.from_hf_dict(MIXED, "m")
    assert mc.architecture == "popanex" and mc.num_layers == 6 and mc.vocab_size == 211 and mc.logit_scale == 1.7
    assert [s.weights_of for s in mc.layer_specs] == [None, None, None, 2, None, 1]
    assert [s.ff for s in mc.layer_specs] == [88, 0, 56, 56, 0, 0] and mc.has_recurrent_state and not mc.is_mla
    assert [mc.layer_is_full_attention(i) for i in range(6)] == [False, True, False, False, False, True]
    assert mc.layer_specs[2].mixer.rot.dims == 16 and mc.layer_specs[1].mixer.q_temp.every == 24
    only = ModelConfig.from_hf_dict(MODELS["attention_only"])
    assert not only.has_recurrent_state
    bad = [("type", lambda c: c["layers"][0].update(type="other")),
           ("feed-forward", lambda c: c["layers"][0]["mlp"].update(kind="experts")),
           ("sizes differ", lambda c: c["layers"][3].update(weights_of=1)),
           ("leads back", lambda c: c["layers"][2].update(weights_of=3)),
           ("rot.dims", lambda c: c["layers"][2]["mixer"]["rot"].update(dims=26)),
           ("decays", lambda c: c["layers"][2]["mixer"].update(decay=[0.5])),
           ("divide", lambda c: c["layers"][1]["mixer"].update(kv_heads=3))]
    for what, change in bad:
        c = json.loads(json.dumps(MIXED))
        change(c)
        with pytest.raises(ValueError, match=what):
            ModelConfig.from_hf_dict(c)
    for cfg, kw in ((MIXED, dict(parallel=ParallelConfig(tensor_parallel_size=4))),
                    (MIXED, dict(parallel=ParallelConfig(pipeline_parallel_size=2))),
                    (MIXED, dict(speculative={"method": "mtp"})),
                    (MIXED, dict(kv_transfer={"kv_connector": "B200HostConnector"})),
                    (MIXED, dict(cache=CacheConfig(kv_cache_dtype="fp8"))),
                    (MODELS["attention_only"], dict(parallel=ParallelConfig(prefill_context_parallel_size=2)))):
        with pytest.raises(ValueError):
            EngineConfig(model=ModelConfig.from_hf_dict(cfg), device="cpu", **kw).finalize()


def test_shared_weights_are_held_once_with_a_cache_per_layer(tmp_path):
    write_model(str(tmp_path), MIXED)
    r = make_replay(str(tmp_path), "float32", 64, "cpu").engine.runner
    m = r.model
    assert m.layers[3].self_attn is m.layers[2].self_attn and m.layers[3].mlp is m.layers[2].mlp
    assert m.layers[5].norm1 is m.layers[1].norm1 and len(m.weight_owners()) == 4
    assert len(r.distinct_kv_caches) == 6 and r.kv_caches[3][0].shape == (5, 3, 24, 40)
    assert r.kv_caches[0][0].shape == (5, 3, 2 * 2 * 16 + 4 * 24) and r.kv_caches[1].shape == (5, 2, 2, 16, 28)
    assert m.kv_bytes_per_block(16, torch.float32) == 2 * (2 * 2 * 16 * 28) * 4


def test_incomplete_checkpoints_are_refused_and_weights_can_be_replaced(tmp_path):
    from safetensors.torch import save_file
    cfg = config([(delta(), 40, None)])
    w = write_model(str(tmp_path / "a"), cfg, seed=0)
    w2 = random_model(cfg, seed=1)
    write_model(str(tmp_path / "b"), cfg)
    save_file({k: v for k, v in w.items() if k != "l0.mix.g1"}, str(tmp_path / "b" / "model.safetensors"))
    with pytest.raises(ValueError, match="l0.mix.g1"):
        make_replay(str(tmp_path / "b"), "float32", 64, "cpu")
    rep = make_replay(str(tmp_path / "a"), "float32", 64, "cpu")
    toks = tokens_of(9, cfg["vocab"])
    part = {k: w2[k] for k in ("l0.mix.q.conv", "l0.mix.k.conv", "l0.mix.v.conv", "l0.mix.A_log", "l0.mix.dt_bias",
                               "l0.mix.norm", "l0.mlp.gate", "l0.mlp.up", "final.norm")}
    rep.engine.update_weights(part)
    assert logit_error(replay_logits(rep, toks, [9]), plain.forward(cfg, w | part, toks)) < LIMIT["float32"]


def test_trace_run_command(tmp_path):
    w = write_model(str(tmp_path / "m"), MIXED)
    toks = tokens_of(12, MIXED["vocab"])
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:7], "want": [0, 6]}, {"id": "b", "tokens": toks[:2], "want": []}],
              "end": ["b"]},
             {"step": 1, "entries": [{"id": "b", "tokens": toks[:1], "want": [0]}, {"id": "a", "tokens": toks[7:], "want": [4]}],
              "end": ["a", "b"]}]
    os.mkdir(tmp_path / "out")
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", "float32",
                        "--out", str(tmp_path / "out"), "--max-tokens", "64", "--device", "cpu"],
                       input="\n".join(map(json.dumps, steps)), capture_output=True, text=True, timeout=120)
    assert r.returncode == 0, r.stderr[-2000:]
    z = plain.forward(MIXED, w, toks)
    for n, rows in ((0, [0, 6]), (1, [0, 11])):
        got = torch.from_numpy(np.fromfile(tmp_path / "out" / f"{n}.f32", "<f4").reshape(-1, MIXED["vocab"]))
        assert logit_error(got, z[rows]) < LIMIT["float32"]


def test_two_tensor_parallel_ranks_match_one():
    """Sharded heads with key heads on one rank each or replicated, and norms over the sharded projections."""
    from test_parallel_cpu import _run
    assert _run(2, "tp", "tiny-popanex") == _run(1, "tp", "tiny-popanex")


def test_server_command_line_builds_the_engine(tmp_path):
    import argparse

    from vllm_torchtpu_b200.entrypoints import cli
    write_model(str(tmp_path), MIXED)
    ap = argparse.ArgumentParser()
    cli.add_engine_args(ap)
    llm = cli.make_llm(ap.parse_args([str(tmp_path), "--device", "cpu", "--max-num-seqs", "2", "--max-model-len", "64"]))
    assert type(llm.engine.runner.model).__name__ == "PopanexForCausalLM"
    out = llm.generate([[1, 2, 3]], SamplingParams(max_tokens=4, temperature=0.7, top_p=0.9, logprobs=2))
    assert len(out[0].outputs[0].token_ids) == 4
    assert model_preset("tiny-popanex").architecture == "popanex"
