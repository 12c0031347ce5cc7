"""Vipolix (gated linear attention; chunked attention beside a delta rule with removal rates; token shift, clamped experts in
groups with a shared one, a token input per layer) against the plain statement in ``plain_vipolix.py``: every mechanism
alone, then the model through the engine's scheduler, caches and kernels."""
import copy
import json
import math
import os
import subprocess

import numpy as np
import plain_vipolix as plain
import pytest
import torch
from test_mazivik import BF16, DEV_DTYPE, DEVS, F32, ROOT, _close, _rand, logit_error, portions, replay_logits, tokens_of
from test_popanex import paged_case
from test_zeganex import state_meta

from vllm_torchtpu_b200 import SamplingParams, ops
from vllm_torchtpu_b200.config import CacheConfig, EngineConfig, ModelConfig, ParallelConfig, model_preset
from vllm_torchtpu_b200.entrypoints.trace_replay import make_replay
from vllm_torchtpu_b200.ops import linear_attention as la
from vllm_torchtpu_b200.ops import token_shift
from vllm_torchtpu_b200.ops.short_conv import ConvAttentionPlan

LIMIT = {"float32": 6e-5, "bfloat16": 5e-2}


def assert_like(got, want, dtype, what="", factor=1.0):
    """Every position in 32-bit.  In bf16 half of them closely and four of five within a few times that: rounding may move a token across a close call of the router, and a
    head's output is divided by its root mean square, however small."""
    d = got.double() - want.double()
    e = (d - d.mean(-1, keepdim=True)).pow(2).mean(-1).sqrt() / want.double().pow(2).mean().sqrt()
    if dtype == "float32":
        assert e.max() < LIMIT[dtype] * factor, (what, e.max())
    else:
        q = e.sort().values
        assert q[int(0.5 * (len(e) - 1))] < LIMIT[dtype] * factor and q[int(0.8 * (len(e) - 1))] < 3 * LIMIT[dtype] * factor, (what, e)
        assert e.max() < 1.5, (what, e)


# ------------------------------------------------------------------------------------------------- configurations
def gla(heads=3, dim=24, vdim=40, tau=9.0, rank=12):
    """``rank`` is no entry of the configuration: the tensors' shapes give it."""
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}, "rank": rank}


def par(heads=4, kv_heads=2, dim=24, vdim=20, conv=3, chunk=19, scale=0.3, dims=12, base=900.0, rheads=3, rdim=16, ls=0.7,
        rs=-0.4, rank=10):
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "mask": {"size": chunk},
            "scale": scale, "rot": {"base": base, "dims": dims}}
    return {"type": "parallel", "rank": rank, "mixer": {"left": left, "right": {"heads": rheads, "dim": rdim},
                                                        "left_scale": ls, "right_scale": rs}}


def moe(experts=8, top=2, ff=24, limit=1.5, count=4, keep=2, scale=1.7, shared=40, slimit=0.9):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "shared": {"ff": shared, "limit": slimit},
            "router": {"experts": experts, "top": top, "scale": scale, "groups": {"count": count, "keep": keep}}}


def config(layers, width=72, vocab=211, eps=3e-6, side=20):
    return {"architecture": "Vipolix", "width": width, "vocab": vocab, "norm": {"eps": eps}, "token_side": {"dim": side},
            "layers": [dict(copy.deepcopy(layer), mlp=mlp) for layer, mlp in layers]}


MIXED = config([(gla(), moe()), (par(), moe(6, 3, 56, count=3, keep=2)), (gla(heads=2, dim=16, vdim=16, tau=1.0, rank=5), None),
                (par(heads=2, kv_heads=1, dim=16, vdim=40, conv=1, chunk=16, dims=16, rheads=2, rdim=40, ls=1.0, rs=1.0),
                 moe(4, 1, 16, count=1, keep=1, shared=16)), (par(conv=5, chunk=33, scale=0.5), None)])
MODELS = {
    "mixed": MIXED,
    "all_sizes_odd": config([(par(heads=3, kv_heads=1, dim=7, vdim=5, conv=2, chunk=6, dims=6, rheads=1, rdim=9, rank=3),
                              moe(5, 3, 11, count=5, keep=4, shared=7)), (gla(heads=1, dim=9, vdim=11, tau=2.5, rank=1), None),
                             (gla(heads=2, dim=10, vdim=3, rank=7), moe(3, 2, 9, count=1, keep=1, shared=13))],
                            width=21, vocab=37, side=5),
    "linear_only": config([(gla(heads=2, dim=32, vdim=64, tau=16.0, rank=16), moe(12, 4, 32, count=2, keep=1)),
                           (gla(heads=2, dim=40, vdim=72, rank=24), None)], width=80, side=8),
    "parallel_only": config([(par(chunk=1), None), (par(heads=18, kv_heads=1, dim=36, vdim=52, conv=7, chunk=500, dims=2,
                                                        rheads=2, rdim=24, ls=0.0, rs=0.5), moe()),
                             (par(heads=20, kv_heads=20, dim=64, vdim=64, chunk=24, dims=64, rheads=4, rdim=9, rs=0.0), None)],
                            width=96),
    "wide": config([(par(heads=16, kv_heads=4, dim=128, vdim=128, conv=4, chunk=40, scale=0.08, dims=64, rheads=8, rdim=64),
                     moe(8, 2, 128, shared=256)), (gla(heads=4, dim=64, vdim=128, tau=16.0, rank=32), moe(16, 4, 128, count=4, keep=3)),
                    (par(heads=8, kv_heads=8, dim=64, vdim=64, chunk=24, dims=32, scale=0.12, rheads=2, rdim=128), None),
                    (par(heads=4, kv_heads=2, dim=160, vdim=144, chunk=31, scale=0.07, dims=32, rheads=1, rdim=256), moe(8, 3, 192))],
                   width=256, vocab=1000, side=64),
}


def random_model(cfg, seed=0, gain=1.0):
    """Weights of ``cfg`` (bfloat16), scaled so that activations stay of order one."""
    g = torch.Generator().manual_seed(seed)

    def rnd(*s, scale=1.0, mean=0.0):
        return (mean + torch.randn(*s, generator=g) * scale).bfloat16()

    def mat(o, i, k=1.0):
        return rnd(o, i, scale=k * gain / math.sqrt(i))
    W, L, sd = cfg["width"], len(cfg["layers"]), cfg["token_side"]["dim"]
    w = {"embed": rnd(cfg["vocab"], W), "side.embed": rnd(cfg["vocab"], L * sd), "final.norm": rnd(W, scale=0.3),
         "head": mat(cfg["vocab"], W)}
    for i, layer in enumerate(cfg["layers"]):
        m, p, q = layer["mixer"], f"l{i}.mix.", f"l{i}."
        w[q + "norm1"], w[q + "shift"] = rnd(W, scale=0.3), rnd(W, mean=0.5, scale=0.3)
        w[q + "side.gate"], w[q + "side.proj"], w[q + "side.norm"] = mat(sd, W), mat(W, sd), rnd(W, mean=0.5, scale=0.3)
        if layer["type"] == "gla":
            H, d, dv, r = m["heads"], m["dim"], m["vdim"], layer["rank"]
            for n, c in (("q", H * d), ("k", H * d), ("v", H * dv), ("g", H * dv), ("a1", r)):
                w[p + n] = mat(c, W)
            w[p + "a2"], w[p + "a2.b"], w[p + "norm"] = mat(H * d, r), rnd(H * d, mean=1.0, scale=2.0), rnd(dv, mean=1.0, scale=0.3)
            w[p + "o"] = mat(W, H * dv)
        else:
            m, r, a, b = m["left"], m["right"], p + "left.", p + "right."
            H, G, d, dv, n = m["heads"], m["kv_heads"], m["dim"], m["vdim"], r["heads"] * r["dim"]
            for t, c in (("q", H * d), ("k", G * d), ("v", G * dv)):
                w[a + t], w[a + t + ".b"], w[a + t + ".conv"] = mat(c, W), rnd(c, scale=0.5), rnd(c, m["conv"], scale=0.7)
            w[a + "temp"], w[a + "o"] = rnd(H, mean=1.0, scale=0.5), mat(W, H * dv)
            for t in "rkvga":
                w[b + t] = mat(n, W)
            w[b + "w1"], w[b + "w2"] = mat(layer["rank"], W), mat(n, layer["rank"], 2.0)
            w[b + "w0"], w[b + "a.b"], w[b + "norm"] = rnd(n, mean=-2.0, scale=1.5), rnd(n), rnd(n, mean=1.0, scale=0.3)
            w[b + "o"] = mat(W, n)
        f = layer["mlp"]
        if f:
            p = q + "mlp."
            w[q + "norm2"], w[p + "router"] = rnd(W, scale=0.3), mat(f["router"]["experts"], W, 2.0)
            w[p + "correction"], w[p + "shared.sg"] = rnd(f["router"]["experts"], mean=-1.5, scale=1.2), mat(1, W)
            for e, ff in [(f"e{e}.", f["expert"]["ff"]) for e in range(f["router"]["experts"])] + [("shared.", f["shared"]["ff"])]:
                w[p + e + "gate"], w[p + e + "up"], w[p + e + "down"] = mat(ff, W), mat(ff, W), mat(W, ff)
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
# four sequences whose portions meet in ragged batches; e takes b's slot and pages
TOTAL = {"a": 61, "b": 19, "c": 3, "e": 40}
SLOT = {"a": 2, "b": 0, "c": 3, "e": 0}
STEPS = [[("a", 1), ("b", 2)], [("b", 1), ("a", 15)], [("a", 1), ("c", 3), ("b", 16)], [("a", 33), ("e", 17)],
         [("a", 1), ("e", 1)], [("e", 22), ("a", 2)], [("a", 8)]]


def batches(dev):
    """(metadata, [(sequence, first row, rows)], rows of padding) of the steps."""
    at = dict.fromkeys(TOTAL, 0)
    for step in STEPS:
        lens, starts = [x for _, x in step], [at[k] for k, _ in step]
        pad = 2 if all(x == 1 and s > 0 for x, s in zip(lens, starts)) else 0
        meta = state_meta(dev, lens, starts, [SLOT[k] for k, _ in step], 64, [[i + 1] for i in range(len(step))], pad)
        yield meta, [(k, at[k], x) for k, x in step], pad
        for k, x in step:
            at[k] += x
    assert at == TOTAL


def run_batches(dev, fn):
    """fn(meta, pieces, padding) -> rows; the rows of every sequence."""
    got = {k: [] for k in TOTAL}
    for meta, pieces, pad in batches(dev):
        y, lo = fn(meta, pieces, pad), 0
        for k, _, n in pieces:
            got[k].append(y[lo:lo + n])
            lo += n
    return {k: torch.cat(v) for k, v in got.items()}


@pytest.mark.parametrize("dev,dtype", DEV_DTYPE)
@pytest.mark.parametrize("width", [8, 72, 77, 1024, 4104, 9008])
@pytest.mark.parametrize("first", ["embedding", "sum", "normed"])
def test_token_shift_behind_the_norm_over_portions_batches_and_reused_slots(dev, dtype, width, first):
    """The previous row comes from the batch, from the state, or is none; r' goes on unshifted in 32-bit."""
    eps, mult = 1e-3, 0.37
    w, shift, post = (_rand(dev, dtype, width, seed=s) * 0.5 for s in (1, 2, 3))
    rdt = dtype if first == "embedding" else F32
    res = {k: _rand(dev, rdt, n, width, seed=10 + n) * 3 for k, n in TOTAL.items()}
    y = {k: _rand(dev, dtype, n, width, seed=90 + n) * 5 for k, n in TOTAL.items()}
    state, sums, raws = torch.full((4, width), 5.0, device=dev), [], []

    def step(meta, pieces, pad):
        r0 = torch.cat([res[k][a:a + n] for k, a, n in pieces] + [res["a"][:pad]])
        y0 = None if first == "embedding" else torch.cat([y[k][a:a + n] for k, a, n in pieces] + [y["a"][:pad]])
        keep = r0.clone()
        h, r, raw = ops.add_rms_norm_shift(y0, r0, w, eps, 1.0, shift, state, meta, post if first == "normed" else None, mult, True)
        assert h.dtype == dtype and r.dtype == raw.dtype == F32 and torch.equal(r0, keep)
        sums.append((pieces, r))
        raws.append((pieces, raw))
        return h
    got = run_batches(dev, step)
    wd, sd, pd = (t.double().cpu() for t in (w, shift, post))
    for k in TOTAL:
        x = res[k].double().cpu()
        if first == "sum":
            x = x + mult * y[k].double().cpu()
        if first == "normed":
            x = x + mult * plain.rms(y[k].double().cpu(), eps) * pd
        h = plain.model_norm(x, wd, eps)
        _close(got[k], plain.token_shift(h, sd), dtype)
        for rows, want in ((sums, x), (raws, h)):
            for pieces, r in rows:
                lo = 0
                for kk, a, n in pieces:
                    if kk == k:
                        _close(r[lo:lo + n], want[a:a + n], F32)
                    lo += n
        if k != "b":
            _close(state[SLOT[k]], h[-1], F32)
    assert (state[1] == 5.0).all()
    before = state.clone()
    token_shift.advance(raws[0][1], state, state_meta(dev, [1, 2], [7, 9], [1, 3], 16, [[1], [1]]))
    assert torch.equal(state[1], raws[0][1][0]) and torch.equal(state[3], raws[0][1][2]) and torch.equal(state[0], before[0])


@pytest.mark.parametrize("dev,dtype", DEV_DTYPE)
@pytest.mark.parametrize("T,W", [(3, 72), (5, 77), (40, 1024)])
def test_small_steps_around_the_stream(dev, dtype, T, W):
    y, z, r = _rand(dev, dtype, T, W), _rand(dev, dtype, T, W, seed=1), _rand(dev, F32, T, W, seed=2) * 9
    w = _rand(dev, dtype, W, seed=4) * 0.3
    want = r.double().cpu() - 0.6 * y.double().cpu()
    h, r1 = ops.add_rms_norm(y, r.clone(), w, 1e-4, 1.0, mult=-0.6)
    _close(r1, want, F32)
    _close(h, plain.model_norm(want, w.double().cpu(), 1e-4), dtype)
    x, r2 = ops.residual_add(y, r.clone(), -0.6)
    assert x.dtype == dtype and r2.dtype == F32
    _close(r2, want, F32)
    assert torch.equal(x, r2.to(dtype))
    g = _rand(dev, F32, T, 9, seed=3) * 3
    _close(ops.add_gated(y, z, g[:, 4]), y.double().cpu() + plain.sigmoid(g[:, 4:5].double().cpu()) * z.double().cpu(), dtype)
    a = _rand(dev, dtype, T, W, seed=5) * 2
    b = a.clone()
    ops.tanh_(b[:, 8:32])
    _close(b[:, 8:32], torch.tanh(a[:, 8:32].double().cpu()), dtype)
    assert torch.equal(b[:, :8], a[:, :8]) and torch.equal(b[:, 32:], a[:, 32:])
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)                       # noqa: E731
    assert ops.resolve_tokens(i32([7, 59, 3, 0]), i32([-1, 2, -1, 0]), i32([50, 51, 52])).tolist() == [7, 52, 3, 50]


def rule_case(rule, dtype, dev, H, d, dv, tau=3.0, bias=(-1.0, 1.5), seed=0, per_head_norm=False):
    """(plan, columns of a row q | k | v | rates with padding between the parts)."""
    up = lambda n: (n + 7) // 8 * 8                                                      # noqa: E731
    k0 = up(H * d)
    v0, a0 = 2 * k0, 2 * k0 + up(H * dv)
    rnd = lambda *s, mean=0.0, scale=1.0, at=0: mean + _rand(dev, F32, *s, seed=seed + at, scale=scale)      # noqa: E731
    p = la.LinearAttentionPlan(H, H, d, dv, (0, k0, v0), "silu" if rule == "channel" else "sigmoid", 1e-5, q_mult=0.3, rule=rule,
                               tau=tau, norm_w=rnd(H * dv if per_head_norm else dv, at=1), dt_bias=rnd(H * d, mean=bias[0],
                               scale=bias[1], at=2), rate_offset=a0, rate_bias=rnd(H * d, at=3))
    return p, a0 + up(H * d)


def rule_plain(p, row, a, gate):
    """Plain result for one request from its first token on (fp64 on the CPU)."""
    H, d, dv = p.heads, p.dim, p.vdim
    c = lambda t: t.double().cpu()                                                       # noqa: E731
    q, k, v = (row[:, o:o + n].reshape(-1, H, n // H) for o, n in zip(p.offsets, (H * d, H * d, H * dv)))
    z = a + c(p.dt_bias)
    if p.rule == "channel":
        o, st = plain.gla_states(q * p.q_mult, k, v, plain.gla_decay(z, p.tau).reshape(-1, H, d))
    else:
        rate = plain.sigmoid(row[:, p.rate_offset:p.rate_offset + H * d] + c(p.rate_bias)).reshape(-1, H, d)
        o, st = plain.removal_states(q * p.q_mult, k, v, plain.removal_decay(z).reshape(-1, H, d), rate)
    n = c(p.norm_w).reshape(-1, dv) if p.norm_stride else c(p.norm_w)
    return (plain.rms(o, p.eps) * n).reshape(-1, H * dv) * (plain.silu if p.gate_act == "silu" else plain.sigmoid)(gate), st


RULES = [("channel", 3, 24, 40, {}), ("channel", 2, 64, 64, {"per_head_norm": True}), ("channel", 1, 10, 3, {"tau": 0.4}),
         ("channel", 2, 128, 200, {"tau": 16.0}), ("channel", 1, 256, 128, {}), ("channel", 1, 264, 12, {}),
         ("removal", 3, 32, 32, {}), ("removal", 2, 64, 64, {"per_head_norm": True}), ("removal", 2, 9, 9, {}),
         ("removal", 2, 128, 128, {}), ("removal", 1, 200, 72, {}), ("removal", 1, 256, 256, {}), ("removal", 1, 264, 12, {}),
         ("removal", 2, 48, 6, {"bias": (8.0, 6.0)})]


@pytest.mark.parametrize("dev,dtype", DEV_DTYPE)
@pytest.mark.parametrize("rule,H,d,dv,kw", RULES, ids=lambda v: str(v) if not isinstance(v, dict) else "-".join(v))
@pytest.mark.parametrize("strided", [False, True])
def test_carried_state_rules_over_portions_batches_and_reused_slots(dev, dtype, rule, H, d, dv, kw, strided):
    p, n = rule_case(rule, dtype, dev, H, d, dv, **kw)
    state = torch.full(p.state_shape(4), 5.0, device=dev)
    seq = {k: (_rand(dev, dtype, t, n, seed=20 + i), _rand(dev, dtype, t, H * d, seed=60 + i) * 2, _rand(dev, dtype, t, H * dv, seed=40 + i))
           for i, (k, t) in enumerate(TOTAL.items())}

    def step(meta, pieces, pad):
        row, a, gate = (torch.cat([seq[k][j][s:s + m] for k, s, m in pieces] + [seq["a"][j][:pad]]) for j in range(3))
        if not strided:
            return ops.carried_state_attention(p, row, a, gate, meta, (state,))
        wide = torch.full((row.shape[0], H * dv + 24), 3.0, dtype=dtype, device=dev)
        y = ops.carried_state_attention(p, row, a, gate, meta, (state,), wide[:, 16:16 + H * dv])
        assert y.data_ptr() == wide[:, 16:].data_ptr() and (wide[:, :16] == 3.0).all() and (wide[:, 16 + H * dv:] == 3.0).all()
        return y
    got = run_batches(dev, step)
    for k, (row, a, gate) in seq.items():
        want, st = rule_plain(p, *(t.double().cpu() for t in (row, a, gate)))
        err = ((got[k].double().cpu() - want).norm() / want.norm()).item()
        assert err < (5e-6 if dtype == F32 else 8e-3), (k, err)
        if k != "b":
            es = ((state[SLOT[k]].double().cpu() - st).norm() / st.norm()).item()
            assert es < (5e-6 if dtype == F32 else 4e-5), (k, es)
    assert (state[1] == 5.0).all()                        # a slot that nobody used


@pytest.mark.parametrize("dev,dtype", DEV_DTYPE)
@pytest.mark.parametrize("rule,tau,bias", [("channel", 0.2, -9.0), ("channel", 64.0, 14.0), ("removal", 1.0, -20.0), ("removal", 1.0, 20.0)])
def test_decays_at_their_ends(dev, dtype, rule, tau, bias):
    """Factors that forget a channel within a token, and factors of (nearly) one over a long prompt."""
    H, d, dv, T = 2, 32, 32, 150
    p, n = rule_case(rule, dtype, dev, H, d, dv, tau=tau, bias=(bias, 1.0))
    row, a, gate = _rand(dev, dtype, T, n, seed=1), _rand(dev, dtype, T, H * d, seed=3), _rand(dev, dtype, T, H * dv, seed=2)
    state = torch.zeros(p.state_shape(1), device=dev)
    y = ops.carried_state_attention(p, row, a, gate, state_meta(dev, [T], [0], [0], 16, [list(range(10))]), (state,))
    want, st = rule_plain(p, *(t.double().cpu() for t in (row, a, gate)))
    assert torch.isfinite(y).all()
    assert ((y.double().cpu() - want).norm() / want.norm()).item() < (3e-5 if dtype == F32 else 1e-2)
    assert ((state[0].double().cpu() - st).norm() / st.norm()).item() < 5e-5


@pytest.mark.gpu
@pytest.mark.parametrize("rule", ["channel", "removal"])
@pytest.mark.parametrize("chunks", [1, 5])
def test_prompts_in_several_slabs_on_two_streams(monkeypatch, rule, chunks):
    """A scratch of few chunks: states cross slabs in the pool, requests of unequal lengths end in different slabs."""
    from vllm_torchtpu_b200.ops import cuda, cuda_linear
    H, d, dv = 2, 64, 96
    per = cuda.lib().b200_linear_attention_chunk_bytes(d, dv, la.RULES.index(rule))
    monkeypatch.setattr(cuda_linear.slabs, "__defaults__", (chunks * H * per,))
    p, n = rule_case(rule, BF16, "cuda", H, d, dv)
    lens, slots = [150, 33, 2, 97], [2, 0, 3, 1]
    seq = [(_rand("cuda", BF16, t, n, seed=i), _rand("cuda", BF16, t, H * d, seed=i + 20), _rand("cuda", BF16, t, H * dv, seed=i + 40))
           for i, t in enumerate(lens)]
    state = torch.full(p.state_shape(4), 5.0, device="cuda")
    meta = state_meta("cuda", lens, [0] * 4, slots, 256, [[1]] * 4)
    y, at = ops.carried_state_attention(p, *(torch.cat(t) for t in zip(*seq)), meta, (state,)), 0
    for x, t, slot in zip(seq, lens, slots):
        want, st = rule_plain(p, *(v.double().cpu() for v in x))
        assert ((y[at:at + t].double().cpu() - want).norm() / want.norm()).item() < 8e-3
        assert ((state[slot].double().cpu() - st).norm() / st.norm()).item() < 4e-5
        at += t


@pytest.mark.parametrize("dev,dtype", DEV_DTYPE)
@pytest.mark.parametrize("H,G,D", [(4, 2, 64), (8, 2, 128), (6, 1, 128), (36, 1, 64), (3, 3, 36), (2, 1, 160)])
@pytest.mark.parametrize("chunk", [1, 16, 23, 64, 500])
def test_chunk_edges_over_pages(dev, dtype, H, G, D, chunk):
    """Each query points at the first key of its chunk or at the last one of the chunk before, in decoding, portions and
    prompts; a sink of 0; the output rows are strided."""
    lens, ctxs = [1, 1, 1, 2, 17, 70, 1], [16, chunk, 95, 2 * chunk - 1, 15, 0, 0]
    q, cache, meta, kv = paged_case(dev, dtype, lens, ctxs, H, G, D)
    at, group = 0, H // G
    for r, (n, c) in enumerate(zip(lens, ctxs)):
        for i in range(n):
            for h in range(H):
                j = (c + i) // chunk * chunk - 1 + h % 2                  # odd heads: the first key that is still seen
                k = kv[r][0]
                if j >= 0:
                    q[at + i, h] = (k[j, h // group] / k[j, h // group].norm() ** 2 * 9.0).to(dtype).to(dev)
        at += n
    T = q.shape[0]
    wide = torch.full((T, H * D + 16), 3.0, dtype=dtype, device=dev)
    sinks = torch.zeros(H, device=dev)
    ops.paged_attention(q, cache, meta, 1.0, sliding_window=-chunk, sinks=sinks, out=wide[:, :H * D])
    assert (wide[:, H * D:] == 3.0).all()
    plainly = ops.paged_attention(q, cache, meta, 1.0, sliding_window=-chunk, sinks=sinks)
    assert torch.equal(wide[:, :H * D], plainly.reshape(T, -1))
    got, at = wide[:, :H * D].double().cpu().reshape(T, H, D), 0
    for n, c, (k, v) in zip(lens, ctxs, kv):
        seen = plain.chunk_mask(c + n, chunk)[c:]
        for h in range(H):
            s = (q[at:at + n, h].double().cpu() @ k[:, h // group].t()).masked_fill(~seen, float("-inf"))
            _close(got[at:at + n, h], plain.sink_softmax(s) @ v[:, h // group], dtype, 3)
        at += n


@pytest.mark.parametrize("dev,dtype", DEV_DTYPE)
@pytest.mark.parametrize("H,G,d,dv,D,taps,dims", [(4, 2, 24, 40, 64, 4, 12), (6, 3, 64, 64, 64, 3, 64), (2, 1, 9, 11, 12, 2, 6),
                                                  (3, 1, 32, 16, 64, 6, 0)])
def test_factor_on_the_queries_of_a_head(dev, dtype, H, G, d, dv, D, taps, dims):
    T, up = 21, lambda n: (n + 7) // 8 * 8
    nq, nk, nv = H * d, G * d, G * dv
    off = (0, up(nq), up(nq) + up(nk))
    row = _rand(dev, dtype, T, up(nq) + up(nk) + up(nv))
    f = torch.linspace(-1.5, 2.0, H, device=dev)
    w = _rand(dev, dtype, taps, nq + nk + nv, seed=5)
    inv = ops.ref.rope_inv_freq(dims, 300.0).to(dev) if dims else None
    got = []
    for scale in (f, None):
        p = ConvAttentionPlan(H, G, d, dv, 1, D, off, taps, w, inv, 1.0, scale)
        cache = torch.zeros(4, 2, G, 16, D, dtype=dtype, device=dev)
        ring = torch.zeros(p.ring_shape(2), dtype=dtype, device=dev)
        q = ops.conv_and_cache(p, row, cache, ring, state_meta(dev, [T], [0], [1], 16, [[3, 1]]))
        got.append((q, cache))
    x = plain.short_conv(row[:, :nq].double().cpu(), w[:, :nq].double().cpu().t()).reshape(T, H, d)
    x = plain.rotate_pairs(x, {"dims": dims, "base": 300.0}) if dims else x
    _close(got[0][0][..., :d], x * f.double().cpu()[:, None], dtype)
    _close(got[1][0][..., :d], x, dtype)
    assert torch.equal(got[0][1], got[1][1])              # keys and values are left alone


@pytest.mark.parametrize("dev,dtype", DEV_DTYPE)
@pytest.mark.parametrize("T,width,dim,first", [(1, 72, 20, 20), (70, 64, 24, 0), (300, 512, 256, 256), (9, 21, 5, 10),
                                               (64, 4096, 256, 512), (3, 2048, 100, 0)])
def test_gate_from_a_row_of_the_token_table(dev, dtype, T, width, dim, first):
    V = 50
    x, w, table = _rand(dev, dtype, T, width), _rand(dev, dtype, dim, width, seed=1) / math.sqrt(width) * 2, _rand(dev, dtype, V, 3 * dim + first, seed=2)
    ids = torch.tensor([(7 * t + 3) % V for t in range(T)], dtype=torch.int32, device=dev)
    want = plain.gelu_tanh(x.double().cpu() @ w.double().cpu().t()) * table.double().cpu()[ids.long().cpu(), first:first + dim]
    _close(ops.gemm_token_gate(x, w, table, first, ids), want, dtype)


@pytest.mark.parametrize("dev,dtype", DEV_DTYPE)
@pytest.mark.parametrize("T,width,ff,limit", [(3, 40, 24, 0.5), (70, 64, 136, 2.0), (300, 128, 200, 1.0), (9, 21, 13, 7.0),
                                              (40, 2048, 64, 1.5), (600, 256, 128, 0.7)])
def test_clamped_gate_and_up_projection(dev, dtype, T, width, ff, limit):
    x, w = _rand(dev, dtype, T, width), _rand(dev, dtype, 2 * ff, width, seed=1) / math.sqrt(width) * 2
    got = ops.gemm_gated(x, w, f"swigluoai:1.702:{limit}")
    wd, eye = w.double().cpu(), torch.eye(ff, dtype=torch.float64)
    want = plain.expert(x.double().cpu(), {"gate": wd[:ff], "up": wd[ff:], "down": eye}, "", limit)
    _close(got, want, dtype)


@pytest.mark.parametrize("dev,dtype", DEV_DTYPE)
@pytest.mark.parametrize("T,width,E,top,count,keep,ff,shared", [
    (1, 40, 8, 2, 4, 2, 24, 16), (33, 72, 6, 3, 3, 2, 40, 56), (300, 128, 16, 4, 4, 3, 128, 128), (9, 21, 5, 3, 5, 4, 13, 7),
    (64, 256, 128, 6, 8, 4, 192, 320), (40, 1024, 8, 8, 2, 2, 128, 64), (50, 64, 12, 1, 1, 1, 32, 24)])
def test_experts_in_groups_with_a_shared_one(dev, dtype, T, width, E, top, count, keep, ff, shared):
    """Corrections that make choice scores negative: experts of dropped groups must not come back as zeros."""
    from vllm_torchtpu_b200.models.qwen3_moe import MoEBlock
    mlp = moe(E, top, ff, 1.2, count, keep, 1.9, shared, 0.8)
    spec = ModelConfig.from_hf_dict(config([(gla(), mlp)], width=width)).layer_specs[0].experts
    cfg = ModelConfig(hidden_size=width, num_experts=E, num_experts_per_tok=top, moe_intermediate_size=ff, hidden_act=spec.act,
                      moe_scoring="sigmoid", moe_score_bias=True, moe_n_group=count, moe_topk_group=keep, moe_router_fp32=True,
                      moe_routed_scaling=1.9, num_shared_experts=1, shared_expert_intermediate_size=shared, shared_expert_gate=True,
                      shared_expert_act=spec.shared_act, dtype=dtype)
    b = MoEBlock("m", cfg, dev, None)
    rnd = lambda *s, seed: _rand("cpu", BF16, *s, seed=seed) / math.sqrt(s[-1])          # noqa: E731
    w = {"router": rnd(E, width, seed=1) * 2, "shared.sg": rnd(1, width, seed=2), "correction": _rand("cpu", BF16, E, seed=4) * 0.4 - 1.5}
    b.experts.gate.load_weight(torch.cat([w["router"], w["shared.sg"]]))
    b.experts.score_bias.copy_(w["correction"])
    for e in range(E):
        w |= {f"e{e}.gate": rnd(ff, width, seed=10 + e), f"e{e}.up": rnd(ff, width, seed=300 + e), f"e{e}.down": rnd(width, ff, seed=600 + e)}
        b.experts.load_gated(e, *(w[f"e{e}.{n}"] for n in ("gate", "up", "down")))
    w |= {"shared.gate": rnd(shared, width, seed=7), "shared.up": rnd(shared, width, seed=8), "shared.down": rnd(width, shared, seed=9)}
    b.shared.gate_up.load_weight(torch.cat([w["shared.gate"], w["shared.up"]]))
    b.shared.down.load_weight(w["shared.down"])
    x = _rand("cpu", BF16, T, width, seed=3).to(dtype).to(dev)
    wd, xd = {k: v.double() for k, v in w.items()}, x.double().cpu()
    want = plain.feed_forward(xd, wd, "", mlp)
    res = _rand(dev, F32, T, width, seed=5) * 3
    rd = res.double().cpu()
    rounded, total = b.forward_add(x, res.clone())
    assert rounded.dtype == dtype and total.dtype == F32 and torch.equal(rounded, total.to(dtype))
    for got in (b.forward(x).double().cpu(), total.double().cpu() - rd):
        e = (got - want).norm(dim=-1) / want.norm(dim=-1)
        if dtype == F32:
            assert e.max() < 2e-5, e.max()
        else:                                             # close calls of the router aside
            assert e.sort().values[int(0.95 * (T - 1))] < 2e-2, e
    if dtype == F32:
        ids, wt = b.experts.route(x)
        pi, pw = plain.route(xd, wd, "", mlp["router"])
        assert (ids.cpu().sort(-1).values == pi.sort(-1).values).all()
        assert ((wt.double().cpu().sum(-1) - 1.9).abs() < 1e-5).all()
    assert (plain.feed_forward(xd, wd, "", mlp, no_shared=True) - want).abs().max() > 1e-2


# ------------------------------------------------------------------------------------------------- the model
@pytest.mark.parametrize("dev", DEVS)
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(MODELS))
def test_prompt_portions_and_single_tokens_match_the_plain_model(tmp_path, dev, dtype, name):
    cfg = MODELS[name]
    if name == "wide" and dev == "cpu":
        pytest.skip("sizes for the tensor-core kernels")
    w = write_model(str(tmp_path), cfg, seed=11)
    toks = tokens_of(83, cfg["vocab"], 1)
    want = plain.forward(cfg, w, toks)
    rep = make_replay(str(tmp_path), dtype, 128, dev)
    for cuts in ([83], [50] + [1] * 33, portions(83, [2, 3]), portions(83, [15, 2, 16, 1, 17, 31])):
        assert_like(replay_logits(rep, toks, cuts), want, dtype, cuts)
    if name == "mixed":
        assert_like(replay_logits(rep, toks, [1] * 83), want, dtype)


@pytest.mark.parametrize("dev", DEVS)
def test_residual_stream_after_every_layer(tmp_path, dev):
    """32-bit layer by layer, so that two mistakes cannot make up for each other."""
    w = write_model(str(tmp_path), MIXED, seed=9)
    toks = tokens_of(41, MIXED["vocab"], 4)
    want: list = []
    plain.forward(MIXED, w, toks, layers_out=want)
    rep = make_replay(str(tmp_path), "float32", 64, dev)
    got = []
    for layer in rep.engine.runner.model.layers:
        fwd = layer.forward

        def spy(*a, fwd=fwd):
            y, post, r = fwd(*a)
            got.append(r.double().cpu() + plain.rms(y.double().cpu(), MIXED["norm"]["eps"]) * post.double().cpu())
            return y, post, r
        layer.forward = spy
    replay_logits(rep, toks, [41])
    assert len(got) == len(want) == len(MIXED["layers"])
    for g, e in zip(got, want):
        assert (g - e).abs().max() < 5e-5 * e.abs().max()


@pytest.mark.parametrize("dev", DEVS)
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_mixed_batches_reused_pages_and_slots_match_each_request_alone(tmp_path, dev, dtype):
    cfg = MIXED
    w = write_model(str(tmp_path), cfg, seed=11)
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
def test_far_keys_chunk_edges_states_sinks_and_shifts_decide_logits(tmp_path, dev):
    """Each mistake that is planted in the plain model moves its logits far; the engine stays with the unspoilt model, in
    prompts, in portions and in decoding."""
    cfg = config([(par(chunk=110, conv=4, scale=0.6), moe()), (gla(tau=30.0), None),
                  (par(chunk=41, scale=0.6, conv=2, ls=0.5, rs=0.6), None)])
    w = write_model(str(tmp_path), cfg, seed=2)
    toks = tokens_of(130, cfg["vocab"], 3)
    want = plain.forward(cfg, w, toks)
    rep = make_replay(str(tmp_path), "float32", 192, dev)
    for cuts in ([97, 2] + [1] * 31, portions(130, [2, 5]), [130], portions(130, [33, 37, 1])):
        assert logit_error(replay_logits(rep, toks, cuts), want) < LIMIT["float32"] * 5, cuts
    left = [{"lost_key": k} for k in (0, 1, 15, 16, 31, 32, 63, 64, 96, 97)] + [{"edge": 1}, {"edge": 109}]
    left += [{"no_sink": True}, {"no_temp": True}] + [{"conv_cut": p} for p in (1, 16, 97, 99, 100)]
    plants = [{0: {"left": x}} for x in left] + [{2: {"left": {"edge": e}}} for e in (1, 40)]
    plants += [{i: {"right": x}} for i in (0, 2) for x in ({"no_removal": True}, {"forget_at": 1}, {"forget_at": 97}, {"forget_at": 120})]
    plants += [{1: {"forget_at": p}} for p in (1, 16, 97, 99)] + [{1: {"no_decay": True}}]
    plants += [{i: {"shift": {"forget_at": p}}} for i in (0, 1, 2) for p in (1, 2, 97, 99, 129)]
    plants += [{i: {"side": False}} for i in (0, 1, 2)] + [{0: {"ff": {"no_shared": True}}}]
    for plant in plants:
        wrong = plain.forward(cfg, w, toks, plant=plant)
        assert logit_error(wrong, want) > 30 * LIMIT["float32"], plant


@pytest.mark.parametrize("dev", DEVS)
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_first_tokens_of_a_sequence_after_a_slot_was_used(tmp_path, dev, dtype):
    w = write_model(str(tmp_path), MIXED, seed=1)
    rep = make_replay(str(tmp_path), dtype, 64, dev)
    for n in (1, 2, 3, 5, 1):
        toks = tokens_of(n, MIXED["vocab"], n)
        want = plain.forward(MIXED, w, toks)
        for cuts in ([n], [1] * n):
            assert_like(replay_logits(rep, toks, cuts), want, dtype, factor=2.0 if dtype == "bfloat16" else 1.0)


@pytest.mark.parametrize("dev", DEVS)
@pytest.mark.parametrize("kw", [{}, {"async_scheduling": True}, {"enforce_eager": True},
                                {"enable_prefix_caching": True}, {"num_gpu_blocks_override": 12},
                                {"speculative_config": {"method": "ngram", "num_speculative_tokens": 3}}],
                         ids=lambda k: next(iter(k), "default"))
def test_greedy_generation_through_the_engine(tmp_path, dev, kw):
    """``LLM.generate`` in 32-bit: chunked prompts (40-token steps), batches of unequal requests, long decoding over chunk
    edges, a pool small enough to preempt (states start over), rejected drafts (states are rolled back), tokens that the host
    has not read yet, against the plain model."""
    from vllm_torchtpu_b200.engine.llm import LLM
    cfg = config([(par(conv=4), moe()), (gla(), None), (par(chunk=30, conv=2, ls=1.0), moe(6, 3, 32, count=3, keep=2))])
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
        assert (top - z[torch.arange(n_out), torch.tensor(ids)] <= 2e-4).all()      # ties aside, the greedy path
    if kw.get("num_gpu_blocks_override") == 12:
        assert llm.engine.scheduler.stats["preemptions"] > 0
    if "speculative_config" in kw:
        assert llm.engine.runner.stats.get("spec_drafted", 0) > 0
    if "enable_prefix_caching" in kw:                     # a prefix has no state to continue from: never reused
        assert llm.generate([prompts[3]], sp)[0].outputs[0].token_ids == outs[3].outputs[0].token_ids
        assert llm.engine.scheduler.stats.get("prefix_hit_tokens", 0) == 0


@pytest.mark.parametrize("dev", DEVS)
def test_rejected_drafts_leave_every_state_as_it_was(tmp_path, dev):
    """Verification steps whose drafts are all wrong, half right and right: neither a convolution, nor a token shift, nor a
    carried state may see a rejected token."""
    from vllm_torchtpu_b200.engine.llm import LLM
    cfg = config([(par(conv=6), None), (gla(), None), (par(conv=1), moe())])
    w = write_model(str(tmp_path), cfg, seed=8)
    prompt = tokens_of(6, cfg["vocab"], 5) * 4            # the n-gram drafter proposes the repetition, the model differs
    llm = LLM(str(tmp_path), device=dev, dtype="float32", max_num_seqs=2, max_model_len=128, init_dist=False,
              num_gpu_blocks_override=32, speculative_config={"method": "ngram", "num_speculative_tokens": 5})
    ids = llm.generate([prompt], SamplingParams(temperature=0.0, max_tokens=40, ignore_eos=True))[0].outputs[0].token_ids
    assert llm.engine.runner.stats.get("state_rollbacks", 0) > 0
    z = plain.forward(cfg, w, prompt + list(ids[:-1]))[len(prompt) - 1:]
    assert (z.max(-1).values - z[torch.arange(40), torch.tensor(ids)] <= 2e-4).all()


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
    """HBM budget with states, graphs of several buckets, 300 decoded tokens."""
    from vllm_torchtpu_b200.engine.llm import LLM
    w = write_model(str(tmp_path), MIXED, seed=4)
    llm = LLM(str(tmp_path), device="cuda", max_num_seqs=4, max_model_len=512, gpu_memory_utilization=0.05, init_dist=False)
    p = tokens_of(20, MIXED["vocab"], 1)
    ids = llm.generate([p], SamplingParams(temperature=0.0, max_tokens=300, ignore_eos=True))[0].outputs[0].token_ids
    z = plain.forward(MIXED, w, p + list(ids[:-1]))[len(p) - 1:]
    short = z.max(-1).values - z[torch.arange(300), torch.tensor(ids)]
    assert short.sort().values[int(0.95 * 299)] < 0.2 * z.std()      # the arg-max up to bf16 rounding (and close calls)


# ------------------------------------------------------------------------------------------------- surroundings
def test_configuration_reads_every_size_and_refuses_what_is_not_built():
    mc = ModelConfig.from_hf_dict(MIXED, "m")
    assert mc.architecture == "vipolix" and mc.num_layers == 5 and mc.vocab_size == 211 and not mc.tie_word_embeddings
    assert mc.rms_norm_eps == 3e-6 and mc.token_side_dim == 20 and mc.has_recurrent_state and mc.is_moe and not mc.is_mla
    s = mc.layer_specs
    assert all(x.token_shift and x.side_dim == 20 for x in s) and [x.mixer.recurrent for x in s] == [True, False, True, False, False]
    assert s[0].mixer.tau == 9.0 and s[2].mixer.tau == 1.0 and (s[0].mixer.heads, s[0].mixer.dim, s[0].mixer.vdim) == (3, 24, 40)
    m = s[1].mixer
    assert (m.left_scale, m.right_scale, m.right.heads, m.right.dim) == (0.7, -0.4, 3, 16)
    assert (m.left.chunk, m.left.window, m.left.mask, m.left.conv, m.left.scale) == (19, None, -19, 3, 0.3)
    assert m.left.rot.dims == 12 and m.left.rot.base == 900.0 and m.left.bias and m.left.head_temp and m.left.zero_sink
    e = s[1].experts
    assert (e.experts, e.top, e.ff, e.groups, e.keep, e.scale, e.shared_ff) == (6, 3, 56, 3, 2, 1.7, 40)
    assert e.act == "swigluoai:1.702:1.5" and e.shared_act == "swigluoai:1.702:0.9" and s[2].experts is None
    bad = [("type", lambda c: c["layers"][0].update(type="other")),
           ("feed-forward", lambda c: c["layers"][1]["mlp"].update(kind="dense")),
           ("rot.dims", lambda c: c["layers"][1]["mixer"]["left"]["rot"].update(dims=26)),
           ("top", lambda c: c["layers"][0]["mlp"]["router"].update(top=5)),
           ("groups", lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=3)),
           ("tau", lambda c: c["layers"][0]["mixer"].update(tau=0)),
           ("tap", lambda c: c["layers"][1]["mixer"]["left"].update(conv=0)),
           ("chunk", lambda c: c["layers"][1]["mixer"]["left"]["mask"].update(size=0)),
           ("divide", lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=3))]
    for what, change in bad:
        c = json.loads(json.dumps(MIXED))
        change(c)
        with pytest.raises(ValueError, match=what):
            ModelConfig.from_hf_dict(c)
    for kw in (dict(parallel=ParallelConfig(tensor_parallel_size=4)), dict(parallel=ParallelConfig(pipeline_parallel_size=2)),
               dict(speculative={"method": "mtp"}), dict(kv_transfer={"kv_connector": "B200HostConnector"}),
               dict(cache=CacheConfig(kv_cache_dtype="fp8")), dict(parallel=ParallelConfig(prefill_context_parallel_size=2))):
        with pytest.raises(ValueError):
            EngineConfig(model=ModelConfig.from_hf_dict(MIXED), device="cpu", **kw).finalize()


def test_caches_hold_the_states_and_pages_of_every_layer(tmp_path):
    write_model(str(tmp_path), MIXED)
    r = make_replay(str(tmp_path), "float32", 64, "cpu").engine.runner
    m, c = r.model, r.kv_caches
    assert all(x[0].shape == (5, 72) and x[0].dtype == F32 for x in c)
    assert c[0][1][0].shape == (5, 3, 24, 40) and c[0][1][0].dtype == F32
    ring, pages, state = c[1][1]
    assert ring.shape == (5, 3, 4 * 24 + 2 * 24 + 2 * 20) and pages.shape == (5, 2, 2, 16, 24) and state.shape == (5, 3, 16, 16)
    assert m.kv_bytes_per_block(16, F32) == (2 * 2 * 24 + 2 * 1 * 40 + 2 * 2 * 24) * 16 * 4
    n = sum(p.numel() for p in random_model(MIXED).values())
    vectors = sum(p.numel() for k, p in random_model(MIXED).items() if p.dim() == 1 or k.endswith(".conv"))
    assert abs(m.weight_bytes() / 4 - (n - vectors)) < 0.2 * n       # padding of the packed parts and of the heads aside


def test_incomplete_checkpoints_are_refused_and_weights_can_be_replaced(tmp_path):
    from safetensors.torch import save_file
    cfg = config([(par(), moe(4, 2, 16, count=2, keep=1)), (gla(), None)])
    w = write_model(str(tmp_path / "a"), cfg, seed=0)
    w2 = random_model(cfg, seed=1)
    write_model(str(tmp_path / "b"), cfg)
    for lost in ("l0.mix.left.k.conv", "l0.mlp.e2.down", "side.embed", "l1.mix.a2.b", "l0.mix.right.w0", "l0.shift", "l1.side.norm"):
        save_file({k: v for k, v in w.items() if k != lost}, str(tmp_path / "b" / "model.safetensors"))
        with pytest.raises(ValueError, match=lost):
            make_replay(str(tmp_path / "b"), "float32", 64, "cpu")
    rep = make_replay(str(tmp_path / "a"), "float32", 64, "cpu")
    toks = tokens_of(9, cfg["vocab"])
    part = {k: w2[k] for k in w2 if k in ("embed", "side.embed", "final.norm", "l0.mlp.router", "l0.mlp.shared.sg", "l0.norm2") or
            k.startswith(("l1.mix.", "l0.mlp.e1.", "l0.side.")) or k.endswith((".conv", "shift"))}
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


@pytest.mark.parametrize("mode", ["tp", "ep"])
def test_two_ranks_match_one(mode):
    """Sharded heads, convolutions, states and experts (tensor parallel), experts by rank (expert parallel)."""
    from test_parallel_cpu import _run
    assert _run(2, mode, "tiny-vipolix") == _run(1, "tp", "tiny-vipolix")


def test_server_command_line_builds_the_engine(tmp_path):
    import argparse

    from vllm_torchtpu_b200.entrypoints import cli
    write_model(str(tmp_path), MIXED)
    ap = argparse.ArgumentParser()
    cli.add_engine_args(ap)
    llm = cli.make_llm(ap.parse_args([str(tmp_path), "--device", "cpu", "--max-num-seqs", "2", "--max-model-len", "64"]))
    assert type(llm.engine.runner.model).__name__ == "VipolixForCausalLM"
    out = llm.generate([[1, 2, 3]], SamplingParams(max_tokens=4, temperature=0.7, top_p=0.9, logprobs=2))
    assert len(out[0].outputs[0].token_ids) == 4
    assert model_preset("tiny-vipolix").architecture == "vipolix"
