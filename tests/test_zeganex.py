"""Zeganex (differential attention, or rotated attention with an output gate, both behind short convolutions and with a
sliding window; bigram embedding; dense and expert feed-forwards) against the plain statement in ``plain_zeganex.py``:
every mechanism alone, then the model through the engine's scheduler, caches and kernels."""
import copy
import json
import math
import os
import subprocess

import numpy as np
import plain_zeganex as plain
import pytest
import torch
from test_mazivik import BF16, DEV_DTYPE, DEVS, F32, ROOT, _close, _rand, logit_error, portions, replay_logits, tokens_of
from test_popanex import paged_case

from vllm_torchtpu_b200 import SamplingParams, ops
from vllm_torchtpu_b200.config import CacheConfig, EngineConfig, ModelConfig, ParallelConfig, model_preset
from vllm_torchtpu_b200.entrypoints.trace_replay import make_replay
from vllm_torchtpu_b200.ops.short_conv import ConvAttentionPlan
from vllm_torchtpu_b200.runner.attn_metadata import AttentionMetadata

LIMIT = {"float32": 2e-5, "bfloat16": 5e-2}


def assert_like(got, want, dtype, what="", factor=1.0):
    """Every position in 32-bit.  In bf16 nine of ten: rounding may move a token across a close call of the router, to an
    expert with other opinions."""
    d = got.double() - want.double()
    e = (d - d.mean(-1, keepdim=True)).pow(2).mean(-1).sqrt() / want.double().pow(2).mean().sqrt()
    if dtype == "float32":
        assert e.max() < LIMIT[dtype] * factor, (what, e.max())
    else:
        assert e.sort().values[int(0.9 * (len(e) - 1))] < LIMIT[dtype] * factor and e.max() < 1.5, (what, e)


# ------------------------------------------------------------------------------------------------- configurations
def diff(heads=4, kv_heads=2, dim=20, vdim=28, conv=3, window=19, lam=0.45, scale=0.25, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "mask": {"size": window},
         "scale": scale, "diff": lam}
    return {"type": "attention", "mixer": m if kv_from is None else dict(m, kv_from=kv_from)}


def gated(heads=6, kv_heads=3, dim=24, vdim=16, conv=4, window=33, scale=0.22, dims=12, base=900.0, factor=3.0, original=50):
    return {"type": "attention_2", "mixer": {
        "heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "mask": {"size": window}, "scale": scale,
        "rot": {"base": base, "dims": dims, "scaling": {"factor": factor, "fast": 8.0, "slow": 0.5, "original": original}}}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts=7, top=2, ff=24):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}


def config(layers, width=72, vocab=211, eps=3e-6, mult=0.6, buckets=151, mul_prev=37, mul_cur=11):
    return {"architecture": "Zeganex", "width": width, "vocab": vocab, "norm": {"eps": eps}, "residual_mult": mult,
            "embedding": {"bigram": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}},
            "layers": [dict(copy.deepcopy(layer), mlp=mlp) for layer, mlp in layers]}


MIXED = config([(diff(), moe()), (gated(), dense(88)), (diff(kv_from=0, conv=2, window=40, scale=0.3, lam=0.2), None),
                (gated(heads=2, kv_heads=1, dim=16, vdim=40, conv=1, window=5, dims=16), moe(4, 3, 56)),
                (diff(heads=3, kv_heads=3, dim=12, vdim=24, conv=5, window=16), moe(3, 1, 16))])
MODELS = {
    "mixed": MIXED,
    "all_sizes_odd": config([(diff(heads=3, kv_heads=1, dim=7, vdim=5, conv=2, window=6), moe(5, 5, 11)),
                             (gated(heads=2, kv_heads=2, dim=9, vdim=13, conv=3, window=7, dims=6), dense(13)),
                             (diff(heads=3, kv_heads=1, dim=7, vdim=5, conv=4, window=11, kv_from=0), moe(2, 1, 9))],
                            width=21, vocab=37, mult=1.0, buckets=1, mul_prev=1, mul_cur=1),
    "wide_windows": config([(diff(window=64), None), (gated(window=1000, dim=64, vdim=64, dims=32), None),
                            (gated(window=1, conv=6), dense(40))], mult=0.35),
    "one_kv_head": config([(diff(heads=18, kv_heads=1, dim=16, vdim=32, window=23), dense(40)),
                           (gated(heads=20, kv_heads=1, dim=32, vdim=48, window=17, dims=8), None)], width=96),
    "wide": config([(diff(heads=8, kv_heads=4, dim=64, vdim=128, conv=4, window=40, scale=0.125), moe(8, 2, 128)),
                    (gated(heads=16, kv_heads=4, dim=128, vdim=128, conv=3, window=50, scale=0.08, dims=64), dense(448)),
                    (diff(heads=8, kv_heads=4, dim=64, vdim=128, conv=2, window=24, scale=0.125, kv_from=0), moe(8, 3, 192)),
                    (gated(heads=4, kv_heads=2, dim=160, vdim=144, window=31, scale=0.08), None)], width=256, vocab=1000),
}


def random_model(cfg, seed=0, gain=1.0):
    """Weights of ``cfg`` (bfloat16), scaled so that activations stay of order one."""
    g = torch.Generator().manual_seed(seed)

    def rnd(*s, scale=1.0, mean=0.0):
        return (mean + torch.randn(*s, generator=g) * scale).bfloat16()

    def mat(o, i, k=1.0):
        return rnd(o, i, scale=k * gain / math.sqrt(i))
    W, b = cfg["width"], cfg["embedding"]["bigram"]
    w = {"embed": rnd(cfg["vocab"], W, scale=0.7), "bigram": rnd(b["buckets"] + 1, W, scale=0.7),
         "final.norm": rnd(W, mean=1.0, scale=0.3)}
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}.mix."
        maps = 2 if layer["type"] == "attention" else 1
        H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        for n in ["norm1", "norm1b"] + (["norm2", "norm2b"] if layer["mlp"] else []):
            w[f"l{i}.{n}"] = rnd(W, mean=1.0, scale=0.3)
        for n, c in (("q", H * maps * d), ("k", G * maps * d), ("v", G * dv)):
            if n == "q" or m.get("kv_from") is None:
                w[p + n], w[p + n + ".b"] = mat(c, W), rnd(c, scale=0.5)
                w[p + n + ".conv"] = rnd(c, m["conv"], scale=0.7)
        w[p + "o"] = mat(W, H * dv)
        if maps == 2:
            for n in ("lq1", "lk1", "lq2", "lk2"):
                w[p + n] = rnd(d, scale=0.5 / d ** 0.25)
        else:
            w[p + "g"], w[p + "o.b"] = mat(H * dv, W, 2.0), rnd(W, scale=0.5)
        f = layer["mlp"]
        if f and f["kind"] == "dense":
            w[f"l{i}.mlp.gate"], w[f"l{i}.mlp.up"], w[f"l{i}.mlp.down"] = mat(f["ff"], W), mat(f["ff"], W), mat(W, f["ff"])
        elif f:
            w[f"l{i}.mlp.router"] = mat(f["router"]["experts"], W, 2.0)
            for e in range(f["router"]["experts"]):
                w[f"l{i}.mlp.e{e}.up"], w[f"l{i}.mlp.e{e}.down"] = mat(f["expert"]["ff"], W), mat(W, f["expert"]["ff"])
    return w


def write_model(path, cfg, seed=0, gain=1.0, edit=None):
    from safetensors.torch import save_file
    w = random_model(cfg, seed, gain)
    if edit:
        edit(w)
    os.makedirs(path, exist_ok=True)
    save_file({k: v.contiguous() for k, v in w.items()}, os.path.join(path, "model.safetensors"))
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    return w


# ------------------------------------------------------------------------------------------------- mechanisms
@pytest.mark.parametrize("dev,dtype", DEV_DTYPE)
@pytest.mark.parametrize("width", [8, 72, 77, 1024, 4104])
def test_normalised_output_joins_the_32_bit_stream(dev, dtype, width):
    """r + m * norm_b(y), then the norm in front of the next sublayer."""
    y, w, post = _rand(dev, dtype, 5, width) * 7, _rand(dev, dtype, width, seed=1), _rand(dev, dtype, width, seed=4)
    eps = 1e-3
    for res in (_rand(dev, dtype, 5, width, seed=2), _rand(dev, F32, 5, width, seed=3) * 30):
        if dtype == F32 and res.dtype != F32:
            continue
        want = res.double().cpu() + 0.37 * plain.rms(y.double().cpu(), eps) * post.double().cpu()
        keep = res.clone()
        h, none = ops.add_rms_norm(y, keep, w, eps, update=False, post=post, mult=0.37)
        assert none is None and torch.equal(keep, res)
        h2, r = ops.add_rms_norm(y, keep, w, eps, post=post, mult=0.37)
        assert r.dtype == F32 and h.dtype == dtype and torch.equal(h, h2)
        _close(r, want, F32)
        _close(h, plain.rms(want, eps) * w.double().cpu(), dtype)
        h0, _ = ops.add_rms_norm(None, res.clone(), w, eps, post=post, mult=0.37)       # nothing to add yet
        _close(h0, plain.rms(res.double().cpu(), eps) * w.double().cpu(), dtype)


@pytest.mark.parametrize("dev,dtype", DEV_DTYPE)
@pytest.mark.parametrize("width,bigram", [(64, (97, 29, 13)), (21, (5, 3, 2)), (40, (1, 1, 1)),
                                          (64, (1009, 2147483629, 2147483587))])
def test_bigram_embedding(dev, dtype, width, bigram):
    """First tokens, pairs, tokens and previous tokens that are still on the device, products beyond 32 bits."""
    V, B = 60, bigram[0]
    table, pairs = _rand(dev, dtype, V, width), _rand(dev, dtype, B + 1, width, seed=1)
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)                       # noqa: E731
    last_tokens, last_inputs = i32([50, 51, 52, 53]), i32([40, 41, 42, 43])
    ids, prev, src = i32([7, 59, 3, 0, 0, 9]), i32([-1, 58, 59, -2, 5, -2]), i32([-1, -1, -1, 2, 0, -1])
    got = ops.embedding_pairs(ids, prev, table, pairs, bigram, src, last_tokens, last_inputs)
    assert got.dtype == F32
    b = dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))
    cur, before = [7, 59, 3, 52, 50, 9], [None, 58, 59, 42, 5, None]
    for t in range(6):
        want = table[cur[t]].double().cpu() + pairs[plain.bigram_row(before[t], cur[t], b)].double().cpu()
        _close(got[t], want, F32)
    assert last_inputs.tolist() == [50, 41, 52, 43]       # what the next step's previous token will be


def state_meta(dev, lens, starts, slots, bs, tables, padded=0):
    """Ragged batch with pages and state slots; ``padded``: more requests and rows without content behind."""
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)                       # noqa: E731
    qsl = np.concatenate([[0], np.cumsum(lens)]).tolist()
    pos = [s + i for n, s in zip(lens, starts) for i in range(n)]
    smap = [tables[r][(s + i) // bs] * bs + (s + i) % bs for r, (n, s) in enumerate(zip(lens, starts)) for i in range(n)]
    nd = 0
    while nd < len(lens) and lens[nd] == 1 and starts[nd] > 0:
        nd += 1
    width, R = max(len(t) for t in tables), len(lens)
    return AttentionMetadata(
        i32(pos + [0] * padded), i32(smap + [-1] * padded), i32([t + [0] * (width - len(t)) for t in tables] + [[0] * width] * padded),
        i32([a + b for a, b in zip(lens, starts)] + [0] * padded), i32(qsl + [qsl[-1]] * padded), R, qsl[-1],
        num_decode_reqs=nd, max_query_len=max(lens), max_seq_len=999, state_slots=i32(slots + [-1] * padded),
        query_start_loc_cpu=torch.tensor(qsl), padded_num_reqs=R + padded if padded else None)


CONVS = [dict(heads=3, kv_heads=3, dim=24, vdim=40, maps=1, width=64, taps=4, dims=12),
         dict(heads=4, kv_heads=2, dim=20, vdim=28, maps=2, width=64, taps=3),
         dict(heads=4, kv_heads=2, dim=64, vdim=128, maps=2, width=128, taps=4),
         dict(heads=2, kv_heads=1, dim=128, vdim=96, maps=1, width=128, taps=2, dims=128),
         dict(heads=2, kv_heads=1, dim=9, vdim=11, maps=1, width=12, taps=3, dims=6),
         dict(heads=3, kv_heads=1, dim=7, vdim=5, maps=2, width=16, taps=6),
         dict(heads=2, kv_heads=2, dim=16, vdim=16, maps=1, width=64, taps=1, dims=4),
         dict(heads=2, kv_heads=1, dim=32, vdim=64, maps=1, width=64, taps=7, dims=32),
         dict(heads=4, kv_heads=0, dim=24, vdim=32, maps=2, width=64, taps=3),
         dict(heads=3, kv_heads=0, dim=5, vdim=8, maps=1, width=12, taps=2, dims=2)]


@pytest.mark.parametrize("dev,dtype", DEV_DTYPE)
@pytest.mark.parametrize("c", CONVS, ids=lambda c: "-".join(str(v) for v in c.values()))
def test_convolution_rotation_and_cache_over_portions_batches_and_reused_slots(dev, dtype, c):
    """Four sequences whose portions meet in ragged batches; a slot comes back with another sequence's leftovers."""
    H, G, d, dv, maps, D, taps = (c[k] for k in ("heads", "kv_heads", "dim", "vdim", "maps", "width", "taps"))
    scaling = {"factor": 2.5, "original": 40, "fast": 6.0, "slow": 0.5}
    rot = {"dims": c["dims"], "base": 300.0, "scaling": scaling} if c.get("dims") else None
    up = lambda n: (n + 7) // 8 * 8                                                      # noqa: E731
    nq, nk, nv = H * maps * d, G * maps * d, G * dv
    off = (0, up(nq), up(nq) + up(nk)) if G else (0, 0, 0)
    n = up(nq) + up(nk) + up(nv) + 8
    w = _rand(dev, dtype, taps, nq + nk + nv, seed=5)
    inv = mult = None
    if rot:
        from vllm_torchtpu_b200.layer_specs import RotarySpec
        rs = RotarySpec(rot["dims"], rot["base"], scaling).rope_scaling
        inv, mult = ops.ref.rope_inv_freq(rot["dims"], rot["base"], rs).to(dev), ops.ref.rope_attention_factor(rs)
    p = ConvAttentionPlan(H, G, d, dv, maps, D, off, taps, w, inv, mult or 1.0)
    bs, pages = 16, 10
    ring = torch.full(p.ring_shape(4), 5.0, dtype=dtype, device=dev)
    cache = torch.full((pages, 2, max(G, 1), bs, D), 9.0, dtype=dtype, device=dev)
    total = {"a": 61, "b": 19, "c": 3, "e": 40}
    tables = {"a": [3, 7, 1, 8], "b": [2, 5], "c": [9], "e": [5, 4, 2]}
    slot_of = {"a": 2, "b": 0, "c": 3, "e": 0}            # e takes b's slot and pages
    seq = {k: _rand(dev, dtype, t, n, seed=20 + i) for i, (k, t) in enumerate(total.items())}
    got, at = {k: [] for k in seq}, dict.fromkeys(seq, 0)
    steps = [[("a", 1), ("b", 2)], [("b", 1), ("a", 15)], [("a", 1), ("c", 3), ("b", 16)], [("a", 33), ("e", 17)],
             [("a", 1), ("e", 1)], [("e", 22), ("a", 2)], [("a", 8)]]
    for step in steps:
        lens, starts = [x for _, x in step], [at[k] for k, _ in step]
        pad = 2 if all(x == 1 and s > 0 for x, s in zip(lens, starts)) else 0
        meta = state_meta(dev, lens, starts, [slot_of[k] for k, _ in step], bs, [tables[k] for k, _ in step], pad)
        row = torch.cat([seq[k][at[k]:at[k] + x] for k, x in step] + [_rand(dev, dtype, pad, n)])
        q = ops.conv_and_cache(p, row, cache, ring, meta)
        lo = 0
        for k, x in step:
            got[k].append(q[lo:lo + x])
            lo += x
            at[k] += x
    assert at == total and (ring[1] == 5.0).all()
    for k, x in seq.items():
        x = x.double().cpu()
        wd = w.double().cpu().t()
        q = plain.short_conv(x[:, :nq], wd[:nq]).reshape(-1, H * maps, d)
        q = plain.rotate_pairs(q, rot) if rot else q
        g = torch.cat(got[k]).reshape(-1, H, maps, D)
        for m in range(maps):
            _close(g[:, :, m, m * d:(m + 1) * d], q.reshape(-1, H, maps, d)[:, :, m], dtype)
            rest = torch.cat([g[:, :, m, :m * d], g[:, :, m, (m + 1) * d:]], -1)
            assert (rest == 0).all()
        if G and k != "b":
            key = plain.short_conv(x[:, off[1]:off[1] + nk], wd[nq:nq + nk]).reshape(-1, G * maps, d)
            key = (plain.rotate_pairs(key, rot) if rot else key).reshape(-1, G, maps * d)
            val = plain.short_conv(x[:, off[2]:off[2] + nv], wd[nq + nk:]).reshape(-1, G, dv)
            c_ = cache[tables[k]].permute(1, 0, 3, 2, 4).reshape(2, -1, G, D)[:, :total[k]]
            _close(c_[0, ..., :maps * d], key, dtype)
            _close(c_[1, ..., :dv], val, dtype)
            assert (c_[0, ..., maps * d:] == 0).all() and (c_[1, ..., dv:] == 0).all()
    assert (cache[[0, 6]] == 9.0).all() and (G or (cache == 9.0).all())
    # replay of rows into the rings alone, as after rejected drafts
    if taps > 1:
        ring2 = ring.clone()
        ops.conv_ring_update(p, seq["c"], ring2, state_meta(dev, [3], [50], [1], bs, [[0] * 4]))
        for pos in range(53 - min(taps, 3), 53):
            row = torch.cat([seq["c"][pos - 50, o:o + s] for o, s in zip(off, (nq, nk, nv)) if s])
            assert torch.equal(ring2[1, pos % taps], row)
        assert torch.equal(ring2[[0, 2, 3]], ring[[0, 2, 3]])


@pytest.mark.parametrize("dev,dtype", DEV_DTYPE)
@pytest.mark.parametrize("H,D,vdim", [(3, 64, 64), (4, 128, 96), (2, 64, 7), (5, 16, 13), (2, 160, 144), (1, 512, 500)])
def test_difference_of_maps_and_output_gate(dev, dtype, H, D, vdim):
    T, eps = 9, 1e-2
    pad = lambda t: torch.nn.functional.pad(t, (0, D - vdim))                            # noqa: E731
    a, lam = pad(_rand(dev, dtype, T, 2 * H, vdim)), torch.tensor([0.63], device=dev)
    row = _rand(dev, dtype, T, H * vdim + 16, seed=2) * 2
    gate = row[:, 8:8 + H * vdim]
    x = a.double().cpu().reshape(T, H, 2, D)[..., :vdim]
    want = plain.combine_maps(x[:, :, 0], x[:, :, 1], lam.double().cpu(), 0.2, eps)
    got = ops.combine_heads(a, vdim, None, lam, 0.2, eps)
    _close(got[..., :vdim], want, dtype)
    assert got.shape == (T, H, D) and (got[..., vdim:] == 0).all()
    g = plain.sigmoid(gate.double().cpu()).reshape(T, H, vdim)
    _close(ops.combine_heads(a, vdim, gate, lam, 0.2, eps)[..., :vdim], want * g, dtype)
    one = a[:, :H].contiguous()
    want1 = one.double().cpu()[..., :vdim] * g
    _close(ops.combine_heads(one, vdim, gate)[..., :vdim], want1, dtype)


@pytest.mark.parametrize("dev,dtype", DEV_DTYPE)
@pytest.mark.parametrize("H,G,D", [(4, 2, 64), (8, 2, 128), (6, 1, 128), (36, 1, 64), (3, 3, 36), (2, 1, 160)])
@pytest.mark.parametrize("window", [1, 16, 23, 64])
def test_window_edges_over_pages(dev, dtype, H, G, D, window):
    """Keys just inside and just outside the window in decoding, portions and prompts: each query is made to point at the
    one or the other, so that a window that is one key off decides the result."""
    lens, ctxs = [1, 1, 1, 2, 17, 70, 1], [16, window, 95, 31, 15, 0, 0]
    q, cache, meta, kv = paged_case(dev, dtype, lens, ctxs, H, G, D)
    scale, at, group = 1.0, 0, H // G
    for r, (n, c) in enumerate(zip(lens, ctxs)):
        for i in range(n):
            for h in range(H):
                j = c + i - window + h % 2 + (1 if window == 1 else 0)       # odd heads: the last key that is still seen
                k = kv[r][0]
                if 0 <= j < len(k):
                    t = k[j, h // group] / k[j, h // group].norm() ** 2 * 9.0
                    q[at + i, h] = t.to(dtype).to(dev)
        at += n
    got, at = ops.paged_attention(q, cache, meta, scale, sliding_window=window).double().cpu(), 0
    for n, c, (k, v) in zip(lens, ctxs, kv):
        for h in range(H):
            s = torch.stack([k[:, h // group] @ q[at + i, h].double().cpu() for i in range(n)]) * scale
            mask = plain.visible(c + n, window)[c:]
            _close(got[at:at + n, h], plain.softmax_rows(s, mask) @ v[:, h // group], dtype, 3)
        at += n


@pytest.mark.parametrize("dev,dtype", DEV_DTYPE)
@pytest.mark.parametrize("H,G,D,vdim", [(2, 1, 64, 40), (8, 2, 128, 128), (8, 2, 128, 72), (2, 2, 128, 100), (16, 2, 128, 96),
                                        (12, 2, 128, 128), (20, 1, 128, 64), (4, 2, 36, 33)])
@pytest.mark.parametrize("maps", [1, 2])
@pytest.mark.parametrize("gated_", [False, True])
def test_attention_finished_in_its_epilogue(dev, dtype, H, G, D, vdim, maps, gated_):
    """Decoded tokens (in a batch of their own, too), portions and prompts: difference of the maps, norm and gate."""
    if maps == 2 and (H // G) % 2:
        pytest.skip("a head's maps belong to one key head")
    eps, scale = 1e-3, 0.3
    for lens, ctxs in (([1, 1, 1, 2, 17, 150], [16, 95, 300, 31, 15, 0]), ([1, 1, 1], [15, 40, 700]), ([1, 33], [0, 100])):
        q, cache, meta, kv = paged_case(dev, dtype, lens, ctxs, H, G, D)
        cache[:, 1, :, :, vdim:] = 0
        T, heads = q.shape[0], H // maps
        wide = _rand(dev, dtype, T, heads * vdim + 16, seed=3) * 2
        gate = wide[:, 8:8 + heads * vdim] if gated_ else None
        lam = torch.tensor([0.71], device=dev) if maps == 2 else None
        got = ops.paged_attention_heads(q, cache, meta, scale, 50, vdim, gate, lam, 0.3, eps)
        assert got.shape == (T, heads, D) and (got[..., vdim:] == 0).all()
        at = 0
        for n, c, (k, v) in zip(lens, ctxs, kv):
            mask = plain.visible(c + n, 50)[c:]
            a = torch.stack([plain.softmax_rows(q[at:at + n, h].double().cpu() @ k[:, h // (H // G)].t() * scale, mask)
                             @ v[:, h // (H // G), :vdim] for h in range(H)], 1)
            if maps == 2:
                a = plain.combine_maps(a[:, 0::2], a[:, 1::2], lam.double().cpu(), 0.3, eps)
            if gated_:
                a = a * plain.sigmoid(gate[at:at + n].double().cpu()).reshape(n, heads, vdim)
            _close(got[at:at + n, :, :vdim], a, dtype, 2)
            at += n


@pytest.mark.parametrize("dev,dtype", DEV_DTYPE)
@pytest.mark.parametrize("T,width,E,top,ff", [(1, 40, 5, 2, 24), (33, 72, 7, 3, 40), (300, 128, 16, 4, 128),
                                              (9, 21, 3, 3, 13), (64, 256, 130, 1, 200), (40, 2048, 8, 2, 192)])
def test_router_and_ungated_experts(dev, dtype, T, width, E, top, ff):
    from vllm_torchtpu_b200.layers.moe import FusedMoE
    cfg = ModelConfig(hidden_size=width, num_experts=E, num_experts_per_tok=top, moe_intermediate_size=ff, hidden_act="relu2",
                      moe_renormalize=False, moe_router_fp32=True, dtype=dtype)
    m = FusedMoE("m", cfg, dev)
    rnd = lambda *s, seed: _rand("cpu", BF16, *s, seed=seed) / math.sqrt(s[-1])          # noqa: E731
    w = {"router": rnd(E, width, seed=1) * 2}
    for e in range(E):
        w[f"e{e}.up"], w[f"e{e}.down"] = rnd(ff, width, seed=10 + e), rnd(width, ff, seed=500 + e)
        m.load_ungated(e, w[f"e{e}.up"], w[f"e{e}.down"])
    m.gate.load_weight(w["router"])
    x = _rand("cpu", BF16, T, width, seed=3).to(dtype).to(dev)
    wd = {k: v.double() for k, v in w.items()}
    want = plain.experts(x.double().cpu(), wd, "", {"router": {"top": top}})
    got = m.forward(x)
    assert got.dtype == dtype
    e = (got.double().cpu() - want).norm(dim=-1) / want.norm(dim=-1)
    if dtype == F32:
        assert e.max() < 2e-5, e.max()
    else:                                                 # close calls of the router aside
        assert e.sort().values[int(0.95 * (T - 1))] < 2e-2, e
    ids, wt = m.route(x)
    chosen = plain.router(x.double().cpu(), wd["router"], top)
    for t in range(0, T, 7):                              # weights are the scores themselves, not renormalised
        assert abs(wt[t].sum().item() - sum(float(s) for _, s in chosen[t])) < 1e-4
        if dtype == F32:
            assert set(ids[t].tolist()) == {i for i, _ in chosen[t]}


def test_frequencies_follow_the_scaling():
    from vllm_torchtpu_b200.layer_specs import RotarySpec
    for dims, base, s in ((16, 900.0, {"factor": 3.0, "original": 50, "fast": 8.0, "slow": 0.5}),
                          (64, 1e6, {"factor": 16.0, "original": 4096, "fast": 32.0, "slow": 1.0}),
                          (4, 10.0, {"factor": 2.0, "original": 7, "fast": 1.0, "slow": 1.0}), (24, 5e4, None)):
        r = RotarySpec(dims, base, s)
        f, mult = plain.frequencies({"dims": dims, "base": base, "scaling": s})
        _close(ops.ref.rope_inv_freq(dims, base, r.rope_scaling), torch.tensor(f, dtype=torch.float64), F32, 0.01)
        assert abs(ops.ref.rope_attention_factor(r.rope_scaling) - mult) < 1e-12


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
            got.append(r.double().cpu() + MIXED["residual_mult"] * plain.rms(y.double().cpu(), MIXED["norm"]["eps"])
                       * post.double().cpu())
            return y, post, r
        layer.forward = spy
    replay_logits(rep, toks, [41])
    assert len(got) == len(want) == len(MIXED["layers"])
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
def test_far_keys_window_edges_maps_gates_pairs_and_convolutions_decide_logits(tmp_path, dev):
    """Each mistake that is planted in the plain model moves its logits far; the engine stays with the unspoilt model, in
    prompts, in portions and in decoding."""
    cfg = config([(diff(window=70, conv=4, scale=0.6), None), (gated(window=41, scale=0.6), dense(48)),
                  (diff(kv_from=0, window=33, scale=0.6, conv=2), None)])
    w = write_model(str(tmp_path), cfg, seed=2)
    toks = tokens_of(130, cfg["vocab"], 3)
    want = plain.forward(cfg, w, toks)
    rep = make_replay(str(tmp_path), "float32", 192, dev)
    for cuts in ([97, 2] + [1] * 31, portions(130, [2, 5]), [130], portions(130, [33, 37, 1])):
        assert logit_error(replay_logits(rep, toks, cuts), want) < LIMIT["float32"] * 5, cuts
    plants = [{0: {"lost_key": k}} for k in (0, 1, 15, 16, 31, 32, 63, 64, 96, 97)]
    plants += [{0: {"window": n}} for n in (69, 71)] + [{1: {"window": n}} for n in (40, 42)]
    plants += [{2: {"window": n}} for n in (32, 34, 70)]
    plants += [{0: {"one_map": True}}, {2: {"one_map": True}}, {1: {"no_gate": True}}]
    plants += [{i: {"conv_cut": p}} for i in (0, 1, 2) for p in (1, 16, 97, 99, 100)]
    for plant in plants:
        wrong = plain.forward(cfg, w, toks, plant=plant)
        assert logit_error(wrong, want) > 30 * LIMIT["float32"], plant
    for p in (1, 2, 97, 99, 129):                         # the token in front of a portion's first is forgotten
        assert logit_error(plain.forward(cfg, w, toks, forget_at=(p,)), want) > 100 * LIMIT["float32"]


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
    """``LLM.generate`` in 32-bit: chunked prompts (40-token steps), batches of unequal requests, long decoding past every
    window, a pool small enough to preempt (states start over), rejected drafts (rings are rolled back), tokens and
    previous tokens that the host has not read yet, against the plain model."""
    from vllm_torchtpu_b200.engine.llm import LLM
    cfg = config([(diff(conv=4), moe()), (gated(window=24), dense(64)), (diff(kv_from=0, conv=2, window=30), None)])
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
    if "enable_prefix_caching" in kw:                     # a prefix has no convolution inputs to continue from: never reused
        assert llm.generate([prompts[3]], sp)[0].outputs[0].token_ids == outs[3].outputs[0].token_ids
        assert llm.engine.scheduler.stats.get("prefix_hit_tokens", 0) == 0


@pytest.mark.parametrize("dev", DEVS)
def test_rejected_drafts_leave_the_rings_as_they_were(tmp_path, dev):
    """Verification steps whose drafts are all wrong, half right and right: the convolutions of what follows must not see
    a rejected token."""
    from vllm_torchtpu_b200.engine.llm import LLM
    cfg = config([(diff(conv=6), None), (gated(conv=3), dense(40))])
    w = write_model(str(tmp_path), cfg, seed=8)
    base = tokens_of(6, cfg["vocab"], 5)
    prompt = base * 4                                     # the n-gram drafter proposes the repetition, the model differs
    llm = LLM(str(tmp_path), device=dev, dtype="float32", max_num_seqs=2, max_model_len=128, init_dist=False,
              num_gpu_blocks_override=32, speculative_config={"method": "ngram", "num_speculative_tokens": 5})
    ids = llm.generate([prompt], SamplingParams(temperature=0.0, max_tokens=40, ignore_eos=True))[0].outputs[0].token_ids
    st = llm.engine.runner.stats
    assert st.get("state_rollbacks", 0) > 0
    z = plain.forward(cfg, w, prompt + list(ids[:-1]))[len(prompt) - 1:]
    assert (z.max(-1).values - z[torch.arange(40), torch.tensor(ids)] <= 1e-4).all()


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
    """HBM budget with rings, graphs of several buckets, 300 decoded tokens."""
    from vllm_torchtpu_b200.engine.llm import LLM
    w = write_model(str(tmp_path), MIXED, seed=4)
    llm = LLM(str(tmp_path), device="cuda", max_num_seqs=4, max_model_len=512, gpu_memory_utilization=0.05, init_dist=False)
    p = tokens_of(20, MIXED["vocab"], 1)
    ids = llm.generate([p], SamplingParams(temperature=0.0, max_tokens=300, ignore_eos=True))[0].outputs[0].token_ids
    z = plain.forward(MIXED, w, p + list(ids[:-1]))[len(p) - 1:]
    short = z.max(-1).values - z[torch.arange(300), torch.tensor(ids)]
    assert short.sort().values[int(0.98 * 299)] < 0.1 * z.std()      # the arg-max up to bf16 rounding (and close calls)


# ------------------------------------------------------------------------------------------------- surroundings
def test_configuration_reads_every_size_and_refuses_what_is_not_built():
    mc = ModelConfig.from_hf_dict(MIXED, "m")
    assert mc.architecture == "zeganex" and mc.num_layers == 5 and mc.vocab_size == 211 and mc.tie_word_embeddings
    assert mc.bigram == (151, 37, 11) and mc.residual_mult == 0.6 and mc.rms_norm_eps == 3e-6
    assert [s.ff for s in mc.layer_specs] == [0, 88, 0, 0, 0] and mc.has_recurrent_state and mc.is_moe and not mc.is_mla
    assert [(s.experts.experts, s.experts.top, s.experts.ff) if s.experts else None for s in mc.layer_specs] == \
        [(7, 2, 24), None, None, (4, 3, 56), (3, 1, 16)]
    mix = [s.mixer for s in mc.layer_specs]
    assert [m.maps for m in mix] == [2, 1, 2, 1, 2] and [m.window for m in mix] == [19, 33, 40, 5, 16]
    assert [m.conv for m in mix] == [3, 4, 2, 1, 5] and mix[2].kv_from == 0 and mix[2].diff == 0.2
    assert mix[1].rot.dims == 12 and mix[1].rot.scaling["original"] == 50 and mix[0].rot is None
    assert mix[1].output_gate and mix[1].out_bias and not mix[0].output_gate and not mix[0].out_bias
    bad = [("type", lambda c: c["layers"][0].update(type="other")),
           ("feed-forward", lambda c: c["layers"][1]["mlp"].update(kind="other")),
           ("kv_from", lambda c: c["layers"][2]["mixer"].update(kv_from=3)),
           ("differ", lambda c: c["layers"][2]["mixer"].update(kv_from=1)),
           ("rot.dims", lambda c: c["layers"][1]["mixer"]["rot"].update(dims=26)),
           ("experts", lambda c: c["layers"][0]["mlp"]["router"].update(top=8)),
           ("tap", lambda c: c["layers"][0]["mixer"].update(conv=0)),
           ("divide", lambda c: c["layers"][1]["mixer"].update(kv_heads=4))]
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


def test_shared_keys_and_values_are_cached_once(tmp_path):
    write_model(str(tmp_path), MIXED)
    r = make_replay(str(tmp_path), "float32", 64, "cpu").engine.runner
    m, c = r.model, r.kv_caches
    assert c[2][1] is c[0][1] and c[2][0].shape == (5, 2, 4 * 2 * 20) and c[0][0].shape == (5, 3, 2 * (4 * 20 + 2 * 20) + 2 * 28)
    assert c[0][1].shape == (5, 2, 2, 16, 40) and c[1][1].shape == (5, 2, 3, 16, 24)
    per_token = 2 * 2 * 40 + 2 * 3 * 24 + 2 * 1 * 40 + 2 * 3 * 24
    assert m.kv_bytes_per_block(16, torch.float32) == per_token * 16 * 4
    assert m.lm_head is m.embed
    tables = 4 * 72 * (211 + 152)                         # embedding (the head as well) and pairs, counted once
    assert m.weight_bytes() == tables + sum(l.self_attn.weight_bytes() + l.mlp.weight_bytes() for l in m.layers)


def test_incomplete_checkpoints_are_refused_and_weights_can_be_replaced(tmp_path):
    from safetensors.torch import save_file
    cfg = config([(diff(), moe(3, 2, 16)), (gated(), None)])
    w = write_model(str(tmp_path / "a"), cfg, seed=0)
    w2 = random_model(cfg, seed=1)
    write_model(str(tmp_path / "b"), cfg)
    for lost in ("l0.mix.k.conv", "l0.mlp.e2.down", "bigram", "l1.mix.o.b"):
        save_file({k: v for k, v in w.items() if k != lost}, str(tmp_path / "b" / "model.safetensors"))
        with pytest.raises(ValueError, match=lost):
            make_replay(str(tmp_path / "b"), "float32", 64, "cpu")
    rep = make_replay(str(tmp_path / "a"), "float32", 64, "cpu")
    toks = tokens_of(9, cfg["vocab"])
    part = {k: w2[k] for k in w2 if k in ("embed", "bigram", "final.norm", "l0.mlp.router", "l0.norm2b", "l1.mix.o.b") or
            k.startswith("l0.mix.l") or k.startswith("l0.mlp.e1.") or k.endswith((".conv", ".b"))}
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
    """Sharded heads, convolutions, biases and experts (tensor parallel), experts by rank (expert parallel)."""
    from test_parallel_cpu import _run
    assert _run(2, mode, "tiny-zeganex") == _run(1, "tp", "tiny-zeganex")


def test_server_command_line_builds_the_engine(tmp_path):
    import argparse

    from vllm_torchtpu_b200.entrypoints import cli
    write_model(str(tmp_path), MIXED)
    ap = argparse.ArgumentParser()
    cli.add_engine_args(ap)
    llm = cli.make_llm(ap.parse_args([str(tmp_path), "--device", "cpu", "--max-num-seqs", "2", "--max-model-len", "64"]))
    assert type(llm.engine.runner.model).__name__ == "ZeganexForCausalLM"
    out = llm.generate([[1, 2, 3]], SamplingParams(max_tokens=4, temperature=0.7, top_p=0.9, logprobs=2))
    assert len(out[0].outputs[0].token_ids) == 4
    assert model_preset("tiny-zeganex").architecture == "zeganex"
