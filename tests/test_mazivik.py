"""Mazivik (latent attention configured per layer) against the plain statement in ``plain_mazivik.py``: every
mechanism alone, then the model through the engine's scheduler, cache and kernels."""
import json
import math
import os
import subprocess
import sys

import numpy as np
import plain_mazivik as plain
import pytest
import torch

from vllm_torchtpu_b200 import SamplingParams, ops
from vllm_torchtpu_b200.config import EngineConfig, LatentMixerSpec, ModelConfig, ParallelConfig, model_preset
from vllm_torchtpu_b200.entrypoints.trace_replay import make_replay
from vllm_torchtpu_b200.runner.attn_metadata import AttentionMetadata

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DEVS = ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)]
F32, BF16 = torch.float32, torch.bfloat16
BOTH = [(d, t) for d in ("cpu", "cuda") for t in (F32, BF16)]
DEV_DTYPE = [pytest.param(d, t, marks=[pytest.mark.gpu] if d == "cuda" else [], id=f"{d}-{str(t)[6:]}") for d, t in BOTH]
TOL = {F32: 2e-5, BF16: 2e-2}


def _rand(dev, dtype, *shape, seed=0, scale=1.0):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(*shape, generator=g) * scale).to(dtype).to(dev)


def _close(got, want, dtype, scale=1.0):
    err = (got.double().cpu() - want.double().cpu()).abs().max().item()
    ref = want.double().abs().max().item()
    assert err <= TOL[dtype] * max(ref, 1e-3) * scale, (err, ref)


# ------------------------------------------------------------------------------------------------- configurations
def mixer(heads=3, dim=24, rot_dim=16, vdim=20, q_rank=40, kv_rank=48, scale=None, base=7000.0, scaling=True, **kw):
    rot = {"base": base, "dims": rot_dim}
    if scaling is True:
        rot["scaling"] = {"factor": 3.0, "original": 96, "fast": 20.0, "slow": 1.5}
    elif scaling:
        rot["scaling"] = scaling
    return {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
            "scale": scale if scale is not None else (dim + rot_dim) ** -0.5, "rot": rot, **kw}


def config(layers, width=72, vocab=211, cap=17.0, eps=3e-6):
    return {"architecture": "Mazivik", "width": width, "vocab": vocab, "norm": {"eps": eps}, "logit_softcap": cap,
            "layers": [{"type": "latent_attention", "mixer": m, "mlp": {"kind": "dense", "ff": ff} if ff else None}
                       for m, ff in layers]}


def shared_config(**kw):
    """Two owners, each serving another layer besides itself; unequal sizes."""
    a, b = mixer(**kw), mixer(heads=2, kv_rank=64, rot_dim=8, dim=16, vdim=32, q_rank=24, base=500.0)
    return config([(a, 88), (dict(b), 56), (dict(a, kv_from=0, heads=4, dim=16, vdim=12, scale=0.3, q_rank=56), 0),
                   (dict(b, kv_from=1), 104)])


def write_model(path, cfg, seed=0, gain=1.0, edit=None):
    from safetensors.torch import save_file
    w = plain.random_model(cfg, seed, gain)
    if edit:
        edit(w)
    os.makedirs(path, exist_ok=True)
    save_file({k: v.contiguous() for k, v in w.items()}, os.path.join(path, "model.safetensors"))
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    return w


def tokens_of(n, vocab, seed=0):
    return np.random.RandomState(seed).randint(0, vocab, size=n).tolist()


def logit_error(got, want):
    """Root mean square of the difference of mean-free logits over the root mean square of the logits."""
    d = got.double() - want.double()
    d = d - d.mean(-1, keepdim=True)
    return (d.pow(2).mean(-1).sqrt() / want.double().pow(2).mean().sqrt()).max().item()


LIMIT = {"float32": 2e-5, "bfloat16": 3e-2}


# ------------------------------------------------------------------------------------------------- mechanisms
@pytest.mark.parametrize("dev,dtype", DEV_DTYPE)
@pytest.mark.parametrize("width", [8, 72, 77, 1024, 4104])
def test_layer_norm_and_residual_add(dev, dtype, width):
    x = _rand(dev, dtype, 5, width) * 3 + 1.5
    w, eps = _rand(dev, dtype, width, seed=1), 1e-3
    got = ops.layer_norm(x, w, eps)
    _close(got, plain.layer_norm(x.double().cpu(), w.double().cpu(), eps), dtype)
    for res in (_rand(dev, dtype, 5, width, seed=2), _rand(dev, F32, 5, width, seed=3) * 30):
        if dtype == F32 and res.dtype != F32:
            continue
        want = res.double().cpu() + plain.layer_norm(x.double().cpu(), w.double().cpu(), eps)
        h, r = ops.layer_norm_add(x, res.clone(), w, eps)
        assert r.dtype == F32 and h.dtype == dtype
        _close(r, want, F32)                              # the stream is 32-bit whatever the model's dtype
        _close(h, want, dtype)
    # a large common offset: the variance is that of the deviations
    x = (_rand(dev, F32, 3, width) + 100.0)
    _close(ops.layer_norm(x, w.float(), eps), plain.layer_norm(x.double().cpu(), w.double().cpu(), eps), F32, 20)


@pytest.mark.parametrize("dev", DEVS)
def test_final_norm_of_the_32_bit_stream_and_softcap(dev):
    x, w = _rand(dev, F32, 4, 96) * 10, _rand(dev, BF16, 96, seed=1)
    got = ops.layer_norm(x, w, 1e-6)
    assert got.dtype == BF16
    _close(got, plain.layer_norm(x.double().cpu(), w.double().cpu(), 1e-6), BF16)
    for dtype in (F32, BF16):
        z = _rand(dev, dtype, 3, 333) * 40
        want = plain.softcap(z.double().cpu(), 12.5)
        got = ops.softcap(z, 12.5)
        assert got.dtype == F32
        _close(got, want, F32)


@pytest.mark.parametrize("scaling", [None, {"factor": 4.0, "original": 128, "fast": 32.0, "slow": 1.0},
                                     {"factor": 1.0, "original": 4096, "fast": 32.0, "slow": 1.0},
                                     {"factor": 8.0, "original": 40, "fast": 8.0, "slow": 2.0},
                                     {"factor": 2.5, "original": 7, "fast": 64.0, "slow": 48.0},
                                     {"factor": 2.0, "original": 10 ** 9, "fast": 4.0, "slow": 4.0}])
@pytest.mark.parametrize("dims,base", [(32, 10000.0), (16, 300.0), (2, 50.0)])
def test_rotary_frequencies(scaling, dims, base):
    spec = LatentMixerSpec.from_dict(mixer(rot_dim=dims, base=base, scaling=scaling))
    freqs, mult = plain.rotary_frequencies({"dims": dims, "base": base, "scaling": scaling})
    got = ops.ref.rope_inv_freq(spec.rot.dims, spec.rot.base, spec.rot.rope_scaling)
    torch.testing.assert_close(got.double(), torch.tensor(freqs, dtype=torch.float64), rtol=1e-6, atol=0)
    assert abs(ops.ref.rope_attention_factor(spec.rot.rope_scaling) - mult) < 1e-12
    if scaling:
        assert abs(mult - (0.1 * math.log(scaling["factor"]) + 1)) < 1e-12


@pytest.mark.parametrize("dev,dtype", DEV_DTYPE)
@pytest.mark.parametrize("Q,L,R,dims", [(40, 48, 16, 16), (33, 57, 6, 6), (24, 512, 64, 64), (16, 24, 12, 8)])
def test_latent_prep_norms_rotates_and_stores(dev, dtype, Q, L, R, dims):
    rot = {"dims": dims, "base": 900.0, "scaling": {"factor": 4.0, "original": 64, "fast": 16.0, "slow": 1.0}}
    spec = LatentMixerSpec.from_dict(mixer(q_rank=Q, kv_rank=L, rot_dim=R) | {"rot": rot})
    T, nb, bs, eps, Dc = 7, 4, 16, 1e-4, (L + R + 15) // 16 * 16
    row = _rand(dev, dtype, T, Q + L + R + 13)
    wq, wc = _rand(dev, dtype, Q, seed=1), _rand(dev, dtype, L, seed=2)
    pos = torch.tensor([0, 1, 5, 63, 64, 1000, 12345], dtype=torch.int32, device=dev)
    slots = torch.tensor([3, 16, 63, -1, 0, 31, 47], dtype=torch.int32, device=dev)
    inv = ops.ref.rope_inv_freq(dims, rot["base"], spec.rot.rope_scaling).to(dev)
    mult = ops.ref.rope_attention_factor(spec.rot.rope_scaling)
    cache = torch.full((nb, bs, Dc), 7.0, dtype=dtype, device=dev)
    cq = ops.latent_prep(row, wq, wc, cache, slots, pos, inv, mult, eps, L, R)
    r = row.double().cpu()
    _close(cq, plain.rms_norm(r[:, :Q], wq.double().cpu(), eps), dtype)
    c = plain.rms_norm(r[:, Q:Q + L], wc.double().cpu(), eps)
    k = plain.rotate_pairs(r[:, Q + L:Q + L + R], pos.tolist(), rot)
    flat, seen = cache.view(nb * bs, Dc).cpu(), set(slots.tolist()) - {-1}
    for t, s in enumerate(slots.tolist()):
        if s >= 0:
            _close(flat[s, :L], c[t], dtype)
            # fp32 angles: position * frequency rounds in its last bit
            _close(flat[s, L:L + R], k[t], dtype, 60 if dtype == F32 else 1)
            assert (flat[s, L + R:] == 7).all()
    assert (flat[[s for s in range(nb * bs) if s not in seen]] == 7).all()
    before = cache.clone()
    cq2 = ops.latent_prep(row, wq, None, cache, slots, pos, inv, mult, eps, L, R)      # a layer that shares a cache
    assert torch.equal(cq2, cq) and torch.equal(cache, before)


@pytest.mark.parametrize("dev,dtype", DEV_DTYPE)
def test_rotation_of_query_heads_into_padded_rows(dev, dtype):
    T, H, nope, R, L, W = 6, 3, 10, 12, 20, 48
    rot = {"dims": 8, "base": 100.0, "scaling": {"factor": 2.0, "original": 32, "fast": 8.0, "slow": 1.0}}
    rs = LatentMixerSpec.from_dict(mixer(rot_dim=R) | {"rot": rot}).rot.rope_scaling
    q, out = _rand(dev, dtype, T, H, nope + R), torch.full((T, H, W), 5.0, dtype=dtype, device=dev)
    pos = torch.tensor([0, 3, 4, 100, 101, 999], dtype=torch.int32, device=dev)
    ops.rope_heads_into(q, out, nope, R, L, pos, ops.ref.rope_inv_freq(8, 100.0, rs).to(dev),
                        ops.ref.rope_attention_factor(rs))
    _close(out[..., L:L + R], plain.rotate_pairs(q[..., nope:].double().cpu(), pos.tolist(), rot), dtype, 20)
    assert (out[..., :L] == 5).all() and (out[..., L + R:] == 0).all()


@pytest.mark.parametrize("dev,dtype", DEV_DTYPE)
@pytest.mark.parametrize("T,N,K", [(1, 80, 80), (5, 33, 19), (64, 200, 96), (130, 128, 640), (1100, 264, 72), (32, 96, 4096)])
def test_gelu_projection(dev, dtype, T, N, K):
    x, w = _rand(dev, dtype, T, K), _rand(dev, dtype, N, K, seed=1, scale=K ** -0.5)
    want = plain.gelu_erf(x.double().cpu() @ w.double().cpu().t())
    _close(ops.gemm_gelu(x, w), want, dtype)
    for cap in (0.0, 1.5):
        z = x.double().cpu() @ w.double().cpu().t()
        got = ops.gemm_softcap(x, w, cap)
        assert got.dtype == F32
        _close(got, plain.softcap(z, cap) if cap else z, F32)
    _close(ops.gemm(x, w), x.double().cpu() @ w.double().cpu().t(), dtype)


@pytest.mark.parametrize("dev,dtype", DEV_DTYPE)
@pytest.mark.parametrize("T,H,N,K,extra", [(1, 3, 48, 24, 16), (7, 5, 20, 48, 0), (33, 2, 130, 64, 32), (70, 4, 40, 9, 3),
                                           (300, 6, 128, 96, 8)])
def test_head_products_with_and_without_gate(dev, dtype, T, H, N, K, extra):
    x, w = _rand(dev, dtype, T, H, K + extra), _rand(dev, dtype, H, N, K, seed=1, scale=K ** -0.5)
    rows = _rand(dev, dtype, T, 11 + H * N, seed=2, scale=2.0)
    gate = rows[:, 11:]
    want = torch.einsum("thk,hnk->thn", x[..., :K].double().cpu(), w.double().cpu())
    out = torch.full((T, H, N + 8), 3.0, dtype=dtype, device=dev)
    ops.gemm_heads(x, w, out=out)
    _close(out[..., :N], want, dtype)
    assert (out[..., N:] == 3).all()
    _close(ops.gemm_heads(x, w, gate=gate), want * torch.sigmoid(gate.double().cpu()).view(T, H, N), dtype)


def _paged_case(dev, dtype, q_lens, ctx, H, L, R, bs, seed=0, stand_out=None):
    """Random latent rows in permuted pages; ``stand_out`` [request] = position whose key outshines all others for
    the request's last query.  Returns (q, cache, meta, [rows per request])."""
    Dc = (L + R + 15) // 16 * 16
    seqs = [a + b for a, b in zip(q_lens, ctx)]
    pages = [-(-s // bs) for s in seqs]
    g = torch.Generator().manual_seed(seed)
    perm = (torch.randperm(sum(pages), generator=g) + 1).to(torch.int32)
    cache = torch.randn(sum(pages) + 1, bs, Dc, generator=g) * 50         # rows of no request must not be read
    q = torch.randn(sum(q_lens), H, Dc, generator=g)
    q[..., L + R:] = 0
    bt = torch.zeros(len(seqs), max(pages) + 1, dtype=torch.int32)
    rows, off, tok = [], 0, 0
    for r, s in enumerate(seqs):
        bt[r, :pages[r]] = perm[off:off + pages[r]]
        off += pages[r]
        row = torch.randn(s, L + R, generator=g)
        last = tok + q_lens[r] - 1
        if stand_out is not None:
            row[stand_out[r]] = q[last, 0, :L + R] * 2.5
            q[last] = q[last, 0]
        row = row.to(dtype).float()
        for p in range(s):
            cache[bt[r, p // bs], p % bs] = 0
            cache[bt[r, p // bs], p % bs, :L + R] = row[p]
        rows.append(row)
        tok += q_lens[r]
    T = sum(q_lens)
    qsl = torch.tensor([0] + list(np.cumsum(q_lens)), dtype=torch.int32)
    meta = AttentionMetadata(None, None, bt.to(dev), torch.tensor(seqs, dtype=torch.int32, device=dev), qsl.to(dev),
                             len(seqs), T, max_query_len=max(q_lens), max_seq_len=max(seqs), padded_num_reqs=len(seqs),
                             padded_num_tokens=T, query_start_loc_cpu=qsl.long())
    return q.to(dtype).to(dev), cache.to(dtype).to(dev), meta, rows


def _plain_paged(q, rows, q_lens, L, width, scale):
    out, tok = [], 0
    for row, n in zip(rows, q_lens):
        row = row.double()
        for i in range(n):
            seen = row[:row.shape[0] - n + i + 1]
            s = q[tok, :, :width].double().cpu() @ seen.t() * scale
            e = torch.exp(s - s.max(-1, keepdim=True).values)
            out.append(e / e.sum(-1, keepdim=True) @ seen[:, :L])
            tok += 1
    return torch.stack(out)


@pytest.mark.parametrize("dev,dtype", DEV_DTYPE)
@pytest.mark.parametrize("H,L,R", [(1, 24, 8), (3, 56, 16), (5, 72, 10), (6, 112, 48), (16, 200, 24), (20, 320, 64),
                                   (33, 512, 64), (2, 640, 32), (4, 33, 4)])
def test_paged_latent_attention(dev, dtype, H, L, R):
    q_lens, ctx = [1, 17, 1, 2, 40], [0, 30, 95, 15, 0]
    q, cache, meta, rows = _paged_case(dev, dtype, q_lens, ctx, H, L, R, 16)
    scale = 0.5 * (L + R) ** -0.5
    got = ops.mla_paged_attention(q, cache, meta, scale, L)
    _close(got, _plain_paged(q, rows, q_lens, L, L + R, scale), dtype, 1.5)
    one = [1, 1, 1]                                          # a decode step: no row list over the requests
    q, cache, meta, rows = _paged_case(dev, dtype, one, [0, 47, 130], H, L, R, 32)
    got = ops.mla_paged_attention(q, cache, meta, scale, L)
    _close(got, _plain_paged(q, rows, one, L, L + R, scale), dtype, 1.5)


@pytest.mark.parametrize("dev,dtype", DEV_DTYPE)
@pytest.mark.parametrize("H,L,R", [(3, 48, 16), (16, 144, 32)])
def test_one_outstanding_key_anywhere_in_the_context(dev, dtype, H, L, R):
    """The last query of each request attends one key almost alone: the output is that key's latent, wherever the
    key lies (first tokens, page borders, portion starts, the query's own position)."""
    S = 150
    places = [0, 1, 15, 16, 17, 63, 64, 127, 128, S - 2, S - 1]
    for q_len in (1, 2, 37):
        lens, ctx = [q_len] * len(places), [S - q_len] * len(places)
        q, cache, meta, rows = _paged_case(dev, dtype, lens, ctx, H, L, R, 16, seed=q_len, stand_out=places)
        got = ops.mla_paged_attention(q, cache, meta, 1.0, L)
        _close(got, _plain_paged(q, rows, lens, L, L + R, 1.0), dtype, 1.5)
        for r, p in enumerate(places):
            _close(got[(r + 1) * q_len - 1, 0], rows[r][p, :L], dtype, 1.5)


@pytest.mark.gpu
def test_padded_rows_of_a_step_come_back_as_zeros():
    q, cache, meta, rows = _paged_case("cuda", BF16, [1, 1], [20, 3], 6, 64, 16, 16)
    pad = torch.full((3, *q.shape[1:]), float("nan"), dtype=BF16, device="cuda")
    q = torch.cat([q, pad])
    meta.query_start_loc = torch.tensor([0, 1, 2, 2, 2, 2], dtype=torch.int32, device="cuda")
    meta.seq_lens = torch.cat([meta.seq_lens, torch.zeros(3, dtype=torch.int32, device="cuda")])
    meta.block_tables = torch.cat([meta.block_tables, torch.zeros(3, meta.block_tables.shape[1], dtype=torch.int32,
                                                                  device="cuda")])
    meta.padded_num_reqs, meta.padded_num_tokens = 5, 5
    got = ops.mla_paged_attention(q, cache, meta, 0.1, 64)
    _close(got[:2], _plain_paged(q, rows, [1, 1], 64, 80, 0.1), BF16)
    assert (got[2:] == 0).all()


# ------------------------------------------------------------------------------------------------- the model
def replay_logits(rep, tokens, cuts, rid="a"):
    """Logits of every position of one request cut into portions."""
    out, at = [], 0
    for n in cuts:
        out.append(rep.step([(rid, tokens[at:at + n], list(range(n)))], [rid] if at + n == len(tokens) else []))
        at += n
    assert at == len(tokens)
    return torch.cat(out)


def portions(total, sizes):
    cuts, i = [], 0
    while sum(cuts) < total:
        cuts.append(min(sizes[i % len(sizes)], total - sum(cuts)))
        i += 1
    return cuts


MODELS = {
    "shared": shared_config(),
    "one_layer_all_sizes_odd": config([(mixer(heads=1, dim=7, rot_dim=6, vdim=5, q_rank=9, kv_rank=11), 13)], width=21,
                                      vocab=37, cap=None),
    "no_scaling_no_mlp": config([(mixer(scaling=None, heads=5, vdim=48, kv_rank=136), 0)] * 2, width=80, eps=1e-2),
    "wide": config([(mixer(heads=16, dim=64, rot_dim=32, vdim=64, q_rank=192, kv_rank=256), 320),
                    (mixer(heads=20, dim=32, rot_dim=32, vdim=40, q_rank=96, kv_rank=256, kv_from=0), 448)], width=256,
                   vocab=1000),
}


@pytest.mark.parametrize("dev", DEVS)
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(MODELS))
def test_prompt_portions_and_single_tokens_match_the_plain_model(tmp_path, dev, dtype, name):
    cfg = MODELS[name]
    w = write_model(str(tmp_path), cfg, seed=3)
    toks = tokens_of(83, cfg["vocab"], 1)
    want = plain.forward(cfg, w, toks)
    rep = make_replay(str(tmp_path), dtype, 128, dev)
    for cuts in ([83], [50] + [1] * 33, portions(83, [2, 3]), portions(83, [15, 2, 16, 1, 17, 31])):
        got = replay_logits(rep, toks, cuts)
        assert logit_error(got, want) < LIMIT[dtype], cuts
    if name == "shared":
        assert logit_error(replay_logits(rep, toks, [1] * 83), want) < LIMIT[dtype]


@pytest.mark.parametrize("dev", DEVS)
def test_residual_stream_after_every_layer(tmp_path, dev):
    """32-bit layer by layer, so that two mistakes cannot make up for each other."""
    cfg = MODELS["shared"]
    w = write_model(str(tmp_path), cfg, seed=9)
    toks = tokens_of(21, cfg["vocab"], 4)
    want: list = []
    plain.forward(cfg, w, toks, layers_out=want)
    rep = make_replay(str(tmp_path), "float32", 64, dev)
    model, got = rep.engine.runner.model, []
    for layer in model.layers:
        fwd = layer.forward

        def spy(*a, fwd=fwd):
            h, r = fwd(*a)
            got.append(r.double().cpu().clone())
            return h, r
        layer.forward = spy
    replay_logits(rep, toks, [21])
    assert len(got) == len(want)
    for g, e in zip(got, want):
        assert (g - e).abs().max() < 3e-5 * e.abs().max()


@pytest.mark.parametrize("dev", DEVS)
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_mixed_batches_and_reused_pages_match_each_request_alone(tmp_path, dev, dtype):
    cfg = MODELS["shared"]
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
        assert logit_error(torch.cat(got[k]), want[k]) < LIMIT[dtype], k
    assert pool.num_free_blocks == free0


def _pointed_model(path, cfg, seed=2):
    """Scores are sharpened (large query norm weights), so that single keys decide the output."""
    def edit(w):
        for k in w:
            if k.endswith("dq.norm"):
                w[k] = (w[k].float() * 9).bfloat16()
    return write_model(path, cfg, seed=seed, edit=edit)


@pytest.mark.parametrize("dev", DEVS)
def test_far_and_border_keys_decide_logits(tmp_path, dev):
    """With pointed attention a key that goes missing shows in the logits: the plain model with the key left out is
    far from the plain model, the engine is not, neither in a prompt nor in decoding."""
    cfg = config([(mixer(), 64), (mixer(kv_from=0), 64)])
    w = _pointed_model(str(tmp_path), cfg)
    toks = tokens_of(130, cfg["vocab"], 3)
    want = plain.forward(cfg, w, toks)
    rep = make_replay(str(tmp_path), "float32", 192, dev)
    got = replay_logits(rep, toks, [97, 2] + [1] * 31)
    assert logit_error(got, want) < LIMIT["float32"] * 5
    for key in (0, 1, 15, 16, 31, 32, 63, 64, 96, 97):
        wrong = plain.forward(cfg, w, toks, hidden_keys=(key,))
        shift = [logit_error(wrong[p:p + 1], want[p:p + 1]) for p in range(key + 1, 130)]
        assert max(shift) > 100 * LIMIT["float32"], key
    assert logit_error(replay_logits(rep, toks, portions(130, [2, 5])), want) < LIMIT["float32"] * 5


@pytest.mark.parametrize("dev", DEVS)
def test_first_tokens_of_a_sequence(tmp_path, dev):
    cfg = MODELS["shared"]
    w = write_model(str(tmp_path), cfg, seed=1)
    rep = make_replay(str(tmp_path), "float32", 64, dev)
    for n in (1, 2, 3):
        toks = tokens_of(n, cfg["vocab"], n)
        assert logit_error(replay_logits(rep, toks, [n]), plain.forward(cfg, w, toks)) < LIMIT["float32"]


@pytest.mark.parametrize("dev", DEVS)
@pytest.mark.parametrize("kw", [{}, {"async_scheduling": True}, {"enforce_eager": True},
                                {"enable_prefix_caching": True}, {"num_gpu_blocks_override": 12},
                                {"speculative_config": {"method": "ngram", "num_speculative_tokens": 3}}],
                         ids=lambda k: next(iter(k), "default"))
def test_greedy_generation_through_the_engine(tmp_path, dev, kw):
    """``LLM.generate`` in 32-bit: chunked prompts (40-token steps), batches of unequal requests, long decoding, and
    a pool small enough to preempt, against greedy decoding with the plain model."""
    from vllm_torchtpu_b200.engine.llm import LLM
    cfg = config([(mixer(), 64), (mixer(kv_from=0, heads=2), 0)], cap=9.0)
    w = write_model(str(tmp_path), cfg, seed=6)
    prompts = [tokens_of(n, cfg["vocab"], n) for n in (3, 52, 17, 41)]
    if "enable_prefix_caching" in kw:
        prompts[3] = prompts[1][:32] + prompts[3][:9]
    llm = LLM(str(tmp_path), device=dev, dtype="float32", max_num_seqs=4, max_num_batched_tokens=40, max_model_len=128,
              init_dist=False, **{"num_gpu_blocks_override": 64, **kw})
    n_out = 48 if not kw else 24
    outs = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=n_out, ignore_eos=True))
    for p, o in zip(prompts, outs):
        ids = o.outputs[0].token_ids
        assert len(ids) == n_out
        z = plain.forward(cfg, w, list(p) + list(ids[:-1]))[len(p) - 1:]
        top = z.max(-1).values
        assert (top - z[torch.arange(n_out), torch.tensor(ids)] <= 1e-4).all()      # ties aside, the greedy path
    if kw.get("num_gpu_blocks_override") == 12:
        assert llm.engine.scheduler.stats["preemptions"] > 0
    if "enable_prefix_caching" in kw:
        again = llm.generate([prompts[3]], SamplingParams(temperature=0.0, max_tokens=n_out, ignore_eos=True))
        assert llm.engine.scheduler.stats["prefix_hit_tokens"] > 0
        assert again[0].outputs[0].token_ids == outs[3].outputs[0].token_ids


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
def test_sampled_decode_graph_captured_with_few_requests_serves_more(tmp_path):
    """A graph captured on first use with two live requests is replayed with four: its kernels must not keep the
    first batch's request count."""
    from vllm_torchtpu_b200.engine.llm import LLM
    cfg = MODELS["wide"]
    w = write_model(str(tmp_path), cfg, seed=8)
    llm = LLM(str(tmp_path), device="cuda", max_num_seqs=4, max_num_batched_tokens=64, num_gpu_blocks_override=64,
              init_dist=False)
    sp = SamplingParams(temperature=1.0, top_k=1, max_tokens=6, ignore_eos=True)       # samples the arg-max
    prompts = [tokens_of(n, cfg["vocab"], n) for n in (5, 33, 40, 18)]
    for n in (2, 4):
        for p, o in zip(prompts, llm.generate(prompts[:n], sp)):
            ids = o.outputs[0].token_ids
            z = plain.forward(cfg, w, p + list(ids[:-1]))[len(p) - 1:]
            short = z.max(-1).values - z[torch.arange(6), torch.tensor(ids)]
            assert (short < 0.1 * z.std()).all(), short          # the arg-max up to bf16 rounding
    assert llm.engine.runner.stats["graph_steps"] >= 10


# ------------------------------------------------------------------------------------------------- surroundings
def test_configuration_reads_every_size_and_refuses_what_is_not_built():
    cfg = shared_config()
    mc = ModelConfig.from_hf_dict(cfg, "m")
    assert mc.architecture == "mazivik" and mc.num_layers == 4 and mc.vocab_size == 211 and mc.final_logit_softcap == 17.0
    assert [s.mixer.kv_from for s in mc.layer_specs] == [None, None, 0, 1]
    assert [s.ff for s in mc.layer_specs] == [88, 56, 0, 104] and mc.is_mla
    w = plain.random_model(cfg)
    assert mc.num_params() == sum(v.numel() for k, v in w.items() if v.dim() == 2)
    bad = [("type", lambda c: c["layers"][0].update(type="other")),
           ("feed-forward", lambda c: c["layers"][0]["mlp"].update(kind="experts")),
           ("kv_from", lambda c: c["layers"][2]["mixer"].update(kv_from=3)),
           ("kv_from", lambda c: c["layers"][3]["mixer"].update(kv_from=2)),
           ("rotation", lambda c: c["layers"][2]["mixer"]["rot"].update(base=1.0))]
    for what, change in bad:
        c = json.loads(json.dumps(cfg))
        change(c)
        with pytest.raises(ValueError, match=what):
            ModelConfig.from_hf_dict(c)
    for kw in (dict(parallel=ParallelConfig(tensor_parallel_size=4)), dict(parallel=ParallelConfig(pipeline_parallel_size=2)),
               dict(speculative={"method": "mtp"})):
        with pytest.raises(ValueError):
            EngineConfig(model=ModelConfig.from_hf_dict(cfg), device="cpu", **kw).finalize()
    mc.quantization = "int8"
    with pytest.raises(ValueError, match="quantised"):
        EngineConfig(model=mc, device="cpu").finalize()


def test_caches_are_allocated_once_per_owner(tmp_path):
    cfg = shared_config()
    write_model(str(tmp_path), cfg)
    r = make_replay(str(tmp_path), "float32", 64, "cpu").engine.runner
    assert r.kv_caches[2] is r.kv_caches[0] and r.kv_caches[3] is r.kv_caches[1] and len(r.distinct_kv_caches) == 2
    assert r.kv_caches[0].shape == (5, 16, 64) and r.kv_caches[1].shape == (5, 16, 80)       # 48 + 16, 64 + 8 padded
    assert r.model.kv_bytes_per_block(16, torch.float32) == 16 * (64 + 80) * 4


def test_incomplete_checkpoints_are_refused_and_weights_can_be_replaced(tmp_path):
    from safetensors.torch import save_file
    cfg = config([(mixer(), 40)])
    w = write_model(str(tmp_path / "a"), cfg, seed=0)
    w2 = plain.random_model(cfg, seed=1)
    write_model(str(tmp_path / "b"), cfg)
    save_file({k: v for k, v in w.items() if k != "l0.mix.uv"}, str(tmp_path / "b" / "model.safetensors"))
    with pytest.raises(ValueError, match="l0.mix.uv"):
        make_replay(str(tmp_path / "b"), "float32", 64, "cpu")
    rep = make_replay(str(tmp_path / "a"), "float32", 64, "cpu")
    toks = tokens_of(9, cfg["vocab"])
    part = {k: w2[k] for k in ("l0.mix.dq", "l0.mix.dkv", "l0.mix.g", "l0.mix.uk", "final.norm")}
    with pytest.raises(ValueError, match="l0.mix.g"):
        rep.engine.update_weights({k: v for k, v in part.items() if k != "l0.mix.g"})
    rep.engine.update_weights(part)
    assert logit_error(replay_logits(rep, toks, [9]), plain.forward(cfg, w | part, toks)) < LIMIT["float32"]


def test_replay_refuses_steps_that_do_not_fit(tmp_path):
    cfg = config([(mixer(), 40)])
    write_model(str(tmp_path), cfg)
    rep = make_replay(str(tmp_path), "float32", 32, "cpu")
    rep.step([("a", [1, 2, 3], [])])
    with pytest.raises(ValueError, match="place"):
        rep.step([("a", [4], [1])])
    rep = make_replay(str(tmp_path), "float32", 32, "cpu")
    rep.step([("a", list(range(17)), [])])
    with pytest.raises(RuntimeError, match="full"):
        rep.step([("b", [1], [0])])
    rep = make_replay(str(tmp_path), "float32", 128, "cpu")
    with pytest.raises(RuntimeError, match="live"):
        rep.step([(f"r{i}", [1], []) for i in range(5)])


def test_trace_run_command(tmp_path):
    cfg = config([(mixer(), 40)])
    w = write_model(str(tmp_path / "m"), cfg)
    toks = tokens_of(12, cfg["vocab"])
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:7], "want": [0, 6]}, {"id": "b", "tokens": toks[:2], "want": []}],
              "end": ["b"]},
             {"step": 1, "entries": [{"id": "a", "tokens": toks[7:9], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": toks[:1], "want": [0]}, {"id": "a", "tokens": toks[9:], "want": [2]}],
              "end": ["a", "b"]}]
    os.mkdir(tmp_path / "out")
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", "float32",
                        "--out", str(tmp_path / "out"), "--max-tokens", "64", "--device", "cpu"],
                       input="\n".join(map(json.dumps, steps)), capture_output=True, text=True, timeout=120)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.split("\n") if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    z = plain.forward(cfg, w, toks)

    def read(n):
        return torch.from_numpy(np.fromfile(tmp_path / "out" / f"{n}.f32", "<f4").reshape(-1, cfg["vocab"]))
    assert sorted(os.listdir(tmp_path / "out")) == ["0.f32", "2.f32"]
    assert logit_error(read(0), z[[0, 6]]) < LIMIT["float32"]
    assert logit_error(read(2), z[[0, 11]]) < LIMIT["float32"]


def test_two_tensor_parallel_ranks_match_one():
    from test_parallel_cpu import _run
    assert _run(2, "tp", "tiny-mazivik") == _run(1, "tp", "tiny-mazivik")


def test_server_command_line_builds_the_engine(tmp_path):
    import argparse

    from vllm_torchtpu_b200.entrypoints import cli
    cfg = config([(mixer(), 40)])
    write_model(str(tmp_path), cfg)
    ap = argparse.ArgumentParser()
    cli.add_engine_args(ap)
    llm = cli.make_llm(ap.parse_args([str(tmp_path), "--device", "cpu", "--max-num-seqs", "2", "--max-model-len", "64"]))
    assert type(llm.engine.runner.model).__name__ == "MazivikForCausalLM"
    out = llm.generate([[1, 2, 3]], SamplingParams(max_tokens=4, temperature=0.7, top_p=0.9, logprobs=2))
    assert len(out[0].outputs[0].token_ids) == 4
    assert model_preset("tiny-mazivik").architecture == "mazivik"


def test_family_library_lists_existing_sources():
    from vllm_torchtpu_b200.csrc import build
    for fam, sources in build.FAMILY_SOURCES.items():
        assert set(sources) <= set(build._sources()), fam
