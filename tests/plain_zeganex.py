"""Plain, slow statement of the Zeganex decoder, one function per mechanism.

Whole sequences, no cache, no state, in the dtype of the tensors it is given (float64 in the tests); shares no code with
the package.  ``cfg`` is the dictionary of a Zeganex ``config.json``; ``w`` maps checkpoint tensor names to tensors.
The keyword arguments beside the model's own are mistakes that a test plants to see whether it would notice them.
"""
import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def relu_squared(z):
    return torch.where(z > 0, z * z, torch.zeros_like(z))


# --------------------------------------------------------------------------------------------- embedding
def bigram_row(prev, cur, b):
    """Row of the pair table; ``prev`` None in front of a sequence's first token."""
    return b["buckets"] if prev is None else (prev * b["mul_prev"] + cur * b["mul_cur"]) % b["buckets"]


def embed(tokens, w, b, forget_at=()):
    """``forget_at``: positions whose previous token is taken for absent."""
    rows = [bigram_row(None if i == 0 or i in forget_at else int(tokens[i - 1]), int(t), b) for i, t in enumerate(tokens)]
    return torch.stack([w["embed"][int(t)] + w["bigram"][r] for t, r in zip(tokens, rows)])


# --------------------------------------------------------------------------------------------- projections
def short_conv(u, taps, before=None):
    """u [S, C], taps [C, K], the last column weighs the current token; zeros (or ``before`` [K - 1, C]) ahead."""
    K, S = taps.shape[1], u.shape[0]
    full = torch.cat([u.new_zeros(K - 1, u.shape[1]) if before is None else before, u])
    y = torch.zeros_like(u)
    for j in range(K):
        y = y + full[j:j + S] * taps[:, j]
    return y


def project(h, w, p, name, cut=None):
    """Projection with bias, then the convolution.  ``cut``: positions in front of which the convolution sees zeros."""
    u = h @ w[p + name].t() + w[p + name + ".b"]
    if not cut:
        return short_conv(u, w[p + name + ".conv"])
    return torch.cat([short_conv(u[:cut], w[p + name + ".conv"]), short_conv(u[cut:], w[p + name + ".conv"])])


def frequencies(rot):
    """Angle per position of every pair, and the factor on cos and sin."""
    dims, base, s = rot["dims"], rot["base"], rot.get("scaling")
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not s:
        return f, 1.0
    at = lambda turns: dims * math.log(s["original"] / (2 * math.pi * turns)) / (2 * math.log(base))    # noqa: E731
    lo, hi = max(math.floor(at(s["fast"])), 0), min(math.ceil(at(s["slow"])), dims - 1)
    out = []
    for i, v in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(v / s["factor"] * r + v * (1 - r))
    return out, 0.1 * math.log(s["factor"]) + 1.0


def rotate_pairs(x, rot, first=0):
    """x [S, heads, d], row t at position first + t: dimension 2i turns with dimension 2i + 1."""
    f, mult = frequencies(rot)
    out = x.clone()
    for i, fi in enumerate(f):
        a = [(first + t) * fi for t in range(x.shape[0])]
        c = torch.tensor([math.cos(v) * mult for v in a], dtype=x.dtype)[:, None]
        s = torch.tensor([math.sin(v) * mult for v in a], dtype=x.dtype)[:, None]
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        out[:, :, 2 * i] = u * c - v * s
        out[:, :, 2 * i + 1] = v * c + u * s
    return out


# --------------------------------------------------------------------------------------------- attention
def visible(S, window, lost_key=None):
    """[query, key] mask: the key itself and the window - 1 tokens before it."""
    i, j = torch.arange(S)[:, None], torch.arange(S)[None, :]
    m = (j <= i) & (i - j < window)
    if lost_key is not None:
        m = m & ~((j == lost_key) & (i > lost_key))
    return m


def softmax_rows(s, mask):
    s = s.masked_fill(~mask, float("-inf"))
    e = torch.exp(s - s.max(-1, keepdim=True).values)
    return e / e.sum(-1, keepdim=True)


def heads_attention(q, k, v, scale, mask):
    """q [S, H, d], k [S, G, d], v [S, G, dv]: query head h uses key and value head h // (H / G)."""
    H, G = q.shape[1], k.shape[1]
    out = []
    for h in range(H):
        g = h // (H // G)
        out.append(softmax_rows((q[:, h] @ k[:, g].t()) * scale, mask) @ v[:, g])
    return torch.stack(out, 1)


def mixing_factor(w, p, diff):
    return torch.exp((w[p + "lq1"] * w[p + "lk1"]).sum()) - torch.exp((w[p + "lq2"] * w[p + "lk2"]).sum()) + diff


def combine_maps(a1, a2, lam, diff, eps):
    return rms(a1 - lam * a2, eps) * (1 - diff)


def differential_attention(h, w, p, m, eps, kv=None, conv_cut=None, window=None, lost_key=None, one_map=False):
    """(output, (keys, values)); ``kv``: those of the layer this one reads."""
    S, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = project(h, w, p, "q", conv_cut).reshape(S, H, 2, d)
    if kv is None:
        kv = (project(h, w, p, "k", conv_cut).reshape(S, G, 2, d), project(h, w, p, "v", conv_cut).reshape(S, G, dv))
    k, v = kv
    mask = visible(S, window or m["mask"]["size"], lost_key)
    a1 = heads_attention(q[:, :, 0], k[:, :, 0], v, m["scale"], mask)
    a2 = heads_attention(q[:, :, 1], k[:, :, 1], v, m["scale"], mask)
    lam = 0.0 if one_map else mixing_factor(w, p, m["diff"])
    return combine_maps(a1, a2, lam, m["diff"], eps).reshape(S, H * dv) @ w[p + "o"].t(), kv


def gated_rotary_attention(h, w, p, m, eps, kv=None, conv_cut=None, window=None, lost_key=None, no_gate=False):
    S, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rotate_pairs(project(h, w, p, "q", conv_cut).reshape(S, H, d), m["rot"])
    k = rotate_pairs(project(h, w, p, "k", conv_cut).reshape(S, G, d), m["rot"])
    v = project(h, w, p, "v", conv_cut).reshape(S, G, dv)
    o = heads_attention(q, k, v, m["scale"], visible(S, window or m["mask"]["size"], lost_key)).reshape(S, H * dv)
    if not no_gate:
        o = o * sigmoid(h @ w[p + "g"].t())
    return o @ w[p + "o"].t() + w[p + "o.b"], (k, v)


MIXERS = {"attention": differential_attention, "attention_2": gated_rotary_attention}


# --------------------------------------------------------------------------------------------- feed-forward
def dense(x, w, p):
    return (silu(x @ w[p + "gate"].t()) * (x @ w[p + "up"].t())) @ w[p + "down"].t()


def router(x, w_router, top):
    """[(expert, weight)] per token: softmax over all experts, the largest ``top``, not renormalised."""
    z = x @ w_router.t()
    e = torch.exp(z - z.max(-1, keepdim=True).values)
    s = e / e.sum(-1, keepdim=True)
    return [[(int(i), row[i]) for i in torch.argsort(row, descending=True)[:top]] for row in s]


def experts(x, w, p, m):
    out = torch.zeros_like(x)
    for t, chosen in enumerate(router(x, w[p + "router"], m["router"]["top"])):
        for e, s in chosen:
            out[t] = out[t] + s * (relu_squared(x[t] @ w[p + f"e{e}.up"].t()) @ w[p + f"e{e}.down"].t())
    return out


def feed_forward(x, w, p, m):
    return dense(x, w, p) if m["kind"] == "dense" else experts(x, w, p, m)


# --------------------------------------------------------------------------------------------- the model
def forward(cfg, w, tokens, *, layers_out=None, dtype=torch.float64, plant=None, forget_at=()):
    """Logits [S, vocab] of one sequence; appends the stream after every layer to ``layers_out``.  ``plant``:
    {layer: keyword arguments of its mixer}."""
    w = {k: v.to(dtype) for k, v in w.items()}
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    x = embed(tokens, w, cfg["embedding"]["bigram"], forget_at)
    kvs = []
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        kv = kvs[m["kv_from"]] if m.get("kv_from") is not None else None
        y, kv = MIXERS[layer["type"]](rms(x, eps) * w[p + "norm1"], w, p + "mix.", m, eps, kv, **(plant or {}).get(i, {}))
        kvs.append(kv)
        x = x + mult * (rms(y, eps) * w[p + "norm1b"])
        if layer.get("mlp"):
            y = feed_forward(rms(x, eps) * w[p + "norm2"], w, p + "mlp.", layer["mlp"])
            x = x + mult * (rms(y, eps) * w[p + "norm2b"])
        if layers_out is not None:
            layers_out.append(x)
    return (rms(x, eps) * w["final.norm"]) @ w["embed"].t()
