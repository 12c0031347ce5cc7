"""Plain, slow statement of the Vipolix decoder, one function per mechanism.

Whole sequences, token by token where a state is carried, no cache, in the dtype of the tensors it is given (float64
in the tests); shares no code with the package.  ``cfg`` is the dictionary of a Vipolix ``config.json``; ``w`` maps
checkpoint tensor names to tensors.  Keyword arguments that are absent from a configuration plant mistakes.
"""
import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def model_norm(x, w, eps):
    return rms(x, eps) * (1.0 + w)


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def token_shift(h, mix, forget_at=None):
    """h [S, width]: every row moves towards the row before it (zeros ahead of the first)."""
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    if forget_at is not None:
        before[forget_at] = 0
    return h + (before - h) * mix


# --------------------------------------------------------------------------------------------- carried states
def outer(k, v):
    """Per head: [H, d], [H, dv] -> [H, d, dv]."""
    return k[:, :, None] * v[:, None, :]


def read(st, q):
    """Per head: st^T q."""
    return (st * q[:, :, None]).sum(1)


def gla_decay(z, tau):
    """Factors sigmoid(z)^(1 / tau)."""
    return sigmoid(z) ** (1.0 / tau)


def gla_states(q, k, v, alpha, state=None):
    """q, k, alpha [S, H, d], v [S, H, dv] -> o [S, H, dv] and the state after the last token."""
    st = torch.zeros(q.shape[1], q.shape[2], v.shape[2], dtype=q.dtype) if state is None else state
    o = []
    for t in range(q.shape[0]):
        st = alpha[t][:, :, None] * st + outer(k[t], v[t])
        o.append(read(st, q[t]))
    return torch.stack(o), st


def gla(h, w, p, m, eps, forget_at=None, no_decay=False):
    S, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].t()).reshape(S, H, d) * d ** -0.5
    k = (h @ w[p + "k"].t()).reshape(S, H, d)
    v = (h @ w[p + "v"].t()).reshape(S, H, dv)
    z = (h @ w[p + "a1"].t()) @ w[p + "a2"].t() + w[p + "a2.b"]
    alpha = gla_decay(z, m["tau"]).reshape(S, H, d)
    if no_decay:
        alpha = torch.ones_like(alpha)
    if forget_at is not None:
        alpha = alpha.clone()
        alpha[forget_at] = 0
    o, _ = gla_states(q, k, v, alpha)
    o = (rms(o, eps) * w[p + "norm"]).reshape(S, H * dv)
    return (o * silu(h @ w[p + "g"].t())) @ w[p + "o"].t()


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def removal_decay(z):
    """Factors exp(-exp(-1/2) sigmoid(z))."""
    return torch.exp(-math.exp(-0.5) * sigmoid(z))


def removal_states(r, k, v, wd, a, state=None, no_removal=False):
    """Decay and removal both read the state of the token before.  All [S, H, d]."""
    S, H, d = r.shape
    st = torch.zeros(H, d, v.shape[2], dtype=r.dtype) if state is None else state
    u = unit(k)
    o = []
    for t in range(S):
        taken = outer(a[t] * u[t], read(st, u[t]))
        st = wd[t][:, :, None] * st + outer(k[t], v[t]) - (0 if no_removal else taken)
        o.append(read(st, r[t]))
    return torch.stack(o), st


def removal(h, w, p, m, eps, forget_at=None, no_removal=False):
    S, H, d = h.shape[0], m["heads"], m["dim"]
    r, k, v = ((h @ w[p + n].t()).reshape(S, H, d) for n in "rkv")
    wd = removal_decay(torch.tanh(h @ w[p + "w1"].t()) @ w[p + "w2"].t() + w[p + "w0"]).reshape(S, H, d)
    a = sigmoid(h @ w[p + "a"].t() + w[p + "a.b"]).reshape(S, H, d)
    if forget_at is not None:
        o = torch.cat([removal_states(*(t[s] for t in (r, k, v, wd, a)), no_removal=no_removal)[0]
                       for s in (slice(0, forget_at), slice(forget_at, S))])
    else:
        o, _ = removal_states(r, k, v, wd, a, no_removal=no_removal)
    return (rms(o, eps).reshape(S, H * d) * w[p + "norm"] * sigmoid(h @ w[p + "g"].t())) @ w[p + "o"].t()


# --------------------------------------------------------------------------------------------- attention
def short_conv(x, taps, cut=None):
    """x [S, C], taps [C, K] (last column: the current token), zeros ahead.  ``cut``: zeros before it once more."""
    if cut is not None:
        return torch.cat([short_conv(x[:cut], taps), short_conv(x[cut:], taps)])
    K = taps.shape[1]
    full = torch.cat([torch.zeros(K - 1, x.shape[1], dtype=x.dtype), x])
    return sum(full[j:j + x.shape[0]] * taps[:, j] for j in range(K))


def rotate_pairs(x, rot):
    """x [S, heads, d], row t at position t: dimensions 2i and 2i + 1 turn together."""
    out = x.clone()
    for i in range(rot["dims"] // 2):
        a = [t * rot["base"] ** (-2.0 * i / rot["dims"]) for t in range(x.shape[0])]
        c = torch.tensor([math.cos(v) for v in a], dtype=x.dtype)[:, None]
        s = torch.tensor([math.sin(v) for v in a], dtype=x.dtype)[:, None]
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        out[:, :, 2 * i] = u * c - v * s
        out[:, :, 2 * i + 1] = v * c + u * s
    return out


def chunk_mask(S, size, off=0):
    """True where query i (row) sees key j: not later and in the same chunk."""
    i = torch.arange(S)
    return (i[:, None] >= i[None]) & ((i[:, None] + off) // size == (i[None] + off) // size)


def sink_softmax(s):
    """One is added to the denominator."""
    top = torch.clamp(s.max(-1, keepdim=True).values, min=0)
    e = torch.exp(s - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(-top))


def attention(h, w, p, m, lost_key=None, edge=0, no_sink=False, no_temp=False, conv_cut=None):
    """``edge``: the chunks begin that many tokens earlier; ``lost_key``: a key that no later query sees."""
    S, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (short_conv(h @ w[p + n].t() + w[p + n + ".b"], w[p + n + ".conv"], conv_cut) for n in "qkv")
    q, k = rotate_pairs(q.reshape(S, H, d), m["rot"]), rotate_pairs(k.reshape(S, G, d), m["rot"])
    v = v.reshape(S, G, dv)
    seen = chunk_mask(S, m["mask"]["size"], edge)
    if lost_key is not None:
        seen[lost_key + 1:, lost_key] = False
    out = torch.zeros(S, H, dv, dtype=h.dtype)
    for hh in range(H):
        g = hh // (H // G)
        s = (q[:, hh] @ k[:, g].t()) * m["scale"]
        s = s if no_temp else s * w[p + "temp"][hh]
        s = s.masked_fill(~seen, float("-inf"))
        out[:, hh] = (torch.softmax(s, -1) if no_sink else sink_softmax(s)) @ v[:, g]
    return out.reshape(S, H * dv) @ w[p + "o"].t()


def parallel(h, w, p, m, eps, left=None, right=None):
    a = attention(h, w, p + "left.", m["left"], **(left or {}))
    b = removal(h, w, p + "right.", m["right"], eps, **(right or {}))
    return m["left_scale"] * a + m["right_scale"] * b


MIXERS = {"gla": gla, "parallel": parallel}


# --------------------------------------------------------------------------------------------- feed-forward
def expert(x, w, p, limit):
    g = torch.clamp(x @ w[p + "gate"].t(), max=limit)
    u = torch.clamp(x @ w[p + "up"].t(), -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].t()


def route(x, w, p, r):
    """Chosen experts [S, top] and their weights."""
    s = sigmoid(x @ w[p + "router"].t())
    choice = s + w[p + "correction"]
    n = r["groups"]["count"]
    per = choice.reshape(len(x), n, -1)
    score = per.sort(-1, descending=True).values[..., :2].sum(-1)
    best = score.argsort(-1, descending=True)[:, :r["groups"]["keep"]]
    kept = torch.zeros(len(x), n, dtype=torch.bool)
    kept[torch.arange(len(x))[:, None], best] = True
    choice = per.masked_fill(~kept[..., None], float("-inf")).reshape(len(x), -1)
    ids = choice.argsort(-1, descending=True)[:, :r["top"]]
    ws = s.gather(-1, ids)
    return ids, ws / (ws.sum(-1, keepdim=True) + 1e-20) * r["scale"]


def feed_forward(x, w, p, mlp, no_shared=False):
    ids, ws = route(x, w, p, mlp["router"])
    out = torch.zeros_like(x)
    for e in range(mlp["router"]["experts"]):
        we = (ws * (ids == e)).sum(-1, keepdim=True)
        out = out + we * expert(x, w, f"{p}e{e}.", mlp["expert"]["limit"])
    if no_shared:
        return out
    return out + expert(x, w, p + "shared.", mlp["shared"]["limit"]) * sigmoid(x @ w[p + "shared.sg"].t())


def token_input(x, w, p, tokens, layer, dim, eps):
    e = w["side.embed"][tokens][:, layer * dim:(layer + 1) * dim]
    y = (gelu_tanh(x @ w[p + "side.gate"].t()) * e) @ w[p + "side.proj"].t()
    return rms(y, eps) * w[p + "side.norm"]


def forward(cfg, w, tokens, *, layers_out=None, dtype=torch.float64, plant=None):
    """Logits [S, vocab] of one sequence; appends the stream after every layer to ``layers_out``.  ``plant``:
    {layer: keyword arguments of its mixer, or shift=... / side=False / ff={...}} (mistakes that must show)."""
    w = {k: v.to(dtype) for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    x = w["embed"][tokens]
    for i, layer in enumerate(cfg["layers"]):
        p, wrong = f"l{i}.", dict((plant or {}).get(i, {}))
        shift, side, ff = wrong.pop("shift", {}), wrong.pop("side", True), wrong.pop("ff", {})
        h = token_shift(model_norm(x, w[p + "norm1"], eps), w[p + "shift"], **shift)
        x = x + MIXERS[layer["type"]](h, w, p + "mix.", layer["mixer"], eps, **wrong)
        if layer.get("mlp"):
            x = x + feed_forward(model_norm(x, w[p + "norm2"], eps), w, p + "mlp.", layer["mlp"], **ff)
        if side:
            x = x + token_input(x, w, p, tokens, i, cfg["token_side"]["dim"], eps)
        if layers_out is not None:
            layers_out.append(x)
    return model_norm(x, w["final.norm"], eps) @ w["head"].t()
