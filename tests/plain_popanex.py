"""Plain, slow statement of the Popanex decoder, one function per mechanism.

Whole sequences, token by token where a state is carried, no cache, in the dtype of the tensors it is given (float64
in the tests); shares no code with the package.  ``cfg`` is the dictionary of a Popanex ``config.json``; ``w`` maps
checkpoint tensor names to tensors.
"""
import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def model_norm(x, w, eps):
    return rms(x, eps) * (1.0 + w)


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def silu(z):
    return z / (1.0 + torch.exp(-z))


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def softplus(z):
    return torch.clamp(z, min=0) + torch.log(1.0 + torch.exp(-z.abs()))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


# --------------------------------------------------------------------------------------------- retention
def rotate_halves(x, rot, first=0):
    """x [S, heads, d], row t at position first + t: dimension i turns with dimension i + dims/2 (i < dims/2)."""
    half = rot["dims"] // 2
    out = x.clone()
    for i in range(half):
        a = [(first + t) * rot["base"] ** (-2.0 * i / rot["dims"]) for t in range(x.shape[0])]
        c = torch.tensor([math.cos(v) for v in a], dtype=x.dtype)[:, None]
        s = torch.tensor([math.sin(v) for v in a], dtype=x.dtype)[:, None]
        u, v = x[:, :, i], x[:, :, i + half]
        out[:, :, i] = u * c - v * s
        out[:, :, i + half] = v * c + u * s
    return out


def outer(k, v):
    """Per head: [H, d], [H, dv] -> [H, d, dv]."""
    return k[:, :, None] * v[:, None, :]


def read(st, q):
    """Per head: st^T q."""
    return (st * q[:, :, None]).sum(1)


def retention_states(q, k, v, decay, state=None):
    """q, k [S, H, d], v [S, H, dv], decay [H] -> o [S, H, dv] and the state after the last token."""
    S, H, d = q.shape
    st = torch.zeros(H, d, v.shape[2], dtype=q.dtype) if state is None else state
    gamma = torch.as_tensor(decay, dtype=q.dtype)[:, None, None]
    o = []
    for t in range(S):
        st = gamma * st + outer(k[t], v[t])
        o.append(read(st, q[t]))
    return torch.stack(o), st


def retention(h, w, p, m, eps, forget_at=None):
    """``forget_at``: a position before which the state is dropped (a planted mistake)."""
    S, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = rotate_halves((h @ w[p + "q"].t()).reshape(S, H, d), m["rot"])
    k = rotate_halves((h @ w[p + "k"].t()).reshape(S, H, d), m["rot"]) * d ** -0.5
    v = (h @ w[p + "v"].t()).reshape(S, H, dv)
    if forget_at:
        o = torch.cat([retention_states(a[0], a[1], a[2], m["decay"])[0] for a in
                       ((q[:forget_at], k[:forget_at], v[:forget_at]), (q[forget_at:], k[forget_at:], v[forget_at:]))])
    else:
        o, _ = retention_states(q, k, v, m["decay"])
    return (rms(o, eps).reshape(S, H * dv) * silu(h @ w[p + "g"].t())) @ w[p + "o"].t()


# --------------------------------------------------------------------------------------------- attention
def query_temperature(p, qt):
    return 1.0 + qt["coef"] * math.log(math.floor((p + 1) / qt["every"]) + 1)


def sink_softmax(scores, sink):
    """scores [..., keys], sink [...]: one more term exp(sink) in the denominator."""
    sink = sink[..., None]
    top = torch.maximum(scores.max(-1, keepdim=True).values, sink)
    e = torch.exp(scores - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - top))


def attention(h, w, p, m, eps, lost_key=None, no_sink=False, no_temp=False):
    """``lost_key``: a key that later queries do not see; ``no_sink``, ``no_temp``: left out (planted mistakes)."""
    S, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (rms(h @ w[p + "q"].t(), eps) * w[p + "q.norm"]).reshape(S, H, d)
    k = (rms(h @ w[p + "k"].t(), eps) * w[p + "k.norm"]).reshape(S, G, d)
    v = (h @ w[p + "v"].t()).reshape(S, G, dv)
    t = [1.0 if no_temp else query_temperature(i, m["q_temp"]) for i in range(S)]
    q = q * torch.tensor(t, dtype=h.dtype)[:, None, None]
    hidden = torch.ones(S, S, dtype=torch.bool).triu(1)
    if lost_key is not None:
        hidden[lost_key + 1:, lost_key] = True
    out = torch.zeros(S, H, dv, dtype=h.dtype)
    for hh in range(H):
        g = hh // (H // G)
        s = ((q[:, hh] @ k[:, g].t()) * m["scale"]).masked_fill(hidden, float("-inf"))
        sink = torch.tensor(-1e9, dtype=h.dtype) if no_sink else w[p + "sink"][hh]
        out[:, hh] = sink_softmax(s, sink.expand(S)) @ v[:, g]
    return out.reshape(S, H * dv) @ w[p + "o"].t()


# --------------------------------------------------------------------------------------------- gated delta rule
def short_conv(x, taps, before=None):
    """x [S, C], taps [C, K] (last column: the current token), zeros (or ``before`` [K - 1, C]) ahead; then silu."""
    S, C = x.shape
    K = taps.shape[1]
    pad = torch.zeros(K - 1, C, dtype=x.dtype) if before is None else before
    full = torch.cat([pad, x])
    return silu(sum(full[j:j + S] * taps[:, j] for j in range(K)))


def delta_states(q, k, v, g, beta, state=None):
    """Unit q (scaled), unit k, decay factors g [S, H, d], beta [S, H]; q, k [S, H, d] with one entry per head."""
    S, H, d = g.shape
    st = torch.zeros(H, d, v.shape[2], dtype=q.dtype) if state is None else state
    o = []
    for t in range(S):
        st = g[t][:, :, None] * st
        u = beta[t][:, None] * (v[t] - read(st, k[t]))
        st = st + outer(k[t], u)
        o.append(read(st, q[t]))
    return torch.stack(o), st


def delta_decay(a, A_log, dt_bias, H):
    """a [S, H * d] -> factors [S, H, d]."""
    S = a.shape[0]
    z = softplus(a + dt_bias).reshape(S, H, -1)
    return torch.exp(-torch.exp(A_log)[None, :, None] * z)


def channel_delta(h, w, p, m, eps, conv_cut=None, **kw):
    """``conv_cut``: the convolutions see zeros before this position (a planted mistake)."""
    S, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]

    def conv(name):
        x = h @ w[p + name].t()
        if conv_cut:
            return torch.cat([short_conv(x[:conv_cut], w[p + name + ".conv"]), short_conv(x[conv_cut:], w[p + name + ".conv"])])
        return short_conv(x, w[p + name + ".conv"])
    q = (unit(conv("q").reshape(S, G, d)) * d ** -0.5).repeat_interleave(H // G, 1)
    k = unit(conv("k").reshape(S, G, d)).repeat_interleave(H // G, 1)
    v = conv("v").reshape(S, H, dv)
    beta = sigmoid(h @ w[p + "b"].t())
    g = delta_decay((h @ w[p + "a1"].t()) @ w[p + "a2"].t(), w[p + "A_log"], w[p + "dt_bias"], H)
    o, _ = delta_states(q, k, v, g, beta)
    gate = sigmoid((h @ w[p + "g1"].t()) @ w[p + "g2"].t())
    return ((rms(o, eps) * w[p + "norm"]).reshape(S, H * dv) * gate) @ w[p + "o"].t()


MIXERS = {"retention": retention, "attention": attention, "channel_delta": channel_delta}


def feed_forward(x, w, p):
    return (gelu_tanh(x @ w[p + "gate"].t()) * (x @ w[p + "up"].t())) @ w[p + "down"].t()


def forward(cfg, w, tokens, *, layers_out=None, dtype=torch.float64, plant=None):
    """Logits [S, vocab] of one sequence; appends the stream after every layer to ``layers_out``.  ``plant``:
    {layer: keyword arguments of its mixer} (mistakes that a test must notice)."""
    w = {k: v.to(dtype) for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{layer.get('weights_of', i)}."
        h = model_norm(x, w[p + "norm1"], eps)
        x = x + MIXERS[layer["type"]](h, w, p + "mix.", layer["mixer"], eps, **(plant or {}).get(i, {}))
        if layer.get("mlp"):
            x = x + feed_forward(model_norm(x, w[p + "norm2"], eps), w, p + "mlp.")
        if layers_out is not None:
            layers_out.append(x)
    return model_norm(x, w["final.norm"], eps) @ w["head"].t() * cfg["logit_scale"]
