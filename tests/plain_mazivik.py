"""Plain, slow statement of the Mazivik decoder, one function per mechanism.

Everything is written out on whole sequences without a cache, in the dtype of the tensors it is given
(float64 in the tests), and shares no code with the package.  ``cfg`` is the dictionary of a Mazivik
``config.json``; ``w`` maps checkpoint tensor names to tensors.
"""
import math

import torch


def layer_norm(x, weight, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * weight


def rms_norm(x, weight, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight


def gelu_erf(z):
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def softcap(z, cap):
    return cap * torch.tanh(z / cap)


def rotary_frequencies(rot):
    """(frequency of every pair, multiplier of cos and sin)."""
    dims, base = rot["dims"], rot["base"]
    freqs = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    s = rot.get("scaling")
    if not s:
        return freqs, 1.0

    def turning_dim(turns):
        return dims * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(turning_dim(s["fast"])), 0)
    hi = min(math.ceil(turning_dim(s["slow"])), dims - 1)
    out = []
    for i, f in enumerate(freqs):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / s["factor"] * r + f * (1.0 - r))
    return out, 0.1 * math.log(s["factor"]) + 1.0


def rotate_pairs(x, positions, rot):
    """x [S, ..., d]: dimensions (2i, 2i + 1) turned by position * frequency_i; dims beyond rot.dims pass."""
    freqs, mult = rotary_frequencies(rot)
    out = x.clone()
    for i, f in enumerate(freqs):
        c = torch.tensor([mult * math.cos(p * f) for p in positions], dtype=x.dtype)
        n = torch.tensor([mult * math.sin(p * f) for p in positions], dtype=x.dtype)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        c, n = (t.reshape(-1, *[1] * (u.dim() - 1)) for t in (c, n))
        out[..., 2 * i] = u * c - v * n
        out[..., 2 * i + 1] = v * c + u * n
    return out


def latent_of(h, w, p, m, eps):
    """(latent c, rotated shared key part) of every position: what a cache would hold."""
    y = h @ w[p + "dkv"].t()
    c = rms_norm(y[:, :m["kv_rank"]], w[p + "dkv.norm"], eps)
    k_rot = rotate_pairs(y[:, m["kv_rank"]:], range(h.shape[0]), m["rot"])
    return c, k_rot


def causal_softmax(scores, hidden_keys=()):
    """Softmax over the keys j <= i; ``hidden_keys`` leaves out a key that should be seen (a planted mistake)."""
    S = scores.shape[-1]
    masked = torch.ones(S, S, dtype=torch.bool).triu(1)
    for k in hidden_keys:
        masked[k + 1:, k] = True
    scores = scores.masked_fill(masked, float("-inf"))
    e = torch.exp(scores - scores.max(-1, keepdim=True).values)
    return e / e.sum(-1, keepdim=True)


def latent_attention(h, w, p, m, eps, c, k_rot, hidden_keys=()):
    """Mixer output [S, width].  c, k_rot: this layer's latent, or the one of the layer it shares."""
    S, H, dn, dr, dv = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    q = rms_norm(h @ w[p + "dq"].t(), w[p + "dq.norm"], eps) @ w[p + "uq"].t()
    q = q.reshape(S, H, dn + dr)
    q_rot = rotate_pairs(q[..., dn:], range(S), m["rot"])
    k = (c @ w[p + "uk"].t()).reshape(S, H, dn)
    v = (c @ w[p + "uv"].t()).reshape(S, H, dv)
    scores = torch.einsum("qhd,khd->hqk", q[..., :dn], k) + torch.einsum("qhd,kd->hqk", q_rot, k_rot)
    o = torch.einsum("hqk,khd->qhd", causal_softmax(scores * m["scale"], hidden_keys), v).reshape(S, H * dv)
    return (o * torch.sigmoid(h @ w[p + "g"].t())) @ w[p + "o"].t()


def feed_forward(x, w, p):
    return gelu_erf(x @ w[p + "up"].t()) @ w[p + "down"].t()


def forward(cfg, w, tokens, *, layers_out=None, dtype=torch.float64, hidden_keys=()):
    """Logits [S, vocab] of one sequence; appends the residual stream after every layer to ``layers_out``."""
    w = {k: v.to(dtype) for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    latents = {}
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}.mix."
        src = m.get("kv_from")
        if src is None:
            latents[i] = latent_of(x, w, p, m, eps)
        y = latent_attention(x, w, p, m, eps, *latents[i if src is None else src], hidden_keys)
        x = x + layer_norm(y, w[f"l{i}.norm1"], eps)
        if layer.get("mlp"):
            x = x + layer_norm(feed_forward(x, w, f"l{i}.mlp."), w[f"l{i}.norm2"], eps)
        if layers_out is not None:
            layers_out.append(x)
    z = layer_norm(x, w["final.norm"], eps) @ w["head"].t()
    cap = cfg.get("logit_softcap")
    return softcap(z, cap) if cap else z


def random_model(cfg, seed=0, gain=1.0):
    """Weights of ``cfg`` (bfloat16), scaled so that activations stay of order one."""
    g = torch.Generator().manual_seed(seed)

    def mat(o, i):
        return (torch.randn(o, i, generator=g) * gain / math.sqrt(i)).bfloat16()

    def vec(n):
        return (1.0 + 0.3 * torch.randn(n, generator=g)).bfloat16()
    D = cfg["width"]
    w = {"embed": torch.randn(cfg["vocab"], D, generator=g).bfloat16(), "final.norm": vec(D),
         "head": mat(cfg["vocab"], D)}
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}.mix."
        H, dn, dr, dv, L, Q = (m[k] for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank"))
        w[f"l{i}.norm1"] = vec(D)
        w[p + "dq"], w[p + "dq.norm"], w[p + "uq"] = mat(Q, D), vec(Q), mat(H * (dn + dr), Q)
        if m.get("kv_from") is None:
            w[p + "dkv"], w[p + "dkv.norm"] = mat(L + dr, D), vec(L)
        w[p + "uk"], w[p + "uv"] = mat(H * dn, L), mat(H * dv, L)
        w[p + "g"], w[p + "o"] = mat(H * dv, D), mat(D, H * dv)
        if layer.get("mlp"):
            F = layer["mlp"]["ff"]
            w[f"l{i}.norm2"], w[f"l{i}.mlp.up"], w[f"l{i}.mlp.down"] = vec(D), mat(F, D), mat(D, F)
    return w
