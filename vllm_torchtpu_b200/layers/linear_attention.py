"""Linear-attention mixers over the carried-state kernels (``ops.linear_attention``): retention, gated linear attention
and two delta rules with one decay per key channel.

    retention       row = [W_q ‖ W_k ‖ W_v ‖ W_g] x;  rotation, S <- decay_h S + k v^T, o = S^T q, norm, silu gate
    channel delta   row = [W_q ‖ W_k ‖ W_v ‖ W_a1 ‖ W_g1 ‖ W_b] x;  decays W_a2 row_a1, gate W_g2 row_g1, short
                    convolutions, unit q and k, delta rule, norm, sigmoid gate
    gated linear    row = [W_q ‖ W_k ‖ W_v ‖ W_g ‖ W_a1] x;  decays W_a2 row_a1 + b per channel, norm, silu gate
    removal         row = [W_r ‖ W_k ‖ W_v ‖ W_g ‖ W_a ‖ W_w1] x;  decays W_w2 tanh(row_w1) + w0 and removal rates per
                    channel, both on the old state; norm over the head with a weight per head, sigmoid gate

followed by W_o.  Heads are sharded over TP, the low ranks are replicated.  A cache is (state,) or (ring, state), both
indexed by the request's batch slot and independent of the KV pages.
"""
from __future__ import annotations

import torch

from .. import ops
from ..config import ModelConfig
from ..layer_specs import DeltaMixerSpec, GlaMixerSpec, RemovalMixerSpec, RetentionMixerSpec
from ..ops.linear_attention import LinearAttentionPlan
from ..parallel.state import get_state
from .linear import RowParallelLinear, seeded_normal
from .packed import PackedLinear, PaddedColumnLinear, Part


class CarriedStateMixer:
    """What both mixers share: the plan, the pools, speculative rollback and the output projection."""
    plan: LinearAttentionPlan

    def _begin(self, name, spec, cfg, device):
        st = get_state()
        self.name, self.spec, self.cfg, self.device = name, spec, cfg, device
        self.tp, self.rank = st.tp.size, st.tp.rank_in_group
        if spec.heads % self.tp:
            raise ValueError(f"{name}: {spec.heads} heads do not divide over tp={self.tp}")
        self.H = spec.heads // self.tp

    def heads_of(self, full: torch.Tensor) -> torch.Tensor:
        """This rank's part of a per-head vector."""
        n = full.shape[0] // self.tp
        return full[self.rank * n:(self.rank + 1) * n].to(device=self.device, dtype=torch.float32).contiguous()

    def init_dummy(self, std: float, seed: int) -> None:
        for lin in self.linears():
            lin.init_dummy(std, seed)

    def weight_bytes(self) -> int:
        return sum(l.weight_bytes() for l in self.linears())

    def allocate_cache(self, num_blocks: int, block_size: int, kv_dtype, device, slots: int):
        p = self.plan
        state = torch.zeros(p.state_shape(slots), dtype=torch.float32, device=device)
        return (torch.zeros(p.ring_shape(slots), dtype=self.cfg.dtype, device=device), state) if p.taps else (state,)

    def bytes_per_block(self, block_size: int, elem: int) -> int:
        return 0

    def recur(self, inputs, meta, cache, out=None):
        """The stateful part over the rows ``meta`` describes; advances the pools in place.  inputs: (row,), (row, decays)
        or (row, decays, gate), a gate that is not among them is in the row."""
        row, decay_in, gate = tuple(inputs) + (None,) * (3 - len(inputs))
        gate = self.gate_of(row) if gate is None else gate
        return ops.carried_state_attention(self.plan, row, decay_in, gate, meta, cache, out)

    def gate_of(self, row):
        at = self.inp.offset[self.gate_part]
        return row[:, at:at + self.H * self.spec.vdim]

    gate_part = "g"                      # part of the packed projection that holds the output gate

    def advance(self, inputs, cache, meta, out=None):
        rb = getattr(meta, "state_rollback", None)
        if rb is not None:
            rb.capture(self, cache, inputs)        # verification step: rejected drafts are rolled back later
        return self.recur(inputs, meta, cache, out)

    def forward(self, x, cache, meta):
        return self.o(self.advance(self.project(x), cache, meta))


class Retention(CarriedStateMixer):
    def __init__(self, name: str, spec: RetentionMixerSpec, cfg: ModelConfig, device, quant=None):
        self._begin(name, spec, cfg, device)
        kw = dict(dtype=cfg.dtype, device=device, quant_config=quant)
        H, d, dv = spec.heads, spec.dim, spec.vdim
        self.inp = PackedLinear(f"{name}.qkvg_proj", cfg.hidden_size, [
            Part("q", H * d, H), Part("k", H * d, H), Part("v", H * dv, H), Part("g", H * dv, H)], **kw)
        self.o = RowParallelLinear(f"{name}.o_proj", H * dv, cfg.hidden_size, **kw)
        at = self.inp.offset
        self.plan = LinearAttentionPlan(
            self.H, self.H, d, dv, (at["q"], at["k"], at["v"]), "silu", cfg.rms_norm_eps, k_mult=d ** -0.5,
            inv_freq=ops.ref.rope_inv_freq(spec.rot.dims, spec.rot.base).to(device),
            decay=self.heads_of(torch.tensor(spec.decay, dtype=torch.float64)))

    def linears(self):
        return [self.inp, self.o]

    def project(self, x):
        return (self.inp(x),)


class ChannelDelta(CarriedStateMixer):
    def __init__(self, name: str, spec: DeltaMixerSpec, cfg: ModelConfig, device, quant=None):
        self._begin(name, spec, cfg, device)
        if spec.kv_heads % self.tp:
            raise ValueError(f"{name}: {spec.kv_heads} query/key heads do not divide over tp={self.tp}")
        kw = dict(dtype=cfg.dtype, device=device, quant_config=quant)
        H, G, d, dv, r = spec.heads, spec.kv_heads, spec.dim, spec.vdim, spec.rank
        self.inp = PackedLinear(f"{name}.in_proj", cfg.hidden_size, [
            Part("q", G * d, G), Part("k", G * d, G), Part("v", H * dv, H), Part("a1", r), Part("g1", r),
            Part("b", H, H)], **kw)
        self.a2 = PaddedColumnLinear(f"{name}.a2_proj", r, H * d, **kw)
        self.g2 = PaddedColumnLinear(f"{name}.g2_proj", r, H * dv, **kw)
        self.o = RowParallelLinear(f"{name}.o_proj", H * dv, cfg.hidden_size, **kw)
        self.plan = LinearAttentionPlan(
            self.H, G // self.tp, d, dv, (0, 0, 0), "sigmoid", cfg.rms_norm_eps, q_mult=d ** -0.5, unit_norm=True,
            norm_w=torch.ones(dv, dtype=torch.float32, device=device), taps=spec.conv)
        self._place()

    def _place(self) -> None:
        at = self.inp.offset
        self.plan.offsets, self.plan.beta_offset = (at["q"], at["k"], at["v"]), at["b"]

    def linears(self):
        return [self.inp, self.a2, self.g2, self.o]

    # ---- weights ---------------------------------------------------------------
    def load_projections(self, q, k, v, a1, g1, b, a2, g2) -> None:
        """The ranks of the two low-rank projections come with their tensors."""
        self.inp.resize(a1=a1.shape[0], g1=g1.shape[0])
        self.a2.full_in, self.g2.full_in = a1.shape[0], g1.shape[0]
        self._place()
        self.inp.load_weight(torch.cat([q, k, v, a1, g1, b], 0))
        self.a2.load_weight(a2)
        self.g2.load_weight(g2)

    def load_conv(self, q, k, v) -> None:
        parts = []
        for w in (q, k, v):
            n = w.shape[0] // self.tp
            parts.append(w[self.rank * n:(self.rank + 1) * n])
        self.plan.conv_w = torch.cat(parts, 0).to(device=self.device, dtype=self.cfg.dtype).contiguous()

    def load_vectors(self, A_log, dt_bias, norm) -> None:
        self.plan.A_log, self.plan.dt_bias = self.heads_of(A_log), self.heads_of(dt_bias)
        self.plan.norm_w.copy_(norm)

    def init_dummy(self, std: float, seed: int) -> None:
        super().init_dummy(std, seed)
        s = self.spec

        def vec(leaf, *shape, scale=0.5, dtype=torch.float32):
            return seeded_normal(f"{self.name}.{leaf}", shape, scale, dtype, self.device, seed)
        n, dt = s.kv_heads * s.dim, self.cfg.dtype
        self.load_conv(vec("q_conv", n, s.conv, dtype=dt), vec("k_conv", n, s.conv, dtype=dt),
                       vec("v_conv", s.heads * s.vdim, s.conv, dtype=dt))
        self.load_vectors(vec("A_log", s.heads), vec("dt_bias", s.heads * s.dim), torch.ones(s.vdim))

    # ---- forward ---------------------------------------------------------------
    def project(self, x):
        row = self.inp(x)
        at = self.inp.offset
        a = self.a2(row[:, at["a1"]:at["a1"] + self.a2.padded_in])
        gate = self.g2(row[:, at["g1"]:at["g1"] + self.g2.padded_in])
        return row, a, gate


class GatedLinear(CarriedStateMixer):
    def __init__(self, name: str, spec: GlaMixerSpec, cfg: ModelConfig, device, quant=None):
        self._begin(name, spec, cfg, device)
        kw = dict(dtype=cfg.dtype, device=device, quant_config=quant)
        H, d, dv, r = spec.heads, spec.dim, spec.vdim, spec.rank
        self.inp = PackedLinear(f"{name}.in_proj", cfg.hidden_size, [
            Part("q", H * d, H), Part("k", H * d, H), Part("v", H * dv, H), Part("g", H * dv, H), Part("a1", r)], **kw)
        self.a2 = PaddedColumnLinear(f"{name}.a2_proj", r, H * d, **kw)
        self.o = RowParallelLinear(f"{name}.o_proj", H * dv, cfg.hidden_size, **kw)
        at = self.inp.offset
        self.plan = LinearAttentionPlan(
            self.H, self.H, d, dv, (at["q"], at["k"], at["v"]), "silu", cfg.rms_norm_eps, q_mult=d ** -0.5,
            norm_w=torch.ones(dv, dtype=torch.float32, device=device), rule="channel", tau=spec.tau,
            dt_bias=torch.zeros(self.H * d, dtype=torch.float32, device=device))

    def linears(self):
        return [self.inp, self.a2, self.o]

    def load_projections(self, q, k, v, g, a1, a2) -> None:
        """The rank of the decay projection comes with its tensors; its part is the last one."""
        self.inp.resize(a1=a1.shape[0])
        self.a2.full_in = a1.shape[0]
        self.inp.load_weight(torch.cat([q, k, v, g, a1], 0))
        self.a2.load_weight(a2)

    def load_vectors(self, decay_bias, norm) -> None:
        self.plan.dt_bias.copy_(self.heads_of(decay_bias))
        self.plan.norm_w.copy_(norm)

    def init_dummy(self, std: float, seed: int) -> None:
        super().init_dummy(std, seed)
        self.load_vectors(2.0 + seeded_normal(f"{self.name}.a2_bias", (self.spec.heads * self.spec.dim,), 1.0, torch.float32,
                                              self.device, seed), torch.ones(self.spec.vdim))

    def project(self, x):
        row = self.inp(x)
        at = self.inp.offset["a1"]
        return row, self.a2(row[:, at:at + self.a2.padded_in])


class RemovalDelta(CarriedStateMixer):
    """Its projections of the input are parts of ``inp``, which the owner computes and shares with another mixer; the owner
    applies the output projection too."""
    gate_part = "right.g"

    @staticmethod
    def parts(spec: RemovalMixerSpec) -> list:
        H, n = spec.heads, spec.heads * spec.dim
        return [Part("right." + p, n, H) for p in "rkvga"] + [Part("right.w1", spec.rank)]

    def __init__(self, name: str, spec: RemovalMixerSpec, cfg: ModelConfig, device, inp: PackedLinear, quant=None):
        self._begin(name, spec, cfg, device)
        H, d = self.H, spec.dim
        self.inp = inp
        self.w2 = PaddedColumnLinear(f"{name}.w2_proj", spec.rank, spec.heads * d, dtype=cfg.dtype, device=device,
                                     quant_config=quant)
        at = inp.offset
        zeros = lambda: torch.zeros(H * d, dtype=torch.float32, device=device)          # noqa: E731
        self.plan = LinearAttentionPlan(
            H, H, d, d, tuple(at["right." + p] for p in "rkv"), "sigmoid", cfg.rms_norm_eps,
            norm_w=torch.ones(H * d, dtype=torch.float32, device=device), rule="removal", dt_bias=zeros(),
            rate_offset=at["right.a"], rate_bias=zeros())

    def linears(self):
        return [self.w2]

    def load_vectors(self, w0, rate_bias, norm, norm_mult: float = 1.0) -> None:
        self.plan.dt_bias.copy_(self.heads_of(w0))
        self.plan.rate_bias.copy_(self.heads_of(rate_bias))
        self.plan.norm_w.copy_(self.heads_of(norm) * norm_mult)

    def init_vectors(self, seed: int, norm_mult: float) -> None:
        n = self.spec.heads * self.spec.dim

        def vec(leaf):
            return seeded_normal(f"{self.name}.{leaf}", (n,), 1.0, torch.float32, self.device, seed)
        self.load_vectors(vec("w0"), vec("rate_bias"), torch.ones(n), norm_mult)

    def decays(self, row):
        at = self.inp.offset["right.w1"]
        return self.w2(ops.tanh_(row[:, at:at + self.w2.padded_in]))
