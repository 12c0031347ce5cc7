"""Per-layer sizes of models whose ``config.json`` lists its layers one by one.

A mixer spec holds what one mixer needs (heads, dimensions, rotation, decays); a ``LayerSpec`` joins it with the
layer's feed-forward.  ``ModelConfig.from_layer_list`` builds them."""
from __future__ import annotations

import math
from dataclasses import dataclass, replace
from typing import Optional, Union


@dataclass(frozen=True)
class RotarySpec:
    """Rotary embedding of one mixer: the first ``dims`` dimensions of the rotated vector turn by
    ``position * base^(-2i / dims)``, optionally with YaRN ``scaling`` ({factor, original, fast, slow})."""
    dims: int
    base: float
    scaling: Optional[dict] = None

    @property
    def rope_scaling(self) -> Optional[dict]:
        """The same scaling under the names ``ops.reference.rope_inv_freq`` reads."""
        if not self.scaling:
            return None
        s = self.scaling
        return {"rope_type": "yarn", "factor": float(s["factor"]),
                "original_max_position_embeddings": float(s["original"]), "beta_fast": float(s["fast"]),
                "beta_slow": float(s["slow"]), "attention_factor": 0.1 * math.log(float(s["factor"])) + 1.0}


@dataclass(frozen=True)
class LatentMixerSpec:
    """Sizes of one latent-attention mixer (multi-head latent attention with a query latent)."""
    heads: int
    dim: int                             # unrotated query / key dimensions per head
    rot_dim: int                         # rotated ones (the key's are shared by all heads)
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot: RotarySpec
    kv_from: Optional[int] = None        # layer whose cached latent and rotated key this layer reads
    output_gate: bool = True             # heads times sigmoid(W_g x) in front of the output projection

    recurrent = carries_state = False

    @staticmethod
    def from_dict(d: dict) -> "LatentMixerSpec":
        r = d["rot"]
        rot = RotarySpec(int(r["dims"]), float(r["base"]), r.get("scaling") or None)
        src = d.get("kv_from")
        if rot.dims > d["rot_dim"] or rot.dims % 2:
            raise ValueError(f"rot.dims {rot.dims} must be even and at most rot_dim {d['rot_dim']}")
        return LatentMixerSpec(int(d["heads"]), int(d["dim"]), int(d["rot_dim"]), int(d["vdim"]), int(d["q_rank"]),
                               int(d["kv_rank"]), float(d["scale"]), rot, None if src is None else int(src))

    def num_params(self, h: int) -> int:
        n = h * self.q_rank + self.q_rank * self.heads * (self.dim + self.rot_dim)
        n += self.kv_rank * self.heads * (self.dim + self.vdim) + self.heads * self.vdim * h * (2 if self.output_gate else 1)
        return n + (h * (self.kv_rank + self.rot_dim) if self.kv_from is None else 0)


@dataclass(frozen=True)
class QueryTemperature:
    """The query at position p is multiplied by 1 + coef * ln(floor((p + 1) / every) + 1)."""
    coef: float
    every: int


@dataclass(frozen=True)
class GroupedMixerSpec:
    """Grouped-query softmax attention with own key and value sizes.  Norms over the whole q and k projections, a query
    temperature and sinks; or short convolutions, with a rotation, a window, an output gate or two softmax maps per head
    (differential attention)."""
    heads: int
    kv_heads: int
    dim: int                             # of one map
    vdim: int
    scale: float
    q_temp: Optional[QueryTemperature] = None
    projection_norm: bool = True
    sinks: bool = True                   # one sink logit per head
    conv: int = 0                        # taps of the short convolutions on q, k and v (0: none)
    rot: Optional[RotarySpec] = None     # rotation of interleaved pairs
    window: Optional[int] = None         # keys a query sees, itself included (None: all)
    maps: int = 1                        # softmax maps per head over the same values; 2: map 1 - lambda * map 2
    diff: float = 0.0                    # constant part of lambda
    bias: bool = False                   # of the q, k and v projections
    out_bias: bool = False
    output_gate: bool = False            # heads times sigmoid(W_g x) in front of the output projection
    kv_from: Optional[int] = None        # layer whose cached keys and values this layer reads
    chunk: Optional[int] = None          # a query sees the keys of its own chunk of that many positions (None: no chunks)
    head_temp: bool = False              # scores times one number per query head
    zero_sink: bool = False              # one is added to the denominator of the softmax (a sink logit of 0)

    recurrent = False

    @property
    def carries_state(self) -> bool:
        return self.conv > 0

    @property
    def mask(self) -> Optional[int]:
        """The window, or minus the size of the chunks, as the attention ops take it."""
        return -self.chunk if self.chunk is not None else self.window

    def __post_init__(self):
        if self.heads % self.kv_heads:
            raise ValueError(f"{self.heads} query heads do not divide over {self.kv_heads} key/value heads")
        if self.rot is not None and (self.rot.dims % 2 or self.rot.dims > self.dim):
            raise ValueError(f"rot.dims {self.rot.dims} must be even and at most dim {self.dim}")
        if any(n is not None and n < 1 for n in (self.window, self.chunk)):
            raise ValueError("a window or a chunk holds at least the token itself")
        if self.window is not None and self.chunk is not None:
            raise ValueError("a window and chunks at the same time are not built")

    @staticmethod
    def sizes_of(d: dict) -> tuple:
        return int(d["heads"]), int(d["kv_heads"]), int(d["dim"]), int(d["vdim"]), float(d["scale"])

    @staticmethod
    def from_dict(d: dict) -> "GroupedMixerSpec":
        t = d.get("q_temp")
        return GroupedMixerSpec(*GroupedMixerSpec.sizes_of(d),
                                QueryTemperature(float(t["coef"]), int(t["every"])) if t else None)

    @staticmethod
    def convolved(d: dict, **kw) -> "GroupedMixerSpec":
        """Biased projections behind short convolutions; ``mask.size`` is the window, ``rot`` the rotation."""
        if int(d["conv"]) < 1:
            raise ValueError("a short convolution has at least one tap")
        r, mask, src = d.get("rot"), d.get("mask"), d.get("kv_from")
        rot = RotarySpec(int(r["dims"]), float(r["base"]), r.get("scaling") or None) if r else None
        return GroupedMixerSpec(*GroupedMixerSpec.sizes_of(d), projection_norm=False, sinks=False, conv=int(d["conv"]),
                                rot=rot, window=int(mask["size"]) if mask else None, bias=True,
                                kv_from=None if src is None else int(src), **kw)

    @staticmethod
    def differential(d: dict) -> "GroupedMixerSpec":
        return GroupedMixerSpec.convolved(d, maps=2, diff=float(d["diff"]))

    @staticmethod
    def gated(d: dict) -> "GroupedMixerSpec":
        return GroupedMixerSpec.convolved(d, out_bias=True, output_gate=True)

    @staticmethod
    def chunked(d: dict) -> "GroupedMixerSpec":
        """``mask.size`` is the size of the chunks; a temperature per head and a sink of 0."""
        s = GroupedMixerSpec.convolved(d, head_temp=True, zero_sink=True)
        return replace(s, chunk=s.window, window=None)

    def num_params(self, h: int) -> int:
        n = h * self.heads * (self.maps * self.dim + self.vdim * (2 if self.output_gate else 1))
        return n + (h * self.kv_heads * (self.maps * self.dim + self.vdim) if self.kv_from is None else 0)


@dataclass(frozen=True)
class RetentionMixerSpec:
    """Linear attention with one fixed decay per head and rotated queries and keys."""
    heads: int
    dim: int
    vdim: int
    rot: RotarySpec
    decay: tuple

    recurrent = carries_state = True

    @staticmethod
    def from_dict(d: dict) -> "RetentionMixerSpec":
        rot = RotarySpec(int(d["rot"]["dims"]), float(d["rot"]["base"]))
        s = RetentionMixerSpec(int(d["heads"]), int(d["dim"]), int(d["vdim"]), rot, tuple(float(x) for x in d["decay"]))
        if rot.dims % 2 or rot.dims > s.dim:
            raise ValueError(f"rot.dims {rot.dims} must be even and at most dim {s.dim}")
        if len(s.decay) != s.heads:
            raise ValueError(f"{len(s.decay)} decays for {s.heads} heads")
        return s

    def num_params(self, h: int) -> int:
        return h * self.heads * (2 * self.dim + 3 * self.vdim)


@dataclass(frozen=True)
class DeltaMixerSpec:
    """Gated delta rule with one decay per head and key channel behind short convolutions."""
    heads: int
    kv_heads: int                        # query / key heads, each serves heads / kv_heads value heads
    dim: int
    vdim: int
    conv: int                            # taps of the short convolutions
    gate_rank: int = 0                   # rank of the decay and output gate projections until a checkpoint sets it

    recurrent = carries_state = True

    @staticmethod
    def from_dict(d: dict) -> "DeltaMixerSpec":
        s = DeltaMixerSpec(int(d["heads"]), int(d["kv_heads"]), int(d["dim"]), int(d["vdim"]), int(d["conv"]),
                           int(d.get("gate_rank", 0)))
        if s.heads % s.kv_heads:
            raise ValueError(f"{s.heads} heads do not divide over {s.kv_heads} query/key heads")
        if s.conv < 1:
            raise ValueError("a short convolution has at least one tap")
        return s

    @property
    def rank(self) -> int:
        return self.gate_rank or self.dim

    def num_params(self, h: int) -> int:
        n = h * (2 * self.kv_heads * self.dim + 2 * self.heads * self.vdim + self.heads + 2 * self.rank)
        return n + self.rank * self.heads * (self.dim + self.vdim)


@dataclass(frozen=True)
class GlaMixerSpec:
    """Gated linear attention: one decay sigmoid(z)^(1 / tau) per head and key channel, z from a low-rank projection."""
    heads: int
    dim: int
    vdim: int
    tau: float
    decay_rank: int = 0                  # rank of the decay projection until a checkpoint sets it

    recurrent = carries_state = True

    @staticmethod
    def from_dict(d: dict) -> "GlaMixerSpec":
        s = GlaMixerSpec(int(d["heads"]), int(d["dim"]), int(d["vdim"]), float(d["tau"]), int(d.get("decay_rank", 0)))
        if s.tau <= 0:
            raise ValueError(f"tau {s.tau} must be positive")
        return s

    @property
    def rank(self) -> int:
        return self.decay_rank or 16

    def num_params(self, h: int) -> int:
        return h * (self.heads * (2 * self.dim + 3 * self.vdim) + self.rank) + self.rank * self.heads * self.dim


@dataclass(frozen=True)
class RemovalMixerSpec:
    """Generalised delta rule: one decay and one removal rate per head and key channel, both acting on the old state."""
    heads: int
    dim: int                             # of keys and values alike
    decay_rank: int = 0                  # rank of the decay projection until a checkpoint sets it

    recurrent = carries_state = True

    @property
    def vdim(self) -> int:
        return self.dim

    @staticmethod
    def from_dict(d: dict) -> "RemovalMixerSpec":
        return RemovalMixerSpec(int(d["heads"]), int(d["dim"]), int(d.get("decay_rank", 0)))

    @property
    def rank(self) -> int:
        return self.decay_rank or 16

    def num_params(self, h: int) -> int:
        return h * (6 * self.heads * self.dim + self.rank) + self.rank * self.heads * self.dim


@dataclass(frozen=True)
class ParallelMixerSpec:
    """Two mixers over the same input, y = left_scale * left + right_scale * right; the left one has pages."""
    left: GroupedMixerSpec
    right: RemovalMixerSpec
    left_scale: float
    right_scale: float

    recurrent = False
    carries_state = True

    @staticmethod
    def from_dict(d: dict) -> "ParallelMixerSpec":
        return ParallelMixerSpec(GroupedMixerSpec.chunked(d["left"]), RemovalMixerSpec.from_dict(d["right"]),
                                 float(d["left_scale"]), float(d["right_scale"]))

    @property
    def heads(self) -> int:
        return math.gcd(self.left.heads, self.right.heads)      # what tensor parallelism has to divide

    @property
    def kv_heads(self) -> int:
        return self.left.kv_heads

    def num_params(self, h: int) -> int:
        return self.left.num_params(h) + self.right.num_params(h)


MixerSpec = Union[LatentMixerSpec, GroupedMixerSpec, RetentionMixerSpec, DeltaMixerSpec, GlaMixerSpec, RemovalMixerSpec,
                  ParallelMixerSpec]


@dataclass(frozen=True)
class ExpertsSpec:
    """Mixture of experts: down(act(up(x))), or down(act(gate(x), up(x))), of the ``top`` chosen experts.  Softmax scores
    that are the weights themselves; or sigmoid scores (``sigmoid``), chosen after a correction within the best groups and
    renormalised.  ``shared_ff``: an expert that every token uses, times the sigmoid of one number per token."""
    experts: int
    top: int
    ff: int
    act: str
    gated: bool = False
    sigmoid: bool = False
    groups: int = 1
    keep: int = 1                        # groups whose experts can be chosen
    scale: float = 1.0
    shared_ff: int = 0
    shared_act: str = ""

    def __post_init__(self):
        if not 1 <= self.top <= self.experts:
            raise ValueError(f"top {self.top} of {self.experts} experts")
        if self.groups < 1 or self.experts % self.groups or not 1 <= self.keep <= self.groups:
            raise ValueError(f"{self.keep} of {self.groups} groups of {self.experts} experts")
        if self.top > self.keep * (self.experts // self.groups):
            raise ValueError(f"top {self.top} experts out of {self.keep} groups of {self.experts // self.groups}")

    @staticmethod
    def from_dict(d: dict, act: str) -> "ExpertsSpec":
        return ExpertsSpec(int(d["router"]["experts"]), int(d["router"]["top"]), int(d["expert"]["ff"]), act)

    @staticmethod
    def clamped(d: dict, act: str) -> "ExpertsSpec":
        """Gated experts whose gate and up projections are clamped at ``limit``, behind sigmoid scores in groups."""
        r, g, sh = d["router"], d["router"].get("groups") or {}, d.get("shared")
        groups = int(g.get("count", 1))
        return ExpertsSpec(int(r["experts"]), int(r["top"]), int(d["expert"]["ff"]), f"{act}:{float(d['expert']['limit'])}",
                           gated=True, sigmoid=True, groups=groups, keep=int(g.get("keep", groups)),
                           scale=float(r.get("scale", 1.0)), shared_ff=int(sh["ff"]) if sh else 0,
                           shared_act=f"{act}:{float(sh['limit'])}" if sh else "")

    def num_params(self, h: int) -> int:
        n = 3 if self.gated else 2
        return self.experts * h * (n * self.ff + 1) + (h * (3 * self.shared_ff + 1) if self.shared_ff else 0)


@dataclass(frozen=True)
class LayerSpec:
    """One entry of a checkpoint configuration that lists its layers one by one."""
    mixer: MixerSpec
    ff: int = 0                          # width of the dense feed-forward, 0 = the layer has none (or experts)
    act: str = "gelu"
    gated: bool = False                  # down(act(gate) * up) instead of down(act(up))
    weights_of: Optional[int] = None     # layer whose weights this one runs with (its cache and state are its own)
    experts: Optional[ExpertsSpec] = None
    token_shift: bool = False            # the mixer's input is mixed with the one of the token before
    side_dim: int = 0                    # width of the layer's own token input behind the feed-forward (0: none)

    @property
    def carries_state(self) -> bool:
        return self.token_shift or self.mixer.carries_state

    def num_params(self, h: int) -> int:
        if self.weights_of is not None:
            return 0
        n = self.mixer.num_params(h) + (3 if self.gated else 2) * h * self.ff + 2 * h * self.side_dim
        return n + (self.experts.num_params(h) if self.experts else 0)


def layer_specs(layers: list, mixers: dict, act: str, gated: bool, expert_act: Optional[str] = None,
                experts=ExpertsSpec.from_dict, dense: bool = True) -> list:
    """``LayerSpec`` of every entry of a configuration's layer list.  ``mixers``: the types the design has and the
    functions that read them; ``expert_act``: activation of its experts (None: it has none), ``experts``: the function that
    reads them; ``dense``: it has dense feed-forwards."""
    kinds = (["dense"] if dense else []) + (["moe"] if expert_act else [])
    specs: list = []
    for i, layer in enumerate(layers):
        if layer["type"] not in mixers:
            raise ValueError(f"layer {i}: unknown mixer type {layer['type']!r}")
        mlp = layer.get("mlp")
        kind = mlp.get("kind") if mlp else None
        if mlp and kind not in kinds:
            raise ValueError(f"layer {i}: unknown feed-forward kind {kind!r}")
        specs.append(LayerSpec(mixers[layer["type"]](layer["mixer"]), int(mlp["ff"]) if kind == "dense" else 0, act, gated,
                               experts=experts(mlp, expert_act) if kind == "moe" else None))
    for i, layer in enumerate(layers):
        src, seen = layer.get("weights_of"), {i}
        if src is None:
            continue
        while layers[src].get("weights_of") is not None and src not in seen:
            seen.add(src)
            src = layers[src]["weights_of"]
        if src in seen:
            raise ValueError(f"layer {i}: weights_of leads back to the layer itself")
        if (specs[i].mixer, specs[i].ff) != (specs[src].mixer, specs[src].ff):
            raise ValueError(f"layer {i}: its sizes differ from those of layer {src}, whose weights it uses")
        specs[i] = replace(specs[i], weights_of=int(src))
    return specs
