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

    recurrent = False

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
    """Grouped-query softmax attention: own key and value sizes, norms over the whole q and k projections, no
    rotation, query temperature, one sink logit per head."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    q_temp: Optional[QueryTemperature] = None
    projection_norm: bool = True
    sinks: bool = True

    recurrent = False

    @staticmethod
    def from_dict(d: dict) -> "GroupedMixerSpec":
        t = d.get("q_temp")
        s = GroupedMixerSpec(int(d["heads"]), int(d["kv_heads"]), int(d["dim"]), int(d["vdim"]), float(d["scale"]),
                             QueryTemperature(float(t["coef"]), int(t["every"])) if t else None)
        if s.heads % s.kv_heads:
            raise ValueError(f"{s.heads} query heads do not divide over {s.kv_heads} key/value heads")
        return s

    def num_params(self, h: int) -> int:
        return h * (self.heads * self.dim + self.kv_heads * (self.dim + self.vdim)) + self.heads * self.vdim * h


@dataclass(frozen=True)
class RetentionMixerSpec:
    """Linear attention with one fixed decay per head and rotated queries and keys."""
    heads: int
    dim: int
    vdim: int
    rot: RotarySpec
    decay: tuple

    recurrent = True

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

    recurrent = True

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


MixerSpec = Union[LatentMixerSpec, GroupedMixerSpec, RetentionMixerSpec, DeltaMixerSpec]
MIXER_TYPES = {"latent_attention": LatentMixerSpec, "attention": GroupedMixerSpec, "retention": RetentionMixerSpec,
               "channel_delta": DeltaMixerSpec}


@dataclass(frozen=True)
class LayerSpec:
    """One entry of a checkpoint configuration that lists its layers one by one."""
    mixer: MixerSpec
    ff: int = 0                          # width of the dense feed-forward, 0 = the layer has none
    act: str = "gelu"
    gated: bool = False                  # down(act(gate) * up) instead of down(act(up))
    weights_of: Optional[int] = None     # layer whose weights this one runs with (its cache and state are its own)

    def num_params(self, h: int) -> int:
        if self.weights_of is not None:
            return 0
        return self.mixer.num_params(h) + (3 if self.gated else 2) * h * self.ff


def layer_specs(layers: list, mixers: tuple, act: str, gated: bool) -> list:
    """``LayerSpec`` of every entry of a configuration's layer list; ``mixers``: the types the design has."""
    specs: list = []
    for i, layer in enumerate(layers):
        if layer["type"] not in mixers:
            raise ValueError(f"layer {i}: unknown mixer type {layer['type']!r}")
        mlp = layer.get("mlp")
        if mlp and mlp.get("kind") != "dense":
            raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
        spec = LayerSpec(MIXER_TYPES[layer["type"]].from_dict(layer["mixer"]), int(mlp["ff"]) if mlp else 0, act, gated)
        specs.append(spec)
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
