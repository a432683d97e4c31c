"""Configuration of the Lipadra decoder family: a list of layers whose RMS norms follow the residual sums, x <- norm(alpha x + sublayer(x)).
Mixers: "attention" (chunked soft-max attention with one added to the denominator), "retention" (linear attention with a fixed decay per
head) and "mamba1" (the selective scan).  The feed-forward is a mixture of experts behind a grouped soft-max router, some of whose choices
are identity experts, plus a gated shared expert (or none).  A layer may use another layer's tensors, with a cache or state of its own.
Every size and constant is read from the checkpoint's `config.json`; nothing is assumed equal between layers."""
from __future__ import annotations

import json
import os
from dataclasses import dataclass, field
from typing import List, Optional

from .configuration_lekapel import RotarySpec


def _rotary(d: Optional[dict], dim: int) -> Optional[RotarySpec]:
    """columns i and i + dims / 2 turn together"""
    if not d:
        return None
    spec = RotarySpec(float(d.get("base", 10000.0)), int(d.get("dims", dim)), layout="halves")
    if spec.dims % 2 or spec.dims > dim:
        raise ValueError(f"a rotation of {spec.dims} columns does not fit heads of {dim}")
    return spec if spec.dims else None


@dataclass
class PlusOneAttentionSpec:
    heads: int
    kv_heads: int
    dim: int                       # query / key size per head
    vdim: int
    scale: float
    rot: Optional[RotarySpec]
    chunk: Optional[int]           # position i sees j <= i with floor(j / chunk) == floor(i / chunk); None: every earlier position

    @classmethod
    def from_dict(cls, d: dict) -> "PlusOneAttentionSpec":
        heads, dim = int(d["heads"]), int(d["dim"])
        size = (d.get("mask") or {}).get("size")
        return cls(heads=heads, kv_heads=int(d.get("kv_heads", heads)), dim=dim, vdim=int(d.get("vdim", dim)), scale=float(d.get("scale", dim ** -0.5)), rot=_rotary(d.get("rot"), dim),
                   chunk=int(size) if size is not None else None)

    def cache_row_width(self) -> int:
        return self.kv_heads * (self.dim + self.vdim)

    def state_width(self) -> int:
        return 0


@dataclass
class RetentionSpec:
    heads: int
    dim: int                       # query / key size per head
    vdim: int
    decay: List[float]             # one per head
    rot: Optional[RotarySpec]

    @classmethod
    def from_dict(cls, d: dict) -> "RetentionSpec":
        heads, dim, decay = int(d["heads"]), int(d["dim"]), [float(x) for x in d["decay"]]
        if len(decay) != heads or not all(0.0 < x <= 1.0 for x in decay):
            raise ValueError(f"retention: one decay in (0, 1] for each of {heads} heads")
        return cls(heads=heads, dim=dim, vdim=int(d.get("vdim", dim)), decay=decay, rot=_rotary(d.get("rot"), dim))

    def cache_row_width(self) -> int:
        return 0

    def state_width(self) -> int:
        return self.heads * self.dim * self.vdim


@dataclass
class SelectiveScanSpec:
    inner: int                     # channels
    state_size: int                # numbers per channel
    dt_rank: int
    conv: int                      # taps of the causal filter

    @classmethod
    def from_dict(cls, d: dict) -> "SelectiveScanSpec":
        return cls(inner=int(d["inner"]), state_size=int(d["state"]), dt_rank=int(d["dt_rank"]), conv=int(d.get("conv", 1)))

    def cache_row_width(self) -> int:
        return 0

    def state_width(self) -> int:
        """the state, then the last conv - 1 inputs of every channel"""
        return self.inner * (self.state_size + self.conv - 1)


@dataclass
class MlpSpec:
    kind: str                      # "moe": grouped soft-max router, gated-SiLU experts, identity experts, a gated shared expert
    ff: int
    experts: int                   # experts with tensors
    identity: int                  # router outputs behind them whose expert is the identity
    top: int
    groups: int                    # equal groups of neighbouring router outputs, of which the best `keep_groups` can be chosen from
    keep_groups: int
    out_scale: float
    shared_ff: Optional[int]

    @classmethod
    def from_dict(cls, d: Optional[dict]) -> Optional["MlpSpec"]:
        if d is None:
            return None
        if d["kind"] != "moe":
            raise ValueError(f"unknown feed-forward kind {d['kind']!r}")
        r = d["router"]
        g = r.get("groups") or {}
        count = int(g.get("count", 1))
        return cls("moe", int(d["expert"]["ff"]), experts=int(r["experts"]), identity=int(r.get("identity") or 0), top=int(r["top"]), groups=count,
                   keep_groups=int(g.get("keep", count)), out_scale=float(r.get("scale", 1.0)), shared_ff=int(d["shared"]["ff"]) if d.get("shared") else None)


@dataclass
class LayerSpec:
    type: str
    mixer: object
    mlp: Optional[MlpSpec]
    weights_of: int                # the layer whose tensors this one uses; itself as a rule


MIXER_SPECS = {"attention": PlusOneAttentionSpec, "retention": RetentionSpec, "mamba1": SelectiveScanSpec}


@dataclass
class LipadraConfig:
    architecture: str = "Lipadra"
    vocab: int = 0
    width: int = 0
    norm_eps: float = 1e-6
    alpha: float = 1.0
    layers: List[LayerSpec] = field(default_factory=list)

    @classmethod
    def from_dict(cls, d: dict) -> "LipadraConfig":
        layers: List[LayerSpec] = []
        owner = [l.get("weights_of") for l in d["layers"]]
        for i, l in enumerate(d["layers"]):
            if l["type"] not in MIXER_SPECS:
                raise ValueError(f"layer {i}: unknown mixer type {l['type']!r}")
            j, seen = i, {i}
            while owner[j] is not None:
                j = int(owner[j])
                if j in seen or not 0 <= j < len(owner):
                    raise ValueError(f"layer {i}: weights_of does not lead to a layer with tensors")
                seen.add(j)
            if j != i and d["layers"][j]["type"] != l["type"]:
                raise ValueError(f"layer {i} uses the tensors of layer {j}, whose mixer is of another type")
            layers.append(LayerSpec(l["type"], MIXER_SPECS[l["type"]].from_dict(l["mixer"]), MlpSpec.from_dict(l.get("mlp")), j))
        for i, l in enumerate(layers):
            o = layers[l.weights_of]
            if (l.mixer, l.mlp) != (o.mixer, o.mlp):
                raise ValueError(f"layer {i} uses the tensors of layer {l.weights_of} but describes other sizes or constants")
        return cls(architecture=d.get("architecture", "Lipadra"), vocab=int(d["vocab"]), width=int(d["width"]), norm_eps=float((d.get("norm") or {}).get("eps", 1e-6)),
                   alpha=float(d.get("postln_alpha", 1.0)), layers=layers)

    @classmethod
    def from_pretrained(cls, path: str) -> "LipadraConfig":
        with open(os.path.join(path, "config.json") if os.path.isdir(path) else path) as f:
            return cls.from_dict(json.load(f))

    # what the cache manager asks of a model
    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    def cache_row_widths(self) -> List[int]:
        return [l.mixer.cache_row_width() for l in self.layers]

    def state_widths(self) -> List[int]:
        return [l.mixer.state_width() for l in self.layers]

    def chunks(self) -> Optional[List[int]]:
        """The chunk lengths of the attention layers, when each of them has one (then keys before the start of the current chunk of the
        longest chunk length are never read again); None when some attention layer reads every earlier position.  No attention layer at
        all: chunks of one token (no layer keeps rows)."""
        c = [l.mixer.chunk for l in self.layers if l.type == "attention"]
        return None if any(x is None for x in c) else c or [1]
