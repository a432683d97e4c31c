"""Configuration of the Rununex decoder family: a list of pre-norm layers (layer norm without bias, residual sums times a constant), each a
mixer and an optional feed-forward.  Mixers: "parallel" (chunked soft-max attention with a logarithmic distance bias, a sink and an
element-wise output gate, side by side with a Mamba-2 state space) and "attention" (differential attention behind short convolutions and a
partial rotation, chunked).  The feed-forward is a mixture of experts whose sigmoid weights multiply the experts' inputs, plus a shared
expert.  Every size and constant is read from the checkpoint's `config.json`; nothing is assumed equal between layers."""
from __future__ import annotations

import json
import os
from dataclasses import dataclass, field
from typing import List, Optional

from .configuration_lekapel import RotarySpec


def _chunk(d: dict) -> Optional[int]:
    size = (d.get("mask") or {}).get("size")
    return int(size) if size is not None else None


def _rotary(d: Optional[dict], dim: int) -> Optional[RotarySpec]:
    """columns 2 i and 2 i + 1 turn together"""
    if not d:
        return None
    s = d.get("scaling")
    base, dims = float(d.get("base", 10000.0)), int(d.get("dims", dim))
    if not s:
        return RotarySpec(base, dims)
    return RotarySpec(base, dims, factor=float(s["factor"]), low=float(s["low"]), high=float(s["high"]), original=float(s["original"]))


@dataclass
class BiasedSinkAttentionSpec:
    heads: int
    kv_heads: int
    dim: int                       # query / key size per head
    vdim: int
    scale: float
    chunk: Optional[int]           # position i sees j <= i with floor(j / chunk) == floor(i / chunk); None: every earlier position

    @classmethod
    def from_dict(cls, d: dict) -> "BiasedSinkAttentionSpec":
        heads, dim = int(d["heads"]), int(d["dim"])
        return cls(heads=heads, kv_heads=int(d.get("kv_heads", heads)), dim=dim, vdim=int(d.get("vdim", dim)), scale=float(d.get("scale", dim ** -0.5)), chunk=_chunk(d))

    def cache_row_width(self) -> int:
        return self.kv_heads * (self.dim + self.vdim)


@dataclass
class StateSpaceSpec:
    heads: int
    vdim: int
    state_size: int
    groups: int                    # B and C runs, shared by heads / groups heads each
    conv: int                      # taps of the causal filter over x, B and C
    norm_groups: int               # equal parts of the gated output that are normed on their own

    @classmethod
    def from_dict(cls, d: dict) -> "StateSpaceSpec":
        return cls(heads=int(d["heads"]), vdim=int(d["vdim"]), state_size=int(d["state"]), groups=int(d.get("groups", 1)), conv=int(d.get("conv", 1)),
                   norm_groups=int(d.get("norm_groups", 1)))

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def channels(self) -> int:
        return self.inner + 2 * self.groups * self.state_size

    def state_width(self) -> int:
        """the state matrices, then the last conv - 1 inputs of every filtered channel"""
        return self.inner * self.state_size + (self.conv - 1) * self.channels


@dataclass
class ParallelSpec:
    left: BiasedSinkAttentionSpec
    right: StateSpaceSpec
    left_scale: float
    right_scale: float

    @classmethod
    def from_dict(cls, d: dict) -> "ParallelSpec":
        return cls(BiasedSinkAttentionSpec.from_dict(d["left"]), StateSpaceSpec.from_dict(d["right"]), float(d.get("left_scale", 1.0)), float(d.get("right_scale", 1.0)))

    @property
    def chunk(self) -> Optional[int]:
        return self.left.chunk

    def cache_row_width(self) -> int:
        return self.left.cache_row_width()

    def state_width(self) -> int:
        return self.right.state_width()


@dataclass
class DifferentialAttentionSpec:
    heads: int
    kv_heads: int
    dim: int                       # query / key size per head and map
    vdim: int
    scale: float
    diff: float                    # the fixed part of the second map's factor; the result is scaled by 1 - diff
    conv: int                      # taps of the causal filter over q, k and v
    rot: Optional[RotarySpec]
    chunk: Optional[int]

    @classmethod
    def from_dict(cls, d: dict) -> "DifferentialAttentionSpec":
        heads, dim = int(d["heads"]), int(d["dim"])
        return cls(heads=heads, kv_heads=int(d.get("kv_heads", heads)), dim=dim, vdim=int(d.get("vdim", dim)), scale=float(d.get("scale", dim ** -0.5)), diff=float(d["diff"]),
                   conv=int(d.get("conv", 1)), rot=_rotary(d.get("rot"), dim), chunk=_chunk(d))

    @property
    def channels(self) -> int:
        return 2 * (self.heads + self.kv_heads) * self.dim + self.kv_heads * self.vdim

    def cache_row_width(self) -> int:
        return self.kv_heads * (2 * self.dim + self.vdim)

    def state_width(self) -> int:
        return (self.conv - 1) * self.channels


@dataclass
class MlpSpec:
    kind: str                      # "moe": sigmoid router whose weights multiply the experts' inputs, gated-SiLU experts, a shared expert
    ff: int
    experts: int
    top: int
    shared_ff: Optional[int]

    @classmethod
    def from_dict(cls, d: Optional[dict]) -> Optional["MlpSpec"]:
        if d is None:
            return None
        if d["kind"] != "moe":
            raise ValueError(f"unknown feed-forward kind {d['kind']!r}")
        return cls("moe", int(d["expert"]["ff"]), int(d["router"]["experts"]), int(d["router"]["top"]), int(d["shared"]["ff"]) if d.get("shared") else None)


@dataclass
class LayerSpec:
    type: str
    mixer: object
    mlp: Optional[MlpSpec]


MIXER_SPECS = {"parallel": ParallelSpec, "attention": DifferentialAttentionSpec}


@dataclass
class RununexConfig:
    architecture: str = "Rununex"
    vocab: int = 0
    width: int = 0
    norm_eps: float = 1e-5
    embedding_scale: float = 1.0
    residual_mult: float = 1.0
    logit_scale: float = 1.0
    layers: List[LayerSpec] = field(default_factory=list)

    @classmethod
    def from_dict(cls, d: dict) -> "RununexConfig":
        layers = []
        for i, l in enumerate(d["layers"]):
            if l["type"] not in MIXER_SPECS:
                raise ValueError(f"layer {i}: unknown mixer type {l['type']!r}")
            layers.append(LayerSpec(l["type"], MIXER_SPECS[l["type"]].from_dict(l["mixer"]), MlpSpec.from_dict(l.get("mlp"))))
        return cls(architecture=d.get("architecture", "Rununex"), vocab=int(d["vocab"]), width=int(d["width"]), norm_eps=float((d.get("norm") or {}).get("eps", 1e-5)),
                   embedding_scale=float((d.get("embedding") or {}).get("scale", 1.0)), residual_mult=float(d.get("residual_mult", 1.0)), logit_scale=float(d.get("logit_scale", 1.0)),
                   layers=layers)

    @classmethod
    def from_pretrained(cls, path: str) -> "RununexConfig":
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
        """The chunk lengths of the layers, when every layer's mask is chunked (then keys before the start of the current chunk of
        the longest chunk length are never read again); None when some layer reads every earlier position."""
        c = [l.mixer.chunk for l in self.layers]
        return None if any(x is None for x in c) else c
