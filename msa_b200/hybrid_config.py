"""Configuration of the layered decoder designs: a list of layers, each with its own mixer and feed-forward, read from
a checkpoint's config.json.  Every size and constant that a checkpoint can choose is a field here; the constants that a
design fixes are fields too, with the design's value as the default, so that another design can use the mechanism with
its own."""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import List, Optional, Tuple, Union


@dataclass(frozen=True)
class LatentAttentionSpec:
    """Attention whose keys and values are expanded from one shared latent of size ``kv_rank``; ``rot_dim`` further
    query / key dimensions are rotated (neighbouring pairs), the key's being shared by all heads."""
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot_base: float
    window: Optional[int]          # tokens a query sees, itself included; None: all

    kind = "latent_attention"

    @classmethod
    def parse(cls, m: dict) -> "LatentAttentionSpec":
        rot = m["rot"]
        if rot.get("dims", m["rot_dim"]) != m["rot_dim"]:
            raise ValueError(f"latent_attention: rot.dims {rot['dims']} differs from rot_dim {m['rot_dim']}")
        mask = m.get("mask") or {}
        return cls(heads=int(m["heads"]), dim=int(m["dim"]), rot_dim=int(m["rot_dim"]), vdim=int(m["vdim"]),
                   kv_rank=int(m["kv_rank"]), scale=float(m["scale"]), rot_base=float(rot["base"]),
                   window=int(mask["size"]) if mask.get("size") is not None else None)


@dataclass(frozen=True)
class DeltaSpec:
    """Gated delta rule behind a short causal convolution of ``taps`` taps; ``heads / kv_heads`` value heads share a
    query / key head."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int

    kind = "delta"

    @classmethod
    def parse(cls, m: dict) -> "DeltaSpec":
        spec = cls(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), taps=int(m["conv"]))
        if spec.heads % spec.kv_heads:
            raise ValueError(f"delta: {spec.heads} heads are not a multiple of {spec.kv_heads} kv_heads")
        return spec

    @property
    def channels(self) -> int:
        return 2 * self.kv_heads * self.dim + self.heads * self.vdim


@dataclass(frozen=True)
class DenseSpec:
    ff: int
    kind = "dense"

    @classmethod
    def parse(cls, m: dict) -> "DenseSpec":
        return cls(ff=int(m["ff"]))


@dataclass(frozen=True)
class MoeSpec:
    """``top`` of ``experts`` small feed-forwards per token, clamped at ``limit``."""
    experts: int
    top: int
    ff: int
    limit: float
    kind = "moe"

    @classmethod
    def parse(cls, m: dict) -> "MoeSpec":
        return cls(experts=int(m["router"]["experts"]), top=int(m["router"]["top"]), ff=int(m["expert"]["ff"]),
                   limit=float(m["expert"]["limit"]))


MIXERS = {c.kind: c for c in (LatentAttentionSpec, DeltaSpec)}
FEED_FORWARDS = {c.kind: c for c in (DenseSpec, MoeSpec)}


@dataclass(frozen=True)
class LayerSpec:
    mixer: Union[LatentAttentionSpec, DeltaSpec]
    mlp: Optional[Union[DenseSpec, MoeSpec]]


@dataclass(frozen=True)
class LoopSpec:
    """Layers ``start .. stop-1`` run ``times`` times in a row."""
    start: int
    stop: int
    times: int


@dataclass(frozen=True)
class HybridConfig:
    architecture: str
    vocab: int
    width: int
    eps: float
    layers: Tuple[LayerSpec, ...]
    loop: Optional[LoopSpec]

    @classmethod
    def parse(cls, raw: dict) -> "HybridConfig":
        layers: List[LayerSpec] = []
        for i, entry in enumerate(raw["layers"]):
            if entry["type"] not in MIXERS:
                raise ValueError(f"layer {i}: unknown mixer {entry['type']!r}")
            mlp = entry.get("mlp")
            if mlp is not None and mlp["kind"] not in FEED_FORWARDS:
                raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
            layers.append(LayerSpec(mixer=MIXERS[entry["type"]].parse(entry["mixer"]),
                                    mlp=None if mlp is None else FEED_FORWARDS[mlp["kind"]].parse(mlp)))
        loop = raw.get("loop")
        if loop is not None:
            loop = LoopSpec(int(loop["start"]), int(loop["stop"]), int(loop["times"]))
            if not (0 <= loop.start < loop.stop <= len(layers) and loop.times >= 1):
                raise ValueError(f"loop {loop} does not fit {len(layers)} layers")
        return cls(architecture=raw.get("architecture", ""), vocab=int(raw["vocab"]), width=int(raw["width"]),
                   eps=float(raw["norm"]["eps"]), layers=tuple(layers), loop=loop)

    @classmethod
    def from_pretrained(cls, path: str) -> "HybridConfig":
        with open(os.path.join(path, "config.json")) as f:
            return cls.parse(json.load(f))

    def runs(self) -> List[Tuple[int, Optional[int]]]:
        """(layer, pass or None) in order of execution; every run has a cache or state of its own."""
        n = len(self.layers)
        if self.loop is None:
            return [(i, None) for i in range(n)]
        a, b = self.loop.start, self.loop.stop
        return ([(i, None) for i in range(a)] + [(i, t) for t in range(self.loop.times) for i in range(a, b)]
                + [(i, None) for i in range(b, n)])

    @property
    def num_hidden_layers(self) -> int:
        return len(self.runs())

    @property
    def windows(self) -> Tuple[Optional[int], ...]:
        """The distinct attention windows, in order of appearance."""
        out: List[Optional[int]] = []
        for layer in self.layers:
            if layer.mixer.kind == "latent_attention" and layer.mixer.window not in out:
                out.append(layer.mixer.window)
        return tuple(out)
