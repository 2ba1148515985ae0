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
class GroupedAttentionSpec:
    """Grouped-query attention over a sliding window, queries, keys and values behind a short causal convolution of ``taps``
    taps; the first ``rot_dims`` dimensions of a head are rotated (neighbouring pairs).  ``sink``: one is added to the
    softmax denominators; ``gate``: every head's output is multiplied by the sigmoid of a projection of the layer's input."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot_dims: int
    rot_base: float
    window: Optional[int]          # tokens a query sees, itself included; None: all
    taps: int
    sink: bool = True
    gate: bool = True

    kind = "attention"

    @classmethod
    def parse(cls, m: dict) -> "GroupedAttentionSpec":
        rot, mask = m.get("rot") or {"dims": 0, "base": 1.0}, m.get("mask") or {}
        spec = cls(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), scale=float(m["scale"]),
                   rot_dims=int(rot["dims"]), rot_base=float(rot["base"]), taps=int(m["conv"]),
                   window=int(mask["size"]) if mask.get("size") is not None else None)
        if spec.heads % spec.kv_heads:
            raise ValueError(f"attention: {spec.heads} heads are not a multiple of {spec.kv_heads} kv_heads")
        if spec.rot_dims % 2 or not 0 <= spec.rot_dims <= spec.dim:
            raise ValueError(f"attention: {spec.rot_dims} rotated dimensions do not fit heads of {spec.dim}")
        return spec

    @property
    def channels(self) -> int:
        return (self.heads + self.kv_heads) * self.dim + self.kv_heads * self.vdim


@dataclass(frozen=True)
class WkvSpec:
    """Recurrence with a decay per key channel and a bonus for the current token; every projection reads its own mix of the
    token's input and the previous token's."""
    heads: int
    dim: int

    kind = "wkv"

    @classmethod
    def parse(cls, m: dict) -> "WkvSpec":
        return cls(heads=int(m["heads"]), dim=int(m["dim"]))

    @property
    def inner(self) -> int:
        return self.heads * self.dim


@dataclass(frozen=True)
class Mamba2Spec:
    """State-space recurrence with one decay per head behind a short convolution; ``heads / groups`` heads share keys and
    queries of size ``state``; the gated output is normalised in ``norm_groups`` parts."""
    heads: int
    vdim: int
    state: int
    groups: int
    norm_groups: int
    taps: int

    kind = "mamba2"

    @classmethod
    def parse(cls, m: dict) -> "Mamba2Spec":
        spec = cls(heads=int(m["heads"]), vdim=int(m["vdim"]), state=int(m["state"]), groups=int(m["groups"]),
                   norm_groups=int(m["norm_groups"]), taps=int(m["conv"]))
        if spec.heads % spec.groups or spec.inner % spec.norm_groups:
            raise ValueError(f"mamba2: {spec.groups} groups / {spec.norm_groups} norm groups do not divide {spec.heads} heads of {spec.vdim}")
        return spec

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def channels(self) -> int:
        return self.inner + 2 * self.groups * self.state


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


MIXERS = {c.kind: c for c in (LatentAttentionSpec, DeltaSpec, GroupedAttentionSpec, WkvSpec, Mamba2Spec)}
FEED_FORWARDS = {c.kind: c for c in (DenseSpec, MoeSpec)}


@dataclass(frozen=True)
class LayerSpec:
    mixer: Union[LatentAttentionSpec, DeltaSpec, GroupedAttentionSpec, WkvSpec, Mamba2Spec]
    mlp: Optional[Union[DenseSpec, MoeSpec]]


@dataclass(frozen=True)
class LoopSpec:
    """Layers ``start .. stop-1`` run ``times`` times in a row."""
    start: int
    stop: int
    times: int


@dataclass(frozen=True)
class BigramSpec:
    """An embedding row per hashed (previous token, token) beside the token's own."""
    buckets: int
    mul_prev: int
    mul_cur: int


@dataclass(frozen=True)
class Structure:
    """What a design fixes about the frame around its layers."""
    block: str                     # "sandwich": mixer, then feed-forward, a norm on both sides of each;
    #                                "parallel": both from the same stream, through a norm each
    loop_input: str                # how a looped pass starts: "project" (a product over [stream, embedding], every pass) or
    #                                "add" (the embedding joins the stream, every pass but the first)
    norm_offset: float             # added to the stored norm weights
    tied: bool                     # the embedding is the output matrix


DESIGNS = {
    "Mutuvik": Structure(block="sandwich", loop_input="project", norm_offset=0.0, tied=True),
    "Nazerax": Structure(block="parallel", loop_input="add", norm_offset=1.0, tied=False),
}


@dataclass(frozen=True)
class HybridConfig:
    architecture: str
    vocab: int
    width: int
    eps: float
    layers: Tuple[LayerSpec, ...]
    loop: Optional[LoopSpec]
    structure: Structure
    bigram: Optional[BigramSpec] = None
    logit_softcap: Optional[float] = None

    @classmethod
    def parse(cls, raw: dict) -> "HybridConfig":
        if raw.get("architecture") not in DESIGNS:
            raise ValueError(f"unknown architecture {raw.get('architecture')!r} (known: {sorted(DESIGNS)})")
        structure = DESIGNS[raw["architecture"]]
        layers: List[LayerSpec] = []
        for i, entry in enumerate(raw["layers"]):
            if entry["type"] not in MIXERS:
                raise ValueError(f"layer {i}: unknown mixer {entry['type']!r}")
            mlp = entry.get("mlp")
            if mlp is not None and mlp["kind"] not in FEED_FORWARDS:
                raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
            if structure.block == "parallel" and mlp is not None and mlp["kind"] != "dense":
                raise ValueError(f"layer {i}: a parallel block takes a dense feed-forward")
            layers.append(LayerSpec(mixer=MIXERS[entry["type"]].parse(entry["mixer"]),
                                    mlp=None if mlp is None else FEED_FORWARDS[mlp["kind"]].parse(mlp)))
        loop = raw.get("loop")
        if loop is not None:
            loop = LoopSpec(int(loop["start"]), int(loop["stop"]), int(loop["times"]))
            if not (0 <= loop.start < loop.stop <= len(layers) and loop.times >= 1):
                raise ValueError(f"loop {loop} does not fit {len(layers)} layers")
        pair, cap = (raw.get("embedding") or {}).get("bigram"), raw.get("logit_softcap")
        if pair is not None:
            pair = BigramSpec(int(pair["buckets"]), int(pair["mul_prev"]), int(pair["mul_cur"]))
        return cls(architecture=raw["architecture"], vocab=int(raw["vocab"]), width=int(raw["width"]),
                   eps=float(raw["norm"]["eps"]), layers=tuple(layers), loop=loop, structure=structure, bigram=pair,
                   logit_softcap=None if cap is None else float(cap))

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
            if hasattr(layer.mixer, "window") and layer.mixer.window not in out:
                out.append(layer.mixer.window)
        return tuple(out)
