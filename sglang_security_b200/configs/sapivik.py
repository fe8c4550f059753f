"""Configuration of the Sapivik design: a decoder-only model over a 32-bit residual with an RMS norm on both
sides of every sublayer and a residual multiplier,

    x += m * post_1(mixer(pre_1(x)))        x += m * post_2(ff(pre_2(x)))

whose mixers are channel-gated matrix memories ("hgrn2") or grouped-query attention with tied keys and values
("attention"), whose feed-forwards are clamped gated MLPs ("dense"), mixtures with identity experts and a
gated shared expert ("moe") or absent, and in which a range of layers may run several times in a row.  Every
size, the order and the loop of the layers and the constants a model may choose are read from config.json."""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import List, Optional, Tuple, Union

from .model_config import register_config


@dataclass
class ChannelMemorySpec:
    heads: int
    dim: int                     # channels of a query / forget gate
    vdim: int


@dataclass
class TiedAttentionSpec:
    heads: int
    kv_heads: int
    dim: int                     # query, key and value size (a value is the projected key)
    scale: float
    softcap: float               # 0 = none
    rope_base: float
    rope_dims: int               # rotated leading coordinates of a head (0 = no rotation)


@dataclass
class ClampedSpec:
    ff: int
    limit: float


@dataclass
class IdentityExpertsSpec:
    experts: int                 # experts with matrices
    identity: int                # experts that return their input, scored after the others
    top: int
    scale: float                 # factor on the router weights
    ff: int
    shared_ff: int               # 0 = no shared expert


@dataclass
class SapivikLayerSpec:
    type: str
    mixer: Union[ChannelMemorySpec, TiedAttentionSpec]
    mlp: Union[ClampedSpec, IdentityExpertsSpec, None]


@dataclass
class SapivikConfig:
    vocab: int
    width: int
    eps: float
    residual_mult: float
    loop: Tuple[int, int, int]   # first layer, one past the last, passes
    layers: List[SapivikLayerSpec] = field(default_factory=list)

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    def layer_runs(self) -> List[Tuple[int, bool]]:
        """(layer, whether the embedding output is added ahead of it) of every layer run, in order.  A run's
        place in this list names its cache rows or state."""
        start, stop, times = self.loop
        runs = [(i, False) for i in range(start)]
        for turn in range(times):
            runs += [(i, turn > 0 and i == start) for i in range(start, stop)]
        return runs + [(i, False) for i in range(stop, len(self.layers))]


def _mixer(kind: str, m: dict) -> Union[ChannelMemorySpec, TiedAttentionSpec]:
    heads, dim = int(m["heads"]), int(m["dim"])
    vdim = int(m.get("vdim", dim))
    if min(heads, dim, vdim) < 1:
        raise ValueError(f"{heads} heads of sizes {dim} / {vdim}")
    if kind == "hgrn2":
        return ChannelMemorySpec(heads=heads, dim=dim, vdim=vdim)
    if kind != "attention":
        raise ValueError(f"unknown mixer type {kind!r}")
    kv_heads = int(m.get("kv_heads", heads))
    if kv_heads < 1 or heads % kv_heads:
        raise ValueError(f"{heads} query heads cannot share {kv_heads} key/value heads")
    if vdim != dim:
        raise ValueError(f"values are the keys: value size {vdim} must be the key size {dim}")
    rot = m.get("rot") or {}
    dims = int(rot.get("dims", dim)) if rot else 0
    if dims % 2 or not 0 <= dims <= dim:
        raise ValueError(f"rotated coordinates {dims} must be even and at most the head size {dim}")
    return TiedAttentionSpec(heads=heads, kv_heads=kv_heads, dim=dim, scale=float(m["scale"]),
                             softcap=float(m.get("softcap") or 0.0), rope_base=float(rot.get("base", 10000.0)),
                             rope_dims=dims)


def _mlp(f: Optional[dict]) -> Union[ClampedSpec, IdentityExpertsSpec, None]:
    if not f:
        return None
    if f.get("kind") == "dense":
        if not float(f["limit"]) > 0:
            raise ValueError(f"clamp limit {f['limit']} must be positive")
        return ClampedSpec(ff=int(f["ff"]), limit=float(f["limit"]))
    if f.get("kind") != "moe":
        raise ValueError(f"unknown feed-forward kind {f.get('kind')!r}")
    r = f["router"]
    spec = IdentityExpertsSpec(experts=int(r["experts"]), identity=int(r.get("identity") or 0), top=int(r["top"]),
                               scale=float(r.get("scale", 1.0)), ff=int(f["expert"]["ff"]),
                               shared_ff=int((f.get("shared") or {}).get("ff") or 0))
    if spec.experts < 1 or spec.identity < 0 or not 0 < spec.top <= spec.experts + spec.identity:
        raise ValueError(f"top {spec.top} of {spec.experts} + {spec.identity} experts")
    return spec


@register_config("Sapivik")
def sapivik_config(raw: dict) -> SapivikConfig:
    layers: List[SapivikLayerSpec] = []
    for i, L in enumerate(raw["layers"]):
        try:
            layers.append(SapivikLayerSpec(type=L["type"], mixer=_mixer(L["type"], L["mixer"]), mlp=_mlp(L.get("mlp"))))
        except ValueError as e:
            raise ValueError(f"layer {i}: {e}") from None
    loop = raw.get("loop")
    start, stop, times = (int(loop["start"]), int(loop["stop"]), int(loop["times"])) if loop else (0, 0, 1)
    if not 0 <= start <= stop <= len(layers) or times < 1:
        raise ValueError(f"loop over layers {start} .. {stop - 1}, {times} times, of {len(layers)} layers")
    return SapivikConfig(vocab=int(raw["vocab"]), width=int(raw["width"]), eps=float(raw["norm"]["eps"]),
                         residual_mult=float(raw.get("residual_mult", 1.0)), loop=(start, stop, times), layers=layers)
