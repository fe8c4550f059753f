"""Configuration of the Luzosun design: a decoder-only model of parallel blocks over a 32-bit residual,

    x <- x + (mixer(c(norm1(x))) + ff(norm2(x))),      c(h) = h + causal convolution of h,

whose mixer is differential attention (two softmax maps per query head over one value head, subtracted
and normed) behind short convolutions on q, k and v, seen in chunks of positions, optionally reading the
keys and values another layer cached; the feed-forward is an ungated MLP with the xIELU activation or
absent.  Every size, the layer order and the constants a model may choose are read from config.json."""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import List, Optional

from .model_config import register_config


@dataclass
class DifferentialSpec:
    heads: int
    kv_heads: int
    dim: int                     # query/key size of ONE map (a head has two)
    vdim: int                    # value size
    scale: float
    diff: float                  # base of the second map's weight; 1 - diff scales the normed difference
    chunk: Optional[int]         # positions per chunk (a position sees its own chunk only); None = all before
    conv: int                    # taps of the convolution on q, k and v (0 = none)
    rope_base: float
    rope_dims: int               # rotated leading coordinates of each map (0 = no rotation)
    rope_factor: float           # every frequency is divided by this
    kv_from: Optional[int]       # layer whose cached keys and values this layer reads


@dataclass
class UngatedSpec:
    ff: int


@dataclass
class LuzosunLayerSpec:
    type: str
    mixer: DifferentialSpec
    mlp: Optional[UngatedSpec]


@dataclass
class LuzosunConfig:
    vocab: int
    width: int
    eps: float
    embedding_scale: float
    canon_taps: int              # taps of the convolution on the mixer's input (0 = none)
    layers: List[LuzosunLayerSpec] = field(default_factory=list)

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    def resolve_shapes(self, shapes) -> None:
        """The taps of a convolution are its tensor's second size: shapes = {tensor name: shape}."""
        canon = {int(shapes[f"l{i}.canon1"][1]) for i in range(len(self.layers)) if f"l{i}.canon1" in shapes}
        if len(canon) == 1:
            self.canon_taps = canon.pop()
        for i, L in enumerate(self.layers):
            if f"l{i}.mix.q.conv" in shapes:
                L.mixer.conv = int(shapes[f"l{i}.mix.q.conv"][1])


def _mixer(m: dict) -> DifferentialSpec:
    heads, kv_heads = int(m["heads"]), int(m.get("kv_heads", m["heads"]))
    if kv_heads < 1 or heads % kv_heads:
        raise ValueError(f"{heads} query heads cannot share {kv_heads} key/value heads")
    mask, rot = m.get("mask") or {}, m.get("rot") or {}
    dims = int(rot.get("dims", m["dim"])) if rot else 0
    if dims % 2 or dims > int(m["dim"]):
        raise ValueError(f"rotated coordinates {dims} must be even and at most the map size {m['dim']}")
    factor = float((rot.get("scaling") or {}).get("factor", 1.0))
    if not factor > 0:
        raise ValueError(f"rotation factor {factor} must be positive")
    src = m.get("kv_from")
    return DifferentialSpec(heads=heads, kv_heads=kv_heads, dim=int(m["dim"]), vdim=int(m["vdim"]),
                            scale=float(m["scale"]), diff=float(m["diff"]),
                            chunk=int(mask["size"]) if mask.get("size") else None, conv=int(m.get("conv") or 0),
                            rope_base=float(rot.get("base", 10000.0)), rope_dims=dims, rope_factor=factor,
                            kv_from=int(src) if src is not None else None)


def _mlp(f: Optional[dict]) -> Optional[UngatedSpec]:
    if not f:
        return None
    if f.get("kind") != "dense":
        raise ValueError(f"unknown feed-forward kind {f.get('kind')!r}")
    return UngatedSpec(ff=int(f["ff"]))


@register_config("Luzosun")
def luzosun_config(raw: dict) -> LuzosunConfig:
    layers: List[LuzosunLayerSpec] = []
    for i, L in enumerate(raw["layers"]):
        if L["type"] != "attention":
            raise ValueError(f"layer {i}: unknown mixer type {L['type']!r}")
        try:
            spec = LuzosunLayerSpec(type=L["type"], mixer=_mixer(L["mixer"]), mlp=_mlp(L.get("mlp")))
        except ValueError as e:
            raise ValueError(f"layer {i}: {e}") from None
        src = spec.mixer.kv_from
        if src is not None:
            if not 0 <= src < i or layers[src].mixer.kv_from is not None:
                raise ValueError(f"layer {i}: kv_from {src} must name an earlier layer with its own keys and values")
            a, b = spec.mixer, layers[src].mixer
            if (a.kv_heads, a.dim, a.vdim) != (b.kv_heads, b.dim, b.vdim):
                raise ValueError(f"layer {i}: key/value sizes differ from layer {src}")
        layers.append(spec)
    return LuzosunConfig(vocab=int(raw["vocab"]), width=int(raw["width"]), eps=float(raw["norm"]["eps"]),
                         embedding_scale=float((raw.get("embedding") or {}).get("scale", 1.0)),
                         canon_taps=int((raw.get("canon") or {}).get("taps") or 0), layers=layers)
