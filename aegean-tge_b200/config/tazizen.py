"""Typed configuration of the Tazizen decoder, read from config.json.

A Tazizen model keeps several residual streams (hyper-connections): every sublayer reads one combination of them and writes
them all.  A layer's mixer is a grouped attention with rotated, unit-RMS queries and keys, or attention over a latent cache;
both look at a sliding window.  Everything that may differ between two models of the design is in config.json::

    architecture        "Tazizen"
    vocab, width        vocabulary and width of a residual stream
    streams             how many streams
    norm.eps            epsilon of every RMS norm
    loop                absent, or {start, stop, times}: layers start..stop-1 run ``times`` times in a row
    layers[i].type      "attention" or "latent_attention"
    layers[i].mixer     attention:        heads, kv_heads, dim, vdim, scale, rot, mask
                        latent_attention: heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, rot, mask
                        rot   {base, dims, scaling {factor, original, fast, slow} (absent: none)} (absent: no rotation)
                        mask  {size} (absent: every earlier token is visible)
    layers[i].mlp       null, or {"kind": "moe", "expert": {"ff"}, "router": {"experts", "top", "scale", "groups" {count,
                        keep} (absent: one group)}, "shared": {"ff"} (absent or null: none)}

The design states no longest sequence: the engine's ``context`` alone bounds a request.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Tuple

from .common import ConfigError
from .kokolorn import Loop, _object
from .lepizen import _int, _number

ARCHITECTURE = "Tazizen"
MAX_STREAMS = 16            # what the kernels of the residual streams take


@dataclass(frozen=True)
class Stretch:
    factor: float
    original: float
    fast: float
    slow: float

    def to_dict(self) -> Dict[str, Any]:
        return {"factor": self.factor, "original": self.original, "fast": self.fast, "slow": self.slow}


@dataclass(frozen=True)
class Rotation:
    base: float
    dims: int                           # the first so many numbers of a head are rotated, in halves
    scaling: Optional[Stretch] = None

    def to_dict(self) -> Dict[str, Any]:
        out: Dict[str, Any] = {"base": self.base, "dims": self.dims}
        if self.scaling is not None:
            out["scaling"] = self.scaling.to_dict()
        return out


def _with_view(out: Dict[str, Any], rot: Optional[Rotation], window: Optional[int]) -> Dict[str, Any]:
    if rot is not None:
        out["rot"] = rot.to_dict()
    if window is not None:
        out["mask"] = {"size": window}
    return out


@dataclass(frozen=True)
class Attention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Optional[Rotation]
    window: Optional[int]

    def to_dict(self) -> Dict[str, Any]:
        return _with_view({"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale},
                          self.rot, self.window)


@dataclass(frozen=True)
class LatentAttention:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot: Optional[Rotation]
    window: Optional[int]

    def to_dict(self) -> Dict[str, Any]:
        return _with_view({"heads": self.heads, "dim": self.dim, "rot_dim": self.rot_dim, "vdim": self.vdim, "q_rank": self.q_rank,
                           "kv_rank": self.kv_rank, "scale": self.scale}, self.rot, self.window)


@dataclass(frozen=True)
class Experts:
    ff: int
    experts: int
    top: int
    scale: float
    group_count: int
    group_keep: int
    shared_ff: Optional[int]

    def to_dict(self) -> Dict[str, Any]:
        router: Dict[str, Any] = {"experts": self.experts, "top": self.top, "scale": self.scale,
                                  "groups": {"count": self.group_count, "keep": self.group_keep}}
        out: Dict[str, Any] = {"kind": "moe", "expert": {"ff": self.ff}, "router": router}
        if self.shared_ff is not None:
            out["shared"] = {"ff": self.shared_ff}
        return out


@dataclass(frozen=True)
class TazizenLayer:
    kind: str                           # "attention" or "latent_attention"
    mixer: Any                          # Attention or LatentAttention
    mlp: Optional[Experts]


def _rotation(where: str, m: Dict[str, Any], width: int) -> Optional[Rotation]:
    if m.get("rot") is None:
        return None
    raw = _object(where, m, "rot")
    dims = _int(where + "rot.", raw, "dims", minimum=0)
    if dims % 2 or dims > width:
        raise ConfigError(f"config.json: {where}rot.dims {dims} must be even and within {width}")
    base = _number(where + "rot.", raw, "base")
    scaling = None
    if raw.get("scaling") is not None:
        s = _object(where + "rot.", raw, "scaling")
        at = where + "rot.scaling."
        scaling = Stretch(factor=_number(at, s, "factor"), original=_number(at, s, "original"), fast=_number(at, s, "fast"),
                          slow=_number(at, s, "slow"))
        if base == 1.0:
            raise ConfigError(f"config.json: {where}rot.base must differ from 1 to be scaled")
    return Rotation(base=base, dims=dims, scaling=scaling) if dims else None


def _window(where: str, m: Dict[str, Any]) -> Optional[int]:
    return None if m.get("mask") is None else _int(where + "mask.", _object(where, m, "mask"), "size")


def _attention(where: str, m: Dict[str, Any]) -> Attention:
    heads, kv_heads, dim = _int(where, m, "heads"), _int(where, m, "kv_heads"), _int(where, m, "dim")
    if heads % kv_heads:
        raise ConfigError(f"config.json: {where}{heads} heads are not a multiple of {kv_heads} kv_heads")
    return Attention(heads=heads, kv_heads=kv_heads, dim=dim, vdim=_int(where, m, "vdim"),
                     scale=_number(where, m, "scale", positive=False), rot=_rotation(where, m, dim), window=_window(where, m))


def _latent(where: str, m: Dict[str, Any]) -> LatentAttention:
    rot_dim = _int(where, m, "rot_dim", minimum=0)
    return LatentAttention(heads=_int(where, m, "heads"), dim=_int(where, m, "dim"), rot_dim=rot_dim, vdim=_int(where, m, "vdim"),
                           q_rank=_int(where, m, "q_rank"), kv_rank=_int(where, m, "kv_rank"),
                           scale=_number(where, m, "scale", positive=False), rot=_rotation(where, m, rot_dim),
                           window=_window(where, m))


def _mlp(where: str, mlp: Any) -> Optional[Experts]:
    if mlp is None:
        return None
    if not isinstance(mlp, dict) or mlp.get("kind") != "moe":
        raise ConfigError(f"config.json: {where}'mlp' must be null or of kind 'moe', got {mlp!r}")
    router = _object(where + "mlp.", mlp, "router")
    at = where + "mlp.router."
    experts, top = _int(at, router, "experts"), _int(at, router, "top")
    count = keep = 1
    if router.get("groups") is not None:
        groups = _object(at, router, "groups")
        count, keep = _int(at + "groups.", groups, "count"), _int(at + "groups.", groups, "keep")
    if experts % count or keep > count or top > experts // count * keep:
        raise ConfigError(f"config.json: {at}{top} of {experts} experts do not fit {keep} of {count} groups")
    if experts > 1024:
        raise ConfigError(f"config.json: {at}experts {experts}: the router takes up to 1024")
    shared = None if mlp.get("shared") is None else _int(where + "mlp.shared.", _object(where + "mlp.", mlp, "shared"), "ff")
    return Experts(ff=_int(where + "mlp.expert.", _object(where + "mlp.", mlp, "expert"), "ff"), experts=experts, top=top,
                   scale=1.0 if router.get("scale") is None else _number(at, router, "scale", positive=False),
                   group_count=count, group_keep=keep, shared_ff=shared)


@dataclass(frozen=True)
class TazizenConfig:
    vocab: int
    width: int
    streams: int
    eps: float
    layers: Tuple[TazizenLayer, ...]
    loop: Optional[Loop]

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    def run_order(self) -> Tuple[int, ...]:
        """The layers in the order they run."""
        count = len(self.layers)
        if self.loop is None:
            return tuple(range(count))
        once = tuple(range(self.loop.start, self.loop.stop))
        return tuple(range(self.loop.start)) + once * self.loop.times + tuple(range(self.loop.stop, count))

    @staticmethod
    def from_dict(raw: Dict[str, Any]) -> "TazizenConfig":
        vocab = _int("", raw, "vocab")
        if vocab >= 2 ** 31:
            raise ConfigError(f"config.json: vocab {vocab} does not fit 32-bit token ids")
        streams = _int("", raw, "streams")
        if streams > MAX_STREAMS:
            raise ConfigError(f"config.json: 'streams' {streams}: at most {MAX_STREAMS}")
        listed = raw.get("layers")
        if not isinstance(listed, list) or not listed:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers: List[TazizenLayer] = []
        for index, entry in enumerate(listed):
            where = f"layers[{index}]."
            if not isinstance(entry, dict):
                raise ConfigError(f"config.json: layers[{index}] must be an object")
            kind, m = entry.get("type"), _object(where, entry, "mixer")
            if kind == "attention":
                mixer: Any = _attention(where + "mixer.", m)
            elif kind == "latent_attention":
                mixer = _latent(where + "mixer.", m)
            else:
                raise ConfigError(f"config.json: {where}'type' must be 'attention' or 'latent_attention', got {kind!r}")
            layers.append(TazizenLayer(kind=kind, mixer=mixer, mlp=_mlp(where, entry.get("mlp"))))
        loop = None
        if raw.get("loop") is not None:
            lp = _object("", raw, "loop")
            loop = Loop(start=_int("loop.", lp, "start", minimum=0), stop=_int("loop.", lp, "stop"), times=_int("loop.", lp, "times"))
            if not loop.start < loop.stop <= len(layers):
                raise ConfigError(f"config.json: loop runs layers {loop.start}..{loop.stop - 1} of {len(layers)}")
        return TazizenConfig(vocab=vocab, width=_int("", raw, "width"), streams=streams,
                             eps=_number("norm.", _object("", raw, "norm"), "eps"), layers=tuple(layers), loop=loop)

    def to_dict(self) -> Dict[str, Any]:
        out: Dict[str, Any] = {"architecture": ARCHITECTURE, "vocab": self.vocab, "width": self.width, "streams": self.streams,
                               "norm": {"eps": self.eps},
                               "layers": [{"type": layer.kind, "mixer": layer.mixer.to_dict(),
                                           "mlp": None if layer.mlp is None else layer.mlp.to_dict()} for layer in self.layers]}
        if self.loop is not None:
            out["loop"] = self.loop.to_dict()
        return out
