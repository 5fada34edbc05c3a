"""Typed configuration of the Fesorax decoder, read from config.json.

A Fesorax model is a list of layers that normalise after each sum (x <- norm(alpha x + sublayer(x))), the sublayers
reading the stream itself.  A layer's mixer is a softmax attention over a window beside which the first tokens of the
request stay visible, or a matrix memory with exponential gates (mLSTM); an attention layer may read an earlier
one's keys and values.  Everything that may differ between two models of the design is in config.json::

    architecture        "Fesorax"
    vocab, width        vocabulary and residual width
    norm.eps            epsilon of every RMS norm
    embedding.scale     factor on the looked-up rows
    postln_alpha        alpha in  x <- norm(alpha x + sublayer(x))
    layers[i].type      "attention" or "mlstm"
    layers[i].mixer     attention: heads, kv_heads, dim, vdim, scale, bias_max (where the bias by distance reaches its
                                   last row), mask {size, keep_first} (absent: every earlier token is visible),
                                   kv_from (absent, or the attention layer whose keys and values this one reads)
                        mlstm:     heads, dim, vdim, gate_cap
    layers[i].mlp       null, or {"kind": "moe", "expert": {"ff", "limit"}, "router": {"experts", "top"},
                        "shared": {"ff", "limit"} (absent or null: none)}

The design states no longest sequence: the engine's ``context`` alone bounds a request.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, List, Optional, Tuple

from .common import ConfigError
from .kokolorn import _object
from .lepizen import _int, _number

ARCHITECTURE = "Fesorax"


@dataclass(frozen=True)
class WindowMask:
    size: int                           # a query sees this many most recent positions, its own included
    keep_first: int                     # and the request's first so many

    def to_dict(self) -> Dict[str, Any]:
        return {"size": self.size, "keep_first": self.keep_first}


@dataclass(frozen=True)
class Attention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    bias_max: float
    mask: Optional[WindowMask]
    kv_from: Optional[int] = None

    def to_dict(self) -> Dict[str, Any]:
        out: Dict[str, Any] = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim,
                               "scale": self.scale, "bias_max": self.bias_max}
        if self.mask is not None:
            out["mask"] = self.mask.to_dict()
        if self.kv_from is not None:
            out["kv_from"] = self.kv_from
        return out


@dataclass(frozen=True)
class MatrixMemory:
    heads: int
    dim: int
    vdim: int
    gate_cap: float

    def to_dict(self) -> Dict[str, Any]:
        return {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "gate_cap": self.gate_cap}


@dataclass(frozen=True)
class GatedFF:
    ff: int
    limit: float

    def to_dict(self) -> Dict[str, Any]:
        return {"ff": self.ff, "limit": self.limit}


@dataclass(frozen=True)
class Experts:
    expert: GatedFF
    experts: int
    top: int
    shared: Optional[GatedFF]

    def to_dict(self) -> Dict[str, Any]:
        out: Dict[str, Any] = {"kind": "moe", "expert": self.expert.to_dict(),
                               "router": {"experts": self.experts, "top": self.top}}
        if self.shared is not None:
            out["shared"] = self.shared.to_dict()
        return out


@dataclass(frozen=True)
class FesoraxLayer:
    kind: str                           # "attention" or "mlstm"
    mixer: Any                          # Attention or MatrixMemory
    mlp: Optional[Experts]


def _attention(where: str, m: Dict[str, Any], earlier: List[FesoraxLayer]) -> Attention:
    heads, kv_heads = _int(where, m, "heads"), _int(where, m, "kv_heads")
    if heads % kv_heads:
        raise ConfigError(f"config.json: {where}{heads} heads are not a multiple of {kv_heads} kv_heads")
    mask = None
    if m.get("mask") is not None:
        raw = _object(where, m, "mask")
        keep = 0 if raw.get("keep_first") is None else _int(where + "mask.", raw, "keep_first", minimum=0)
        mask = WindowMask(size=_int(where + "mask.", raw, "size"), keep_first=keep)
    out = Attention(heads=heads, kv_heads=kv_heads, dim=_int(where, m, "dim"), vdim=_int(where, m, "vdim"),
                    scale=_number(where, m, "scale"), bias_max=_number(where, m, "bias_max"), mask=mask)
    source = m.get("kv_from")
    if source is None:
        return out
    if isinstance(source, bool) or not isinstance(source, int) or not 0 <= source < len(earlier):
        raise ConfigError(f"config.json: {where}'kv_from' must name an earlier layer, got {source!r}")
    other = earlier[source].mixer
    if not isinstance(other, Attention) or other.kv_from is not None:
        raise ConfigError(f"config.json: {where}'kv_from' names layer {source}, which has no keys and values of its own")
    if (other.kv_heads, other.dim, other.vdim) != (out.kv_heads, out.dim, out.vdim):
        raise ConfigError(f"config.json: {where}kv_heads, dim and vdim must equal those of layer {source}, whose keys and values it reads")
    return Attention(**{**out.__dict__, "kv_from": source})


def _gated(where: str, raw: Dict[str, Any]) -> GatedFF:
    return GatedFF(ff=_int(where, raw, "ff"), limit=_number(where, raw, "limit"))


def _mlp(where: str, mlp: Any) -> Optional[Experts]:
    if mlp is None:
        return None
    if not isinstance(mlp, dict) or mlp.get("kind") != "moe":
        raise ConfigError(f"config.json: {where}'mlp' must be null or of kind 'moe', got {mlp!r}")
    router = _object(where + "mlp.", mlp, "router")
    experts, top = _int(where + "mlp.router.", router, "experts"), _int(where + "mlp.router.", router, "top")
    if top > experts:
        raise ConfigError(f"config.json: {where}mlp.router takes {top} of {experts} experts")
    if experts > 1024:
        raise ConfigError(f"config.json: {where}mlp.router.experts {experts}: the router takes up to 1024")
    shared = None if mlp.get("shared") is None else _gated(where + "mlp.shared.", _object(where + "mlp.", mlp, "shared"))
    return Experts(expert=_gated(where + "mlp.expert.", _object(where + "mlp.", mlp, "expert")), experts=experts, top=top,
                   shared=shared)


@dataclass(frozen=True)
class FesoraxConfig:
    vocab: int
    width: int
    eps: float
    embedding_scale: float
    alpha: float
    layers: Tuple[FesoraxLayer, ...]

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def hidden_size(self) -> int:
        return self.width

    @staticmethod
    def from_dict(raw: Dict[str, Any]) -> "FesoraxConfig":
        vocab = _int("", raw, "vocab")
        if vocab >= 2 ** 31:
            raise ConfigError(f"config.json: vocab {vocab} does not fit 32-bit token ids")
        width = _int("", raw, "width")
        eps = _number("norm.", _object("", raw, "norm"), "eps")
        scale = 1.0
        if raw.get("embedding") is not None:
            scale = _number("embedding.", _object("", raw, "embedding"), "scale", positive=False)
        listed = raw.get("layers")
        if not isinstance(listed, list) or not listed:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers: List[FesoraxLayer] = []
        for index, entry in enumerate(listed):
            where = f"layers[{index}]."
            if not isinstance(entry, dict):
                raise ConfigError(f"config.json: layers[{index}] must be an object")
            kind = entry.get("type")
            m = _object(where, entry, "mixer")
            if kind == "attention":
                mixer: Any = _attention(where + "mixer.", m, layers)
            elif kind == "mlstm":
                mixer = MatrixMemory(heads=_int(where + "mixer.", m, "heads"), dim=_int(where + "mixer.", m, "dim"),
                                     vdim=_int(where + "mixer.", m, "vdim"), gate_cap=_number(where + "mixer.", m, "gate_cap"))
            else:
                raise ConfigError(f"config.json: {where}'type' must be 'attention' or 'mlstm', got {kind!r}")
            layers.append(FesoraxLayer(kind=kind, mixer=mixer, mlp=_mlp(where, entry.get("mlp"))))
        return FesoraxConfig(vocab=vocab, width=width, eps=eps, embedding_scale=scale,
                             alpha=_number("", raw, "postln_alpha", positive=False), layers=tuple(layers))

    def to_dict(self) -> Dict[str, Any]:
        return {"architecture": ARCHITECTURE, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.eps},
                "embedding": {"scale": self.embedding_scale}, "postln_alpha": self.alpha,
                "layers": [{"type": layer.kind, "mixer": layer.mixer.to_dict(),
                            "mlp": None if layer.mlp is None else layer.mlp.to_dict()} for layer in self.layers]}
