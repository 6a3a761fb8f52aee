"""Typed configuration of the Sumuvik design, read from its own config.json keys.

A Sumuvik model is a list of layers, each with one of two mixers and a dense or mixture-of-experts feed-forward (or none)
that reads the same stream as the mixer:

    {"architecture": "Sumuvik", "vocab": V, "width": D, "norm": {"eps": e}, "embedding": {"scale": s},
     "layers": [{"type": "attention" | "rglru", "mixer": {...}, "mlp": {...} | null}, ...]}

    attention mixer:  heads, kv_heads, dim, vdim, scale, mask.size (optional: a sliding window), mask.keep_first (optional:
                      first tokens seen beside the window), rot.base, rot.dims (optional: no rotation without them),
                      rot.scaling {factor, low, high, original} (optional)
    rglru mixer:      width, blocks, conv
    mlp:              kind "dense": ff, limit
                      kind "moe":   expert {ff, limit}, router {experts, top, scale (optional), groups {count, keep}
                                    (optional)}, shared {ff, limit} (optional)

Every size and constant that may differ between models comes from here; what the design fixes lives with the parts
(``models/sumuvik.py`` passes it as parameters).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Mapping, Optional, Tuple

from .errors import ConfigError
from .rusadra import _get

MIXERS = ("attention", "rglru")


@dataclass(frozen=True)
class WavelengthScaling:
    factor: float
    low: float
    high: float
    original: float

    def to_dict(self) -> Dict[str, Any]:
        return {"factor": self.factor, "low": self.low, "high": self.high, "original": self.original}


@dataclass(frozen=True)
class WindowMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int          # mask.size: a token sees itself and the window - 1 before it; 0 (no mask key): all before it
    keep_first: int      # mask.keep_first: tokens of the sequence's start that stay visible
    rot_base: float
    rot_dims: int        # 0: no rotation
    scaling: Optional[WavelengthScaling] = None

    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim,
                             "scale": self.scale}
        if self.window:
            d["mask"] = {"size": self.window, "keep_first": self.keep_first}
        if self.rot_dims:
            d["rot"] = {"base": self.rot_base, "dims": self.rot_dims}
            if self.scaling is not None:
                d["rot"]["scaling"] = self.scaling.to_dict()
        return d


@dataclass(frozen=True)
class RecurrentMixer:
    width: int
    blocks: int
    conv: int

    def to_dict(self) -> Dict[str, Any]:
        return {"width": self.width, "blocks": self.blocks, "conv": self.conv}


@dataclass(frozen=True)
class Unit:
    """A clamped gated unit: its size and the limit of gate and up."""
    ff: int
    limit: float

    def to_dict(self) -> Dict[str, Any]:
        return {"ff": self.ff, "limit": self.limit}


@dataclass(frozen=True)
class DenseMLP:
    unit: Unit

    def to_dict(self) -> Dict[str, Any]:
        return {"kind": "dense", **self.unit.to_dict()}


@dataclass(frozen=True)
class MoEMLP:
    expert: Unit
    experts: int
    top: int
    scale: float
    groups: int = 1
    keep: int = 1
    shared: Optional[Unit] = None

    def to_dict(self) -> Dict[str, Any]:
        router: Dict[str, Any] = {"experts": self.experts, "top": self.top, "scale": self.scale}
        if (self.groups, self.keep) != (1, 1):
            router["groups"] = {"count": self.groups, "keep": self.keep}
        d: Dict[str, Any] = {"kind": "moe", "expert": self.expert.to_dict(), "router": router}
        if self.shared is not None:
            d["shared"] = self.shared.to_dict()
        return d


@dataclass(frozen=True)
class SumuvikLayer:
    type: str
    mixer: Any           # WindowMixer or RecurrentMixer
    mlp: Any             # DenseMLP, MoEMLP or None


def _object(raw: Mapping, key: str, where: str) -> Optional[Mapping]:
    """An optional object: None where the key is absent or null."""
    node = raw.get(key)
    if node is not None and not isinstance(node, Mapping):
        raise ConfigError(f"{where}: {key} must be an object, got {node!r}")
    return node


def _unit(raw: Mapping, where: str) -> Unit:
    unit = Unit(_get(raw, "ff", int, where, 1), _get(raw, "limit", float, where))
    if not unit.limit > 0:
        raise ConfigError(f"{where}: limit must be positive, got {unit.limit}")
    return unit


def _window_mixer(m: Mapping, where: str) -> WindowMixer:
    heads, dim = _get(m, "heads", int, where, 1), _get(m, "dim", int, where, 1)
    kv_heads = _get(m, "kv_heads", int, where, 1, optional=True) or heads
    if heads % kv_heads:
        raise ConfigError(f"{where}: {heads} heads are no multiple of {kv_heads} kv_heads")
    window = keep = 0
    mask = _object(m, "mask", where)
    if mask is not None:
        window = _get(mask, "size", int, where + ".mask", 1)
        keep = _get(mask, "keep_first", int, where + ".mask", 0, optional=True) or 0
    rot_dims, base, scaling = 0, 1.0, None
    rot = _object(m, "rot", where)
    if rot is not None:
        rw = where + ".rot"
        rot_dims = _get(rot, "dims", int, rw, 0)
        if rot_dims % 2 or rot_dims > dim:
            raise ConfigError(f"{where}: rot.dims {rot_dims} must be even and at most dim {dim}")
        base = _get(rot, "base", float, rw) if rot_dims else 1.0
        if base <= 0:
            raise ConfigError(f"{where}: rot.base must be positive, got {base}")
        sc = _object(rot, "scaling", rw)
        if sc is not None:
            sw = rw + ".scaling"
            scaling = WavelengthScaling(*(_get(sc, k, float, sw) for k in ("factor", "low", "high", "original")))
            if min(scaling.factor, scaling.low, scaling.high, scaling.original) <= 0 or scaling.high < scaling.low:
                raise ConfigError(f"{sw}: factor, low, high and original must be positive, and high at least low")
    return WindowMixer(heads=heads, kv_heads=kv_heads, dim=dim, vdim=_get(m, "vdim", int, where, 1, optional=True) or dim,
                       scale=_get(m, "scale", float, where), window=window, keep_first=keep, rot_base=base,
                       rot_dims=rot_dims, scaling=scaling if rot_dims else None)


def _recurrent_mixer(m: Mapping, where: str) -> RecurrentMixer:
    mixer = RecurrentMixer(_get(m, "width", int, where, 1), _get(m, "blocks", int, where, 1), _get(m, "conv", int, where, 1))
    if mixer.width % mixer.blocks:
        raise ConfigError(f"{where}: width {mixer.width} is no multiple of {mixer.blocks} blocks")
    return mixer


def _mlp(f: Any, where: str):
    if f is None:
        return None
    if not isinstance(f, Mapping) or f.get("kind") not in ("dense", "moe"):
        raise ConfigError(f"{where}: mlp.kind must be 'dense' or 'moe' (or mlp null)")
    if f["kind"] == "dense":
        return DenseMLP(_unit(f, where + ".mlp"))
    expert, shared = _object(f, "expert", where), _object(f, "shared", where)
    if expert is None:
        raise ConfigError(f"{where}: mlp.expert missing from config")
    router = _object(f, "router", where) or {}
    rw = where + ".mlp.router"
    count = keep = 1
    groups = _object(router, "groups", rw)
    if groups is not None:
        count, keep = _get(groups, "count", int, rw + ".groups", 1), _get(groups, "keep", int, rw + ".groups", 1)
    scale = _get(router, "scale", float, rw, optional=True)
    mlp = MoEMLP(expert=_unit(expert, where + ".mlp.expert"), experts=_get(router, "experts", int, rw, 1),
                 top=_get(router, "top", int, rw, 1), scale=1.0 if scale is None else scale, groups=count, keep=keep,
                 shared=None if shared is None else _unit(shared, where + ".mlp.shared"))
    if mlp.experts % count or keep > count:
        raise ConfigError(f"{rw}: {mlp.experts} experts in {count} groups of which {keep} are kept")
    if mlp.top > keep * (mlp.experts // count):
        raise ConfigError(f"{rw}: top {mlp.top} exceeds the {keep * (mlp.experts // count)} experts that can be chosen")
    return mlp


@dataclass(frozen=True)
class SumuvikConfig:
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    layers: Tuple[SumuvikLayer, ...]
    torch_dtype: str = "bfloat16"

    architecture = "Sumuvik"
    model_type = "sumuvik"

    @classmethod
    def from_dict(cls, raw: Dict[str, Any]) -> "SumuvikConfig":
        layers_raw = raw.get("layers")
        if not isinstance(layers_raw, list) or not layers_raw:
            raise ConfigError("config: layers must be a non-empty list")
        layers = []
        for i, lr in enumerate(layers_raw):
            where = f"layers[{i}]"
            if not isinstance(lr, Mapping) or lr.get("type") not in MIXERS:
                raise ConfigError(f"{where}: type must be one of {MIXERS}, got "
                                  f"{lr.get('type') if isinstance(lr, Mapping) else lr!r}")
            m = _object(lr, "mixer", where)
            if m is None:
                raise ConfigError(f"{where}: mixer missing from config")
            mixer = _window_mixer(m, where) if lr["type"] == "attention" else _recurrent_mixer(m, where)
            layers.append(SumuvikLayer(lr["type"], mixer, _mlp(lr.get("mlp"), where)))
        scale = _get(raw, "embedding.scale", float, "config", optional=True)
        return cls(vocab=_get(raw, "vocab", int, "config", 1), width=_get(raw, "width", int, "config", 1),
                   norm_eps=_get(raw, "norm.eps", float, "config", 0.0), embedding_scale=1.0 if scale is None else scale,
                   layers=tuple(layers), torch_dtype=str(raw.get("torch_dtype", "bfloat16")))

    def to_dict(self) -> Dict[str, Any]:
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
                "norm": {"eps": self.norm_eps}, "embedding": {"scale": self.embedding_scale},
                "layers": [{"type": l.type, "mixer": l.mixer.to_dict(),
                            "mlp": None if l.mlp is None else l.mlp.to_dict()} for l in self.layers]}
