"""Typed configuration of the Kopatar design, read from its own config.json keys.

A Kopatar model is a list of pre-norm layers, each with one of three mixers and a dense feed-forward (or none), with tied
embedding and head; a stretch of the layers may run several times:

    {"architecture": "Kopatar", "vocab": V, "width": D, "norm": {"eps": e},
     "loop": {"start": a, "stop": b, "times": n} (optional),
     "layers": [{"type": "channel_delta" | "retention" | "parallel", "mixer": {...},
                 "mlp": {"kind": "dense", "ff": F} | null}, ...]}

    channel_delta mixer  heads, kv_heads, dim, vdim, conv (taps)
    retention mixer      heads, dim, vdim, decay (one number per head), rot.base, rot.dims
    parallel mixer       left: heads, kv_heads, dim, vdim, scale, mask.size (a sliding window);
                         right: heads, vdim, state, groups, conv (taps), norm_groups; left_scale, right_scale

The ranks of a channel_delta mixer's two low-rank projections are rows of their tensors: they are read from the folder
when it is at hand; without it (a configuration made in memory) the keys ``decay_rank`` and ``gate_rank`` say them.
Constants the design fixes live with the parts (``models/kopatar.py`` passes them as parameters).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Mapping, Optional, Tuple

from .errors import ConfigError
from .fekolorn import DenseMLP
from .pozelix import Loop
from .rusadra import _get

MIXERS = ("channel_delta", "retention", "parallel")


@dataclass(frozen=True)
class ChannelDeltaMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    decay_rank: int
    gate_rank: int

    def to_dict(self) -> Dict[str, Any]:
        return {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "conv": self.conv,
                "decay_rank": self.decay_rank, "gate_rank": self.gate_rank}


@dataclass(frozen=True)
class RetentionMixer:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]
    rot_base: float
    rot_dims: int

    def to_dict(self) -> Dict[str, Any]:
        d = {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "decay": list(self.decay)}
        if self.rot_dims:
            d["rot"] = {"base": self.rot_base, "dims": self.rot_dims}
        return d


@dataclass(frozen=True)
class WindowMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int = 0      # mask.size: a token sees itself and the window - 1 before it; 0 (no mask key): all before it

    def to_dict(self) -> Dict[str, Any]:
        d = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale}
        if self.window:
            d["mask"] = {"size": self.window}
        return d


@dataclass(frozen=True)
class StateSpaceMixer:
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int

    def to_dict(self) -> Dict[str, Any]:
        return {"heads": self.heads, "vdim": self.vdim, "state": self.state, "groups": self.groups, "conv": self.conv,
                "norm_groups": self.norm_groups}


@dataclass(frozen=True)
class ParallelMixer:
    left: WindowMixer
    right: StateSpaceMixer
    left_scale: float
    right_scale: float

    def to_dict(self) -> Dict[str, Any]:
        return {"left": self.left.to_dict(), "right": self.right.to_dict(), "left_scale": self.left_scale,
                "right_scale": self.right_scale}


@dataclass(frozen=True)
class KopatarLayer:
    type: str
    mixer: Any
    mlp: Optional[DenseMLP]


def _kv_heads(m: Mapping, heads: int, where: str) -> int:
    kv_heads = _get(m, "kv_heads", int, where, 1, optional=True) or heads
    if heads % kv_heads:
        raise ConfigError(f"{where}: {heads} heads are no multiple of {kv_heads} kv_heads")
    return kv_heads


def _channel_delta(m: Mapping, where: str, prefix: str, shapes) -> ChannelDeltaMixer:
    heads, dim = _get(m, "heads", int, where, 1), _get(m, "dim", int, where, 1)

    def rank(key: str, tensor: str) -> int:
        if shapes is not None and len(shapes.get(prefix + tensor, ())) == 2:
            return int(shapes[prefix + tensor][0])
        return _get(m, key, int, where, 1)
    return ChannelDeltaMixer(
        heads=heads, kv_heads=_kv_heads(m, heads, where), dim=dim,
        vdim=_get(m, "vdim", int, where, 1, optional=True) or dim, conv=_get(m, "conv", int, where, 1),
        decay_rank=rank("decay_rank", "a1"), gate_rank=rank("gate_rank", "g1"))


def _retention(m: Mapping, where: str) -> RetentionMixer:
    heads, dim = _get(m, "heads", int, where, 1), _get(m, "dim", int, where, 1)
    decay = m.get("decay")
    if not isinstance(decay, list) or len(decay) != heads or \
            not all(isinstance(d, (int, float)) and not isinstance(d, bool) and 0 <= d <= 1 for d in decay):
        raise ConfigError(f"{where}: decay must list one number from 0 to 1 per head ({heads}), got {decay!r}")
    rot_dims = _get(m, "rot.dims", int, where, 0, optional=True) or 0
    if rot_dims % 2 or rot_dims > dim:
        raise ConfigError(f"{where}: rot.dims {rot_dims} must be even and at most dim {dim}")
    return RetentionMixer(heads=heads, dim=dim, vdim=_get(m, "vdim", int, where, 1, optional=True) or dim,
                          decay=tuple(float(d) for d in decay),
                          rot_base=_get(m, "rot.base", float, where) if rot_dims else 1.0, rot_dims=rot_dims)


def _parallel(m: Mapping, where: str) -> ParallelMixer:
    left, right = m.get("left"), m.get("right")
    if not isinstance(left, Mapping) or not isinstance(right, Mapping):
        raise ConfigError(f"{where}: a parallel mixer needs left and right")
    lw, rw = where + ".left", where + ".right"
    heads, dim = _get(left, "heads", int, lw, 1), _get(left, "dim", int, lw, 1)
    window = WindowMixer(
        heads=heads, kv_heads=_kv_heads(left, heads, lw), dim=dim,
        vdim=_get(left, "vdim", int, lw, 1, optional=True) or dim, scale=_get(left, "scale", float, lw),
        window=_get(left, "mask.size", int, lw, 1, optional=True) or 0)
    r_heads, vdim = _get(right, "heads", int, rw, 1), _get(right, "vdim", int, rw, 1)
    groups = _get(right, "groups", int, rw, 1, optional=True) or 1
    norm_groups = _get(right, "norm_groups", int, rw, 1, optional=True) or 1
    if r_heads % groups:
        raise ConfigError(f"{rw}: {r_heads} heads are no multiple of {groups} groups")
    if (r_heads * vdim) % norm_groups:
        raise ConfigError(f"{rw}: {r_heads * vdim} channels do not fall into {norm_groups} equal norm_groups")
    space = StateSpaceMixer(heads=r_heads, vdim=vdim, state=_get(right, "state", int, rw, 1), groups=groups,
                            conv=_get(right, "conv", int, rw, 1), norm_groups=norm_groups)
    scale = lambda key: _get(m, key, float, where) if key in m else 1.0
    return ParallelMixer(left=window, right=space, left_scale=scale("left_scale"), right_scale=scale("right_scale"))


@dataclass(frozen=True)
class KopatarConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: Tuple[KopatarLayer, ...]
    loop: Optional[Loop] = None
    torch_dtype: str = "bfloat16"

    architecture = "Kopatar"
    model_type = "kopatar"
    wants_tensor_shapes = True      # ``load_config`` passes the folder's tensor shapes to ``from_dict``

    @classmethod
    def from_dict(cls, raw: Dict[str, Any], tensor_shapes: Optional[Mapping[str, Tuple[int, ...]]] = None):
        vocab = _get(raw, "vocab", int, "config", 1)
        width = _get(raw, "width", int, "config", 1)
        eps = _get(raw, "norm.eps", float, "config", 0.0)
        layers_raw = raw.get("layers")
        if not isinstance(layers_raw, list) or not layers_raw:
            raise ConfigError("config: layers must be a non-empty list")
        layers = []
        for i, lr in enumerate(layers_raw):
            where = f"layers[{i}]"
            if not isinstance(lr, Mapping) or lr.get("type") not in MIXERS:
                raise ConfigError(f"{where}: type must be one of {MIXERS}, got "
                                  f"{lr.get('type') if isinstance(lr, Mapping) else lr!r}")
            m = lr.get("mixer")
            if not isinstance(m, Mapping):
                raise ConfigError(f"{where}: mixer missing from config")
            if lr["type"] == "channel_delta":
                mixer: Any = _channel_delta(m, where, f"l{i}.mix.", tensor_shapes)
            elif lr["type"] == "retention":
                mixer = _retention(m, where)
            else:
                mixer = _parallel(m, where)
            mlp_raw, mlp = lr.get("mlp"), None
            if mlp_raw is not None:
                if not isinstance(mlp_raw, Mapping) or mlp_raw.get("kind") != "dense":
                    raise ConfigError(f"{where}: mlp.kind must be 'dense' (or mlp null)")
                mlp = DenseMLP(_get(mlp_raw, "ff", int, where, 1))
            layers.append(KopatarLayer(lr["type"], mixer, mlp))
        loop = None
        if raw.get("loop") is not None:
            loop = Loop(_get(raw, "loop.start", int, "config", 0), _get(raw, "loop.stop", int, "config", 1),
                        _get(raw, "loop.times", int, "config", 1))
            if not loop.start < loop.stop <= len(layers):
                raise ConfigError(f"config: loop from {loop.start} to {loop.stop} over {len(layers)} layers")
        return cls(vocab=vocab, width=width, norm_eps=eps, layers=tuple(layers), loop=loop,
                   torch_dtype=str(raw.get("torch_dtype", "bfloat16")))

    def to_dict(self) -> Dict[str, Any]:
        d = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
             "layers": [{"type": l.type, "mixer": l.mixer.to_dict(), "mlp": None if l.mlp is None else l.mlp.to_dict()}
                        for l in self.layers]}
        if self.loop is not None:
            d["loop"] = self.loop.to_dict()
        return d
