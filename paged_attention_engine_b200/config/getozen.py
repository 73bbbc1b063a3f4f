"""Typed configuration of the Getozen decoder, read from its own config.json keys.

    {"architecture": "Getozen", "vocab": V, "width": W, "norm": {"eps": e},
     "layers": [{"type": ..., "mixer": {...}, "mlp": {"kind": "dense", "ff": F} | null, "weights_of": j}, ...]}

A layer's mixer is one of

  parallel            left, right, left_scale, right_scale: an attention and a retention side by side.
                      left: heads, kv_heads, dim (query/key head size), vdim, scale, rot {base, dims,
                      scaling {factor}} (`scaling` absent: plain frequencies).
                      right: heads, dim, vdim, decay (a number per head), rot {base, dims}.
  mamba2, mamba2_2    heads, vdim, state, groups, conv (taps), norm_groups. The two names stand for the
                      same mixer in two sets of sizes.

`weights_of` (absent: the layer has tensors of its own) names the layer whose tensors this one runs
with; the rest of the entry repeats that layer's.

Every size and constant that can differ between two models of the design is read here; nothing
has a default except where a key's absence means that the mechanism is absent.
"""

from __future__ import annotations

import json
from dataclasses import dataclass, replace
from pathlib import Path
from typing import Any, Mapping

from .errors import ConfigError
from .zugarax import Rotation, _get, _positive

LAYER_TYPES = ("parallel", "mamba2", "mamba2_2")


@dataclass(frozen=True)
class BiasedAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Rotation

    def to_dict(self) -> dict[str, Any]:
        return {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale,
                "rot": self.rot.to_dict()}


@dataclass(frozen=True)
class RetentionHeads:
    heads: int
    dim: int
    vdim: int
    decay: tuple[float, ...]
    rot: Rotation

    def to_dict(self) -> dict[str, Any]:
        return {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "decay": list(self.decay), "rot": self.rot.to_dict()}


@dataclass(frozen=True)
class ParallelMixers:
    left: BiasedAttention
    right: RetentionHeads
    left_scale: float
    right_scale: float

    def to_dict(self) -> dict[str, Any]:
        return {"left": self.left.to_dict(), "right": self.right.to_dict(), "left_scale": self.left_scale, "right_scale": self.right_scale}


@dataclass(frozen=True)
class SelectiveStateSpace:
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int

    def to_dict(self) -> dict[str, Any]:
        return {"heads": self.heads, "vdim": self.vdim, "state": self.state, "groups": self.groups, "conv": self.conv,
                "norm_groups": self.norm_groups}


@dataclass(frozen=True)
class GetozenLayer:
    type: str
    mixer: Any
    ff: int                     # 0: the layer has no feed-forward
    weights_of: int | None      # the layer whose tensors this one runs with

    def to_dict(self) -> dict[str, Any]:
        out = {"type": self.type, "mixer": self.mixer.to_dict(), "mlp": {"kind": "dense", "ff": self.ff} if self.ff else None}
        if self.weights_of is not None:
            out["weights_of"] = self.weights_of
        return out


def _rotation(raw, where: str, dim: int, scaling_keys: tuple[str, ...]) -> Rotation:
    rot = Rotation.read(raw.get("rot"), where + "rot.", scaling_keys)
    if rot.dims > dim:
        raise ConfigError(f"config.json: {where}rot.dims {rot.dims} exceeds dim {dim}")
    return rot


def _read_parallel(raw, m: str) -> ParallelMixers:
    for side in ("left", "right"):
        if not isinstance(raw.get(side), Mapping):
            raise ConfigError(f"config.json: key '{m}{side}' is missing")
    size = lambda side, key: _positive(_get(raw[side], key, int, f"{m}{side}."), f"{m}{side}.{key}")
    heads, kv_heads = size("left", "heads"), size("left", "kv_heads")
    if heads % kv_heads:
        raise ConfigError(f"config.json: {m}left.heads {heads} is not a multiple of kv_heads {kv_heads}")
    dim = size("left", "dim")
    left = BiasedAttention(heads, kv_heads, dim, size("left", "vdim"), _get(raw["left"], "scale", float, m + "left."),
                           _rotation(raw["left"], m + "left.", dim, ("factor",)))
    decay = raw["right"].get("decay")
    if not isinstance(decay, (list, tuple)) or len(decay) != size("right", "heads"):
        raise ConfigError(f"config.json: {m}right.decay is not a number for each of the heads")
    decay = tuple(float(x) for x in decay)
    if min(decay) < 0.0:
        raise ConfigError(f"config.json: {m}right.decay has a negative number")
    dim = size("right", "dim")
    right = RetentionHeads(size("right", "heads"), dim, size("right", "vdim"), decay, _rotation(raw["right"], m + "right.", dim, ("factor",)))
    return ParallelMixers(left, right, _get(raw, "left_scale", float, m), _get(raw, "right_scale", float, m))


def _read_state_space(raw, m: str) -> SelectiveStateSpace:
    size = lambda key: _positive(_get(raw, key, int, m), m + key)
    out = SelectiveStateSpace(size("heads"), size("vdim"), size("state"), size("groups"), size("conv"), size("norm_groups"))
    if out.heads % out.groups:
        raise ConfigError(f"config.json: {m}heads {out.heads} is not a multiple of groups {out.groups}")
    if out.heads * out.vdim % out.norm_groups:
        raise ConfigError(f"config.json: {m}norm_groups {out.norm_groups} does not divide the {out.heads * out.vdim} inner channels")
    return out


@dataclass(frozen=True)
class GetozenConfig:
    vocab: int
    width: int
    norm_eps: float
    layers: tuple[GetozenLayer, ...]
    architecture: str = "Getozen"

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "GetozenConfig":
        layers_raw = raw.get("layers")
        if not isinstance(layers_raw, (list, tuple)) or not layers_raw:
            raise ConfigError("config.json: key 'layers' is missing or empty")
        layers: list[GetozenLayer] = []
        for i, entry in enumerate(layers_raw):
            where = f"layers[{i}]."
            kind = _get(entry, "type", str, where)
            if kind not in LAYER_TYPES:
                raise ConfigError(f"config.json: {where}type '{kind}' is not one of {', '.join(LAYER_TYPES)}")
            if not isinstance(entry.get("mixer"), Mapping):
                raise ConfigError(f"config.json: key '{where}mixer' is missing")
            mixer = (_read_parallel if kind == "parallel" else _read_state_space)(entry["mixer"], where + "mixer.")
            ff = 0
            if entry.get("mlp") is not None:
                mlp_kind = _get(entry["mlp"], "kind", str, where + "mlp.")
                if mlp_kind != "dense":
                    raise ConfigError(f"config.json: {where}mlp.kind '{mlp_kind}' is not supported (dense)")
                ff = _positive(_get(entry["mlp"], "ff", int, where + "mlp."), where + "mlp.ff")
            shared = entry.get("weights_of")
            layers.append(GetozenLayer(kind, mixer, ff, None if shared is None else int(shared)))
        for i, layer in enumerate(layers):
            j = layer.weights_of
            if j is None:
                continue
            if not 0 <= j < len(layers) or j == i or layers[j].weights_of is not None:
                raise ConfigError(f"config.json: layers[{i}].weights_of {j} does not name another layer with tensors of its own")
            if replace(layer, weights_of=None) != layers[j]:
                raise ConfigError(f"config.json: layers[{i}] differs from layer {j}, whose weights it uses")
        return cls(
            vocab=_positive(_get(raw, "vocab", int, ""), "vocab"),
            width=_positive(_get(raw, "width", int, ""), "width"),
            norm_eps=_positive(_get(raw.get("norm"), "eps", float, "norm."), "norm.eps"),
            layers=tuple(layers),
            architecture=str(raw.get("architecture", "Getozen")),
        )

    @classmethod
    def from_json(cls, path: str | Path) -> "GetozenConfig":
        return cls.from_dict(json.loads(Path(path).read_text()))

    def to_dict(self) -> dict[str, Any]:
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
                "layers": [layer.to_dict() for layer in self.layers]}
