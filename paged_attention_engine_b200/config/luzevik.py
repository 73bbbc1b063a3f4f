"""Typed configuration of the Luzevik decoder, read from its own config.json keys.

    {"architecture": "Luzevik", "vocab": V, "width": W, "embedding": {"scale": s}, "norm": {"eps": e},
     "layers": [{"type": ..., "mixer": {...}, "mlp": {...} | null}, ...]}

A layer's mixer is one of

  latent_attention  heads, dim (unrotated query/key channels per head), rot_dim (rotated ones), vdim,
                    kv_rank and q_rank (the two latents' sizes), scale, rot {base, dims}, kv_from
                    (absent: the layer projects its own latent; j: it reads layer j's).
  parallel          left, right: an attention and a gated delta rule side by side.
                    left: heads, kv_heads, dim (query/key head size), vdim, scale, rot {base, dims,
                    scaling {factor}} (`scaling` absent: plain frequencies).
                    right: heads, kv_heads, dim, vdim, conv (taps).

and its feed-forward {"kind": "dense", "ff"}, or {"kind": "moe", "expert": {"ff"}, "router": {"experts",
"top"}}, or null.

Every size and constant that can differ between two models of the design is read here; nothing
has a default except where a key's absence means that the mechanism is absent.
"""

from __future__ import annotations

import json
from dataclasses import dataclass
from pathlib import Path
from typing import Any, Mapping

from .errors import ConfigError
from .getozen import BiasedAttention, _rotation
from .zugarax import Rotation, _get, _positive

LAYER_TYPES = ("latent_attention", "parallel")


@dataclass(frozen=True)
class SinkLatentAttention:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    q_rank: int
    scale: float
    rot: Rotation
    kv_from: int | None     # the layer whose latent this one reads; None: it has one of its own

    def to_dict(self) -> dict[str, Any]:
        out: dict[str, Any] = {"heads": self.heads, "dim": self.dim, "rot_dim": self.rot_dim, "vdim": self.vdim, "kv_rank": self.kv_rank,
                               "q_rank": self.q_rank, "scale": self.scale, "rot": self.rot.to_dict()}
        if self.kv_from is not None:
            out["kv_from"] = self.kv_from
        return out


@dataclass(frozen=True)
class GatedDeltaHeads:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int

    def to_dict(self) -> dict[str, Any]:
        return {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "conv": self.conv}


@dataclass(frozen=True)
class ParallelMixers:
    left: BiasedAttention
    right: GatedDeltaHeads

    def to_dict(self) -> dict[str, Any]:
        return {"left": self.left.to_dict(), "right": self.right.to_dict()}


@dataclass(frozen=True)
class FeedForward:
    kind: str               # "dense" or "moe"
    ff: int                 # dense: the hidden size; moe: an expert's
    experts: int = 0
    top: int = 0

    def to_dict(self) -> dict[str, Any]:
        if self.kind == "dense":
            return {"kind": "dense", "ff": self.ff}
        return {"kind": "moe", "expert": {"ff": self.ff}, "router": {"experts": self.experts, "top": self.top}}


@dataclass(frozen=True)
class LuzevikLayer:
    type: str
    mixer: Any
    mlp: FeedForward | None

    def to_dict(self) -> dict[str, Any]:
        return {"type": self.type, "mixer": self.mixer.to_dict(), "mlp": self.mlp.to_dict() if self.mlp else None}


def _read_latent(raw, m: str) -> SinkLatentAttention:
    size = lambda key: _positive(_get(raw, key, int, m), m + key)
    rot_dim = size("rot_dim")
    rot = _rotation(raw, m, rot_dim, ("factor",))
    return SinkLatentAttention(size("heads"), size("dim"), rot_dim, size("vdim"), size("kv_rank"), size("q_rank"), _get(raw, "scale", float, m),
                               rot, _get(raw, "kv_from", int, m) if raw.get("kv_from") is not None else None)


def _read_parallel(raw, m: str) -> ParallelMixers:
    for side in ("left", "right"):
        if not isinstance(raw.get(side), Mapping):
            raise ConfigError(f"config.json: key '{m}{side}' is missing")
    size = lambda side, key: _positive(_get(raw[side], key, int, f"{m}{side}."), f"{m}{side}.{key}")
    for side in ("left", "right"):
        if size(side, "heads") % size(side, "kv_heads"):
            raise ConfigError(f"config.json: {m}{side}.heads {size(side, 'heads')} is not a multiple of kv_heads {size(side, 'kv_heads')}")
    dim = size("left", "dim")
    left = BiasedAttention(size("left", "heads"), size("left", "kv_heads"), dim, size("left", "vdim"), _get(raw["left"], "scale", float, m + "left."),
                           _rotation(raw["left"], m + "left.", dim, ("factor",)))
    right = GatedDeltaHeads(*(size("right", key) for key in ("heads", "kv_heads", "dim", "vdim", "conv")))
    return ParallelMixers(left, right)


def _read_mlp(raw, w: str) -> FeedForward:
    kind = _get(raw, "kind", str, w)
    if kind == "dense":
        return FeedForward("dense", _positive(_get(raw, "ff", int, w), w + "ff"))
    if kind != "moe":
        raise ConfigError(f"config.json: {w}kind '{kind}' is not one of dense, moe")
    experts = _positive(_get(raw.get("router"), "experts", int, w + "router."), w + "router.experts")
    top = _positive(_get(raw["router"], "top", int, w + "router."), w + "router.top")
    if top > experts:
        raise ConfigError(f"config.json: {w}router.top {top} exceeds the {experts} experts")
    return FeedForward("moe", _positive(_get(raw.get("expert"), "ff", int, w + "expert."), w + "expert.ff"), experts, top)


@dataclass(frozen=True)
class LuzevikConfig:
    vocab: int
    width: int
    embedding_scale: float
    norm_eps: float
    layers: tuple[LuzevikLayer, ...]
    architecture: str = "Luzevik"

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "LuzevikConfig":
        layers_raw = raw.get("layers")
        if not isinstance(layers_raw, (list, tuple)) or not layers_raw:
            raise ConfigError("config.json: key 'layers' is missing or empty")
        layers: list[LuzevikLayer] = []
        for i, entry in enumerate(layers_raw):
            where = f"layers[{i}]."
            kind = _get(entry, "type", str, where)
            if kind not in LAYER_TYPES:
                raise ConfigError(f"config.json: {where}type '{kind}' is not one of {', '.join(LAYER_TYPES)}")
            if not isinstance(entry.get("mixer"), Mapping):
                raise ConfigError(f"config.json: key '{where}mixer' is missing")
            mixer = (_read_parallel if kind == "parallel" else _read_latent)(entry["mixer"], where + "mixer.")
            mlp = _read_mlp(entry["mlp"], where + "mlp.") if entry.get("mlp") is not None else None
            layers.append(LuzevikLayer(kind, mixer, mlp))
        for i, layer in enumerate(layers):
            j = getattr(layer.mixer, "kv_from", None)
            if j is None:
                continue
            if not 0 <= j < i or layers[j].type != "latent_attention" or layers[j].mixer.kv_from is not None:
                raise ConfigError(f"config.json: layers[{i}].mixer.kv_from {j} does not name an earlier latent attention with a latent of its own")
            mine, theirs = layer.mixer, layers[j].mixer
            if (mine.kv_rank, mine.rot_dim, mine.rot) != (theirs.kv_rank, theirs.rot_dim, theirs.rot):
                raise ConfigError(f"config.json: layers[{i}] reads layer {j}'s latent and differs from it in kv_rank, rot_dim or rot")
        return cls(
            vocab=_positive(_get(raw, "vocab", int, ""), "vocab"),
            width=_positive(_get(raw, "width", int, ""), "width"),
            embedding_scale=_get(raw.get("embedding"), "scale", float, "embedding."),
            norm_eps=_positive(_get(raw.get("norm"), "eps", float, "norm."), "norm.eps"),
            layers=tuple(layers),
            architecture=str(raw.get("architecture", "Luzevik")),
        )

    @classmethod
    def from_json(cls, path: str | Path) -> "LuzevikConfig":
        return cls.from_dict(json.loads(Path(path).read_text()))

    def to_dict(self) -> dict[str, Any]:
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "embedding": {"scale": self.embedding_scale},
                "norm": {"eps": self.norm_eps}, "layers": [layer.to_dict() for layer in self.layers]}
