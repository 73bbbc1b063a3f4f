"""Small Getozen configurations and the glue between model folders and the plain implementation."""

from __future__ import annotations

import json
from pathlib import Path

import torch

from plain import getozen_plain as plain


def rot(dims, base, factor=None):
    out = {"base": base, "dims": dims}
    if factor:
        out["scaling"] = {"factor": factor}
    return out


def parallel(left, right, scales=(1.0, 1.0), ff=None):
    """left: (heads, kv_heads, dim, vdim, scale, rot); right: (dim, vdim, decays, rot)."""
    heads, kv_heads, dim, vdim, scale, left_rot = left
    rdim, rvdim, decay, right_rot = right
    return {"type": "parallel", "mixer": {
        "left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": left_rot},
        "right": {"heads": len(decay), "dim": rdim, "vdim": rvdim, "decay": list(decay), "rot": right_rot},
        "left_scale": scales[0], "right_scale": scales[1]}, "mlp": mlp(ff)}


def mamba(heads, vdim, state, groups, conv, norm_groups, ff=None, kind="mamba2"):
    return {"type": kind, "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups},
            "mlp": mlp(ff)}


def mlp(ff):
    return {"kind": "dense", "ff": ff} if ff else None


def again(layers, i):
    """Layer i once more, with its weights."""
    return dict(layers[i], weights_of=i)


def config(vocab, width, layers, eps=1e-5):
    return {"architecture": "Getozen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


# Odd sizes: value heads larger and smaller than key heads, partly rotated heads on both sides, a state of
# 7, three groups, three and five taps, norm groups that cut through heads, a layer without a
# feed-forward, two layers that run again, one of them before its neighbour has.
_a = [
    parallel((4, 2, 12, 20, 0.3, rot(8, 40.0, 3.0)), (10, 6, (0.5, 0.97, 1.0), rot(6, 30.0)), (1.3, 0.8), 40),
    mamba(6, 10, 7, 3, 3, 4, 24),
    mamba(4, 16, 20, 1, 5, 1, None, "mamba2_2"),
]
SMALL_A = config(211, 64, _a + [again(_a, 1), again(_a, 0), parallel((3, 3, 16, 8, 0.25, rot(16, 900.0)), (8, 24, (0.9, 0.0), rot(8, 100.0, 2.0)))])
# Sizes that the tensor-core kernels take: attention by the plain kernels (one head size), by the
# scored ones (two), retention and state space in chunks.
_b = [
    mamba(4, 64, 32, 2, 4, 2, 256, "mamba2_2"),
    parallel((4, 2, 64, 64, 0.125, rot(64, 10000.0, 4.0)), (64, 128, (0.96875, 0.998), rot(64, 10000.0)), (0.9, 1.1), 192),
    mamba(6, 24, 16, 3, 2, 6, 128),
    parallel((2, 1, 32, 128, 0.17, rot(16, 5000.0, 2.0)), (32, 16, (0.99, 0.75, 0.9999), rot(32, 1000.0)), (1.2, 0.6), 128),
]
SMALL_B = config(257, 128, _b + [again(_b, 0), again(_b, 1)], eps=1e-6)
# One of everything, no convolution state (a single tap), a width that is no multiple of 8.
ONES = config(97, 52, [
    parallel((1, 1, 8, 24, 0.4, rot(2, 100.0, 1.5)), (6, 10, (0.8,), rot(4, 50.0)), (1.0, 1.0), 20),
    mamba(1, 12, 8, 1, 1, 1, 28),
    mamba(1, 8, 1, 1, 2, 2),
])
# Keys and states wider than 128 channels, value heads wider than a block's columns, the longest convolution.
WIDE = config(97, 64, [
    mamba(2, 80, 144, 1, 17, 5, 48),
    parallel((2, 2, 128, 128, 0.09, rot(96, 10000.0, 8.0)), (136, 72, (0.95, 0.995), rot(136, 10000.0)), (0.7, 1.4), 64),
])
SMALL = {"small_a": (SMALL_A, 4, 51), "small_b": (SMALL_B, 16, 52), "ones": (ONES, 8, 53), "wide": (WIDE, 16, 54)}   # config, page size, seed


def write_model(folder: Path, raw: dict, seed: int, dtype=torch.bfloat16, sharpen: float = 4.0) -> Path:
    """A random model folder whose numbers make faults visible: projections scaled up (one key's score
    stands out, a state's terms differ in size), biases, gates, taps, steps, rates and slopes of a size that
    matters. Steps and rates are spread so that some heads forget within a few tokens and others hold
    what they saw hundreds of tokens ago."""
    from safetensors.torch import load_file, save_file

    from paged_attention_engine_b200.weights import write_random_model

    write_random_model(folder, raw, seed, dtype)
    path = str(Path(folder) / "model.safetensors")
    tensors = load_file(path)
    gen = torch.Generator().manual_seed(seed + 1000)
    for name in list(tensors):
        t = tensors[name].float()
        if name.endswith((".left.q", ".left.k", ".left.v", ".right.q", ".right.k", ".right.v", ".mix.in", ".up", ".gate", ".o", ".down")):
            t = t * sharpen
        elif name.endswith((".left.g", ".right.g")):
            t = t * 15.0
        elif name.endswith((".q.b", ".k.b", ".v.b", ".conv.b", "norm1.b", "norm2.b", "final.norm.b")):
            t = torch.randn(t.shape, generator=gen) * 0.3
        elif name.endswith(".dt_bias"):
            t = torch.rand(t.shape, generator=gen) * 4.0 - 4.0
        elif name.endswith(".A_log"):
            t = torch.rand(t.shape, generator=gen) * 4.0 - 3.0
        elif name.endswith(".D"):
            t = torch.randn(t.shape, generator=gen)
        elif name.endswith(".alpha"):
            t = 0.3 + torch.rand(t.shape, generator=gen) * 0.9
        elif name.endswith(("norm1", "norm2", "final.norm", ".mix.norm")):
            t = (0.5 + torch.rand(t.shape, generator=gen)) * (torch.randint(0, 2, t.shape, generator=gen) * 2.0 - 1.0)
        elif name == "embed":
            t = t * 40.0
        elif name == "head":
            t = t * 12.0
        tensors[name] = t.to(tensors[name].dtype)
    save_file(tensors, path)
    return Path(folder)


def read_model(folder: Path):
    from safetensors.torch import load_file

    return json.loads((Path(folder) / "config.json").read_text()), load_file(str(Path(folder) / "model.safetensors"))


def plain_logits(folder: Path, tokens) -> torch.Tensor:
    raw, tensors = read_model(folder)
    return plain.forward(raw, tensors, tokens).float()


def random_requests(raw: dict, lengths, seed: int) -> dict[str, list[int]]:
    gen = torch.Generator().manual_seed(seed)
    return {f"r{i}": torch.randint(0, raw["vocab"], (n,), generator=gen).tolist() for i, n in enumerate(lengths)}


FP32_RTOL = 5e-5
BF16_RTOL = 2.0 ** -5


def tolerance(dtype, reference: torch.Tensor) -> float:
    top = max(1.0, float(reference.abs().max()))
    return (FP32_RTOL if dtype in (torch.float32, "float32") else BF16_RTOL) * top


_rounding: dict = {}


def rounding_error(folder: Path, tokens) -> torch.Tensor:
    """Per position, how far the plain model's logits move when what a bfloat16 engine hands from kernel to
    kernel is rounded to bfloat16."""
    key = (str(folder), tuple(tokens))
    if key not in _rounding:
        raw, tensors = read_model(folder)
        exact = plain.forward(raw, tensors, list(tokens))
        plain.narrow = lambda h: h.to(torch.bfloat16).to(h.dtype)
        try:
            rounded = plain.forward(raw, tensors, list(tokens))
        finally:
            plain.narrow = None
        _rounding[key] = (rounded - exact).abs().max(dim=1).values.float()
    return _rounding[key]


ROUNDINGS = 4.0


def row_tolerance(dtype, reference: torch.Tensor, folder: Path, tokens) -> torch.Tensor:
    """The tolerance per position: `tolerance`, and in bfloat16 at least ROUNDINGS times what
    `rounding_error` says. These models' weights are scaled up to make faults visible; the same scaling
    lets a head that is almost empty turn a rounding into a visible change."""
    flat = torch.full((reference.shape[0],), tolerance(dtype, reference))
    if dtype in (torch.float32, "float32"):
        return flat
    return torch.maximum(flat, ROUNDINGS * rounding_error(folder, tokens))
