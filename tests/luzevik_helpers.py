"""Small Luzevik configurations and the glue between model folders and the plain implementation."""

from __future__ import annotations

import json
from pathlib import Path

import torch

from plain import luzevik_plain as plain


def rot(dims, base, factor=None):
    out = {"base": base, "dims": dims}
    if factor:
        out["scaling"] = {"factor": factor}
    return out


def latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, base=10000.0, kv_from=None, mlp=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "scale": scale,
         "rot": rot(rot_dim, base)}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def parallel(left, right, mlp=None):
    """left: (heads, kv_heads, dim, vdim, scale, rot); right: (heads, kv_heads, dim, vdim, conv)."""
    return {"type": "parallel", "mixer": {
        "left": dict(zip(("heads", "kv_heads", "dim", "vdim", "scale", "rot"), left)),
        "right": dict(zip(("heads", "kv_heads", "dim", "vdim", "conv"), right))}, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def config(vocab, width, layers, scale=3.0, eps=1e-5):
    return {"architecture": "Luzevik", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "norm": {"eps": eps}, "layers": layers}


# Odd sizes: a width that is no multiple of 8, value heads larger and smaller than key heads, a partly and a
# wholly rotated head, with and without scaling, groups of two, of three and of one, three and five taps;
# two latents of different sizes, each read by later layers, one of them across the other; layers
# without a feed-forward; a mixture that chooses every expert.
SMALL_A = config(211, 60, [
    latent(3, 10, 6, 14, 20, 18, 0.3, 40.0, mlp=dense(44)),
    parallel((4, 2, 12, 20, 0.3, rot(8, 40.0, 3.0)), (6, 3, 10, 6, 3), moe(24, 5, 2)),
    latent(2, 8, 6, 10, 20, 12, 0.35, 40.0, kv_from=0),
    latent(4, 6, 8, 6, 12, 24, 0.4, 90.0, mlp=moe(16, 3, 3)),
    parallel((3, 3, 16, 8, 0.25, rot(16, 900.0)), (2, 1, 7, 9, 5)),
    latent(5, 12, 8, 4, 12, 10, 0.3, 90.0, kv_from=3, mlp=dense(20)),
    latent(3, 10, 6, 14, 20, 18, 0.3, 40.0, kv_from=0, mlp=moe(8, 6, 1)),
])
# Sizes that the tensor-core kernels take: the plain attention kernels (one head size), the scored ones (two),
# latent attention, the delta rule in chunks, grouped experts with the gate in the product's epilogue.
SMALL_B = config(257, 128, [
    parallel((4, 2, 64, 64, 0.125, rot(64, 10000.0, 4.0)), (4, 2, 64, 32, 4), dense(256)),
    latent(4, 48, 16, 32, 80, 96, 0.14, 20000.0, mlp=moe(64, 7, 2)),
    parallel((6, 3, 32, 128, 0.17, rot(16, 5000.0, 2.0)), (6, 2, 32, 64, 2), moe(32, 16, 4)),
    latent(9, 16, 16, 16, 80, 64, 0.2, 20000.0, kv_from=1, mlp=dense(160)),
], scale=7.0, eps=1e-6)
# One of everything: heads, groups, taps, experts; factors and scales of 1.
ONES = config(97, 56, [
    parallel((1, 1, 8, 24, 0.4, rot(2, 100.0, 1.0)), (1, 1, 8, 16, 1), moe(20, 1, 1)),
    latent(1, 8, 2, 8, 8, 8, 0.4, 100.0, mlp=dense(28)),
], scale=1.0)
# A latent wider than 256 channels, more heads than a block's rows, keys of the delta rule wider than 128 and than
# 256 channels, value heads wider than a block's columns, the longest convolution, a head of 48 value channels.
WIDE = config(97, 64, [
    latent(40, 16, 16, 16, 288, 40, 0.2, mlp=dense(64)),
    parallel((2, 1, 128, 48, 0.09, rot(96, 10000.0, 8.0)), (2, 2, 136, 72, 17), moe(16, 9, 3)),
    parallel((2, 2, 128, 128, 0.09, rot(128, 10000.0)), (2, 1, 264, 16, 4), dense(48)),
], scale=5.0)
# As SMALL_B, every expert chosen by every token: long prompts need no drawing.
ALL_CHOSEN = dict(SMALL_B, layers=[dict(e, mlp=moe(32, 3, 3) if e["mlp"]["kind"] == "moe" else e["mlp"]) for e in SMALL_B["layers"]])
SMALL = {"small_a": (SMALL_A, 4, 61), "small_b": (SMALL_B, 16, 62), "ones": (ONES, 8, 63), "wide": (WIDE, 16, 64)}   # config, page size, seed


def write_model(folder: Path, raw: dict, seed: int, dtype=torch.bfloat16, sharpen: float = 3.0) -> Path:
    """A random model folder whose numbers make faults visible: projections scaled up (one key's score
    stands out), sinks, biases, gates, taps, decays and rates of a size that matters, norm weights of
    both signs, router logits far enough apart that the choice is no close call and a bias that changes
    it. Decays are spread so that some heads forget within a few tokens and others hold what they saw long ago."""
    from safetensors.torch import load_file, save_file

    from paged_attention_engine_b200.weights import write_random_model

    write_random_model(folder, raw, seed, dtype)
    path = str(Path(folder) / "model.safetensors")
    tensors = load_file(path)
    gen = torch.Generator().manual_seed(seed + 1000)
    for name in list(tensors):
        t = tensors[name].float()
        if name.endswith(("norm1", "norm2", "final.norm", ".right.norm", ".left.out", ".right.out", ".left.q.norm", ".left.k.norm")):
            t = (0.5 + torch.rand(t.shape, generator=gen)) * (torch.randint(0, 2, t.shape, generator=gen) * 2.0 - 1.0)
        elif name.endswith((".dq.norm", ".dkv.norm")):
            t = 1.0 + torch.rand(t.shape, generator=gen)
        elif name.endswith(".sink"):
            t = torch.randn(t.shape, generator=gen) * 1.5
        elif name.endswith((".q.b", ".k.b", ".v.b")):
            t = torch.randn(t.shape, generator=gen) * 0.3
        elif name.endswith(".router"):
            t = t * 12.0
        elif name.endswith(".router.b"):
            t = torch.randn(t.shape, generator=gen) * 0.5
        elif name.endswith((".right.g", ".right.a")):
            t = t * 8.0
        elif name.endswith(".dt_bias"):
            t = torch.rand(t.shape, generator=gen) * 4.0 - 4.0
        elif name.endswith(".A_log"):
            t = torch.rand(t.shape, generator=gen) * 4.0 - 3.0
        elif name == "embed":
            t = t * 20.0
        elif t.dim() == 2 and not name.endswith(".conv"):
            t = t * sharpen
        tensors[name] = t.to(tensors[name].dtype)
    save_file(tensors, path)
    return Path(folder)


def read_model(folder: Path):
    from safetensors.torch import load_file

    return json.loads((Path(folder) / "config.json").read_text()), load_file(str(Path(folder) / "model.safetensors"))


def plain_logits(folder: Path, tokens) -> torch.Tensor:
    raw, tensors = read_model(folder)
    return plain.forward(raw, tensors, list(tokens)).float()


# How many times the plain model's own roundings a bfloat16 engine, which rounds in other places, may be off.
ROUNDINGS = 4.0
# A router's choice is a step function of its input: where two experts' logits are closer than rounding can
# move them, the engine may choose otherwise than the plain model, and rightly so. The tests' prompts
# avoid such tokens: a token whose choice is closer than this (in any routed layer), after several times what
# a bfloat16 engine's roundings do to that very choice is taken off, is drawn again.
CLEAR_CHOICE = 0.1


def margins_of(raw, tensors, tokens):
    """(logits, per position the closest choice of any router, less ROUNDINGS times what rounding moves it by)."""
    exact, rounded = [], []
    out = plain.forward(raw, tensors, tokens, margins=exact)
    if not exact:
        return out, torch.full((len(tokens),), float("inf"))
    plain.narrow = lambda h: h.to(torch.bfloat16).to(h.dtype)
    try:
        plain.forward(raw, tensors, tokens, margins=rounded)
    finally:
        plain.narrow = None
    exact, rounded = torch.stack(exact), torch.stack(rounded)
    return out, (exact - ROUNDINGS * (exact - rounded).abs()).min(dim=0).values


def clear_requests(folder: Path, lengths, seed: int, margin: float = CLEAR_CHOICE):
    """(requests, logits): prompts of the given lengths for which no router's choice is a close
    call, drawn from `seed`, and the plain model's logits for them."""
    key = (str(folder), tuple(lengths), seed, margin)
    if key not in _drawn:
        _drawn[key] = _draw(folder, lengths, seed, margin)
    return _drawn[key]


_drawn: dict = {}


def _draw(folder: Path, lengths, seed: int, margin: float):
    raw, tensors = read_model(folder)
    gen = torch.Generator().manual_seed(seed)
    requests, logits = {}, {}
    for i, n in enumerate(lengths):
        tokens = torch.randint(0, raw["vocab"], (n,), generator=gen).tolist()
        for _ in range(60 + 2 * n):
            out, closest = margins_of(raw, tensors, tokens)
            close = (closest < margin).nonzero()
            if not len(close):
                break
            tokens[int(close[0])] = int(torch.randint(0, raw["vocab"], (1,), generator=gen))
        else:
            raise AssertionError(f"no prompt of {n} tokens with clear choices was found")
        requests[f"r{i}"], logits[f"r{i}"] = tokens, out.float()
    return requests, logits


FP32_RTOL = 5e-5
BF16_RTOL = 2.0 ** -5


def tolerance(dtype, reference: torch.Tensor) -> float:
    top = max(1.0, float(reference.abs().max()))
    return (FP32_RTOL if dtype in (torch.float32, "float32") else BF16_RTOL) * top


_rounding: dict = {}


def rounding_error(folder: Path, tokens) -> torch.Tensor:
    """Per position, how far the plain model's logits move when what a bfloat16 engine hands from kernel to
    kernel is rounded to bfloat16: the most of three grids of the same fineness, since one draw of the
    roundings may happen to cancel where another does not."""
    key = (str(folder), tuple(tokens))
    if key not in _rounding:
        raw, tensors = read_model(folder)
        exact = plain.forward(raw, tensors, list(tokens))
        errors = []
        for grid in (1.0, 1.1, 1.3):
            plain.narrow = lambda h: (h * grid).to(torch.bfloat16).to(h.dtype) / grid
            try:
                errors.append((plain.forward(raw, tensors, list(tokens)) - exact).abs().max(dim=1).values.float())
            finally:
                plain.narrow = None
        _rounding[key] = torch.stack(errors).max(dim=0).values
    return _rounding[key]


def row_tolerance(dtype, reference: torch.Tensor, folder: Path, tokens) -> torch.Tensor:
    """The tolerance per position: `tolerance`, and in bfloat16 at least ROUNDINGS times what
    `rounding_error` says: these models' weights are scaled up to make faults visible, and the same
    scaling lets a head whose read-out nearly cancels turn a rounding into a visible change."""
    flat = torch.full((reference.shape[0],), tolerance(dtype, reference))
    if dtype in (torch.float32, "float32"):
        return flat
    return torch.maximum(flat, ROUNDINGS * rounding_error(folder, tokens))
