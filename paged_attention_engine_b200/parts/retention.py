"""Retention: linear attention with a fixed decay per head, without softmax or denominator.

With q = W_q h and k = W_k h (heads x d), v = W_v h (heads x dv), q and k rotated by the step's
positions and k multiplied by d^(-1/2) afterwards:

    S_t = decay S_(t-1) + k_t v_t^T,        o_t = S_t^T q_t

Each head's o is divided by its root mean square, multiplied by silu(W_g h), and projected by W_o.
The state starts at zero, is float32, and is the request's per-request state [heads, d, dv].
"""

from __future__ import annotations

import torch

from ..config.model_spec import PartSpec
from .base import MIXERS, ProjectedMixer, StateNeed, TensorSpec


@MIXERS.register("retention")
class Retention(ProjectedMixer):
    """params: hidden_size, num_heads, head_dim, value_dim, decay (a number per head), norm_eps, pairing
    ("half", the default, or "interleaved"), position_encoding (a dict with its `kind` and `dims`, or
    None). tensors: q, k [heads * head_dim, hidden]; v, g [heads * value_dim, hidden]; o [hidden, heads *
    value_dim]."""

    @classmethod
    def _sizes(cls, spec: PartSpec):
        p = spec.params
        d = int(p["head_dim"])
        return int(p["num_heads"]), d, int(p.get("value_dim") or d)

    @classmethod
    def tensor_specs(cls, spec: PartSpec) -> list[TensorSpec]:
        hidden = int(spec.params["hidden_size"])
        heads, d, dv = cls._sizes(spec)
        name = spec.tensor_name
        return ([TensorSpec(name(n), (heads * d, hidden), "matrix") for n in ("q", "k")]
                + [TensorSpec(name(n), (heads * dv, hidden), "matrix") for n in ("v", "g")]
                + [TensorSpec(name("o"), (hidden, heads * dv), "matrix")])

    @classmethod
    def sub_parts(cls, spec: PartSpec) -> list[tuple[str, PartSpec]]:
        enc = spec.params.get("position_encoding")
        if enc is None:
            return []
        return [("position_encoding", PartSpec(enc["kind"], {k: v for k, v in enc.items() if k != "kind"}, spec.prefix))]

    @classmethod
    def state_need(cls, spec: PartSpec) -> StateNeed:
        return StateNeed(cls._sizes(spec), torch.float32)

    def __init__(self, spec, tensors, runtime):
        super().__init__(spec, tensors, runtime)
        p = spec.params
        self.num_heads, self.head_dim, self.value_dim = self._sizes(spec)
        decay = [float(x) for x in p["decay"]]
        if len(decay) != self.num_heads or min(decay) < 0.0:
            raise ValueError(f"retention: decays {decay} for {self.num_heads} heads")
        self.decay = torch.tensor(decay, dtype=torch.float32, device=runtime.device)
        self.norm_eps = float(p["norm_eps"])
        if p.get("pairing", "half") not in ("half", "interleaved"):
            raise ValueError(f"retention: pairing '{p.get('pairing')}' (half, interleaved)")
        self.interleaved = p.get("pairing", "half") == "interleaved"
        # One product for q | k | v | g: the columns of its output in that order.
        self.in_weight = torch.cat([tensors.pop(spec.tensor_name(n)) for n in ("q", "k", "v", "g")], dim=0).contiguous()
        self.o_weight = tensors.pop(spec.tensor_name("o"))
        built = self.build_sub_parts(tensors)
        self.position_encoding = built[0] if built else None

    def mix(self, ctx, proj, offset, cache, out, out_offset, mult):
        ops = self.ops
        heads, d, dv = self.num_heads, self.head_dim, self.value_dim
        proj = ops.materialized(proj)
        dtype, tokens = self.runtime.dtype, proj.shape[0]
        k_off, v_off, g_off = offset + heads * d, offset + 2 * heads * d, offset + 2 * heads * d + heads * dv
        k = torch.empty((tokens, heads * d), dtype=dtype, device=proj.device)
        v = torch.empty((tokens, heads * dv), dtype=dtype, device=proj.device)
        q = ops.head_prep(
            proj, q_off=offset, k_off=k_off, v_off=v_off, heads=heads, kv_heads=heads, q_dim=d, k_dim=d, value_dim=dv,
            q_norm=None, k_norm=None, q_span=0, k_span=0, eps=0.0,
            table=self.position_encoding.table(ctx) if self.position_encoding is not None else None,
            interleaved=self.interleaved, q_rot0=0, k_rot0=0, slots=None, keys=k, values=v, page_size=1, out_dtype=dtype, direct=True)
        o = ops.decay_memory((q, 0), (k, 0), (v, 0), cache.state, ctx.q_start, ctx.state_slot, ctx.num_seqs, heads, heads, d, dv,
                             head_decay=self.decay, k_scale=float(d) ** -0.5, max_q_len=ctx.max_q_len, num_single=ctx.num_single,
                             multi_index=ctx.multi_index)
        ops.gated_group_norm(o, proj, g_off, heads, self.norm_eps, dtype, mult=mult, out=out, out_off=out_offset)
