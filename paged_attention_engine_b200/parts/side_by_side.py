"""Mixers side by side: several mixers read the same input, and the layer gets the weighted sum of their
outputs, each as it is or each normed first.

Every one of them has the form W_o mix(W_in h) (a `ProjectedMixer`), so the plain sum needs no kernel of its own:
the input projections are one product whose columns the mixers share out, each mixer writes its
scaled operand into its own columns of one matrix, and the output projections, laid beside each other
along their input channels, are one product over all of them, which adds the outputs up in its
float32 accumulator.

With `out_norm_eps` every output is RMS-normed over the model's width, with a weight of its own, before it
is scaled and added. The input product is shared as before; the output products are one per mixer, and the
norms and the sum are left to the kernel that reads the layer's output (`ops.normed_branches`).
"""

from __future__ import annotations

import torch

from ..config.model_spec import PartSpec
from .base import MIXERS, CacheNeed, ProjectedMixer, StateNeed, TensorSpec


@MIXERS.register("side_by_side")
class SideBySide(ProjectedMixer):
    """params: mixers, a list of {"kind", "params", "name" (its tensors are under <prefix>.<name>), "scale"}.
    At most one of the mixers may need pages and at most one per-request state. out_norm_eps (absent: the outputs
    are not normed) and, with it, hidden_size. No tensors of its own but, with out_norm_eps, <name>.out [hidden] for
    every mixer."""

    @classmethod
    def tensor_specs(cls, spec: PartSpec) -> list[TensorSpec]:
        if spec.params.get("out_norm_eps") is None:
            return []
        return [TensorSpec(spec.tensor_name(f"{m['name']}.out"), (int(spec.params["hidden_size"]),), "scale") for m in spec.params["mixers"]]

    @classmethod
    def sub_parts(cls, spec: PartSpec) -> list[tuple[str, PartSpec]]:
        return [("mixer", PartSpec(m["kind"], m["params"], spec.tensor_name(m["name"]))) for m in spec.params["mixers"]]

    @classmethod
    def _only(cls, spec: PartSpec, which: str):
        found = []
        for _, sub in cls.sub_parts(spec):
            need = getattr(MIXERS.get(sub.kind), which)(sub)
            if need is not None:
                found.append(need)
        if len(found) > 1:
            raise ValueError(f"side_by_side: {len(found)} mixers have a {which}; one layer run has one cache and one state")
        return found[0] if found else None

    @classmethod
    def cache_need(cls, spec: PartSpec) -> CacheNeed | None:
        return cls._only(spec, "cache_need")

    @classmethod
    def state_need(cls, spec: PartSpec) -> StateNeed | None:
        return cls._only(spec, "state_need")

    def __init__(self, spec, tensors, runtime):
        super().__init__(spec, tensors, runtime)
        self.out_norm_eps = spec.params.get("out_norm_eps")
        if self.out_norm_eps is not None:
            self.out_norms = [tensors.pop(spec.tensor_name(f"{m['name']}.out")) for m in spec.params["mixers"]]
        self.mixers = self.build_sub_parts(tensors)
        for m in self.mixers:
            if not isinstance(m, ProjectedMixer):
                raise ValueError(f"side_by_side: a '{m.spec.kind}' mixer is not one product in front and one behind")
        self.scales = [float(m.get("scale", 1.0)) for m in spec.params["mixers"]]
        columns = [int(m.in_weight.shape[0]) for m in self.mixers]
        if any(m.in_bias is not None for m in self.mixers):
            self.in_bias = torch.cat([m.in_bias if m.in_bias is not None else torch.zeros(n, dtype=torch.float32, device=runtime.device)
                                      for m, n in zip(self.mixers, columns)]).contiguous()
        self.in_weight = torch.cat([m.in_weight for m in self.mixers], dim=0).contiguous()
        self.o_weights = [m.o_weight for m in self.mixers]
        if self.out_norm_eps is None:
            self.o_weight = torch.cat(self.o_weights, dim=1).contiguous()
            self.o_weights = None
        self.places, at, out_at = [], 0, 0
        for m, n in zip(self.mixers, columns):
            self.places.append((at, out_at))
            at, out_at = at + n, out_at + m.out_width
        for m in self.mixers:           # their weights live in the shared products
            m.in_weight = m.in_bias = m.o_weight = None

    def mix(self, ctx, proj, offset, cache, out, out_offset, mult):
        for m, scale, (at, out_at) in zip(self.mixers, self.scales, self.places):
            m.mix(ctx, proj, offset + at, cache, out, out_offset + out_at, mult * scale)

    def forward(self, ctx, x, residual, cache):
        if self.out_norm_eps is None:
            return super().forward(ctx, x, residual, cache)
        if residual is not None:
            raise ValueError("side_by_side: normed outputs leave without a residual")
        ops = self.ops
        proj = ops.linear(x, self.in_weight, self.in_bias, None, out_dtype=torch.float32)
        branches = []
        for m, scale, weight, norm, (at, _) in zip(self.mixers, self.scales, self.o_weights, self.out_norms, self.places):
            operand = m.operand(ctx, proj, at, cache, int(weight.shape[1]))
            branches.append((ops.linear(operand, weight, None, None, out_dtype=torch.float32), norm, scale))
        return ops.normed_branches(branches, float(self.out_norm_eps))
