"""Mixers side by side: several mixers read the same input, and the layer gets the weighted sum of their
outputs.

Every one of them has the form W_o mix(W_in h) (a `ProjectedMixer`), so the sum needs no kernel of its own:
the input projections are one product whose columns the mixers share out, each mixer writes its
scaled operand into its own columns of one matrix, and the output projections, laid beside each other
along their input channels, are one product over all of them, which adds the outputs up in its
float32 accumulator.
"""

from __future__ import annotations

import torch

from ..config.model_spec import PartSpec
from .base import MIXERS, CacheNeed, ProjectedMixer, StateNeed


@MIXERS.register("side_by_side")
class SideBySide(ProjectedMixer):
    """params: mixers, a list of {"kind", "params", "name" (its tensors are under <prefix>.<name>), "scale"}.
    At most one of the mixers may need pages and at most one per-request state. No tensors of its own."""

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
        self.o_weight = torch.cat([m.o_weight for m in self.mixers], dim=1).contiguous()
        self.places, at, out_at = [], 0, 0
        for m, n in zip(self.mixers, columns):
            self.places.append((at, out_at))
            at, out_at = at + n, out_at + m.out_width
        for m in self.mixers:           # their weights live in the shared products
            m.in_weight = m.in_bias = m.o_weight = None

    def mix(self, ctx, proj, offset, cache, out, out_offset, mult):
        for m, scale, (at, out_at) in zip(self.mixers, self.scales, self.places):
            m.mix(ctx, proj, offset + at, cache, out, out_offset + out_at, mult * scale)
