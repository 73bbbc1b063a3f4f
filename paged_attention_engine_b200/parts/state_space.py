"""The selective state space of Mamba-2 (state-space duality): a recurrent mixer with a matrix state
per head and a decay that each token chooses.

W_in h is z | x | B | C | dt (heads x dv, heads x dv, groups x n, groups x n, heads). x, B and C pass a
short causal convolution per channel, with bias, and silu. With the step dt' = softplus(dt + dt_bias)
and the rate A = exp(A_log) per head, head h reading B and C of group h // (heads / groups):

    S_t = exp(-A dt') S_(t-1) + dt' B_t x_t^T,        y_t = S_t^T C_t + D x_t

y is multiplied by silu(z), RMS-normed in equal parts of its channels with a weight, and projected by
W_o. The request's per-request state is S [heads, n, dv] and the last taps - 1 rows that entered the
convolution, float32; step, decay and recurrence are float32.
"""

from __future__ import annotations

import torch

from ..config.model_spec import PartSpec
from .base import MIXERS, ProjectedMixer, StateNeed, TensorSpec


@MIXERS.register("state_space")
class StateSpace(ProjectedMixer):
    """params: hidden_size, num_heads, value_dim, state_dim, groups, conv_taps, norm_groups, norm_eps.
    tensors: in [2 * inner + 2 * groups * state_dim + heads, hidden] (inner = heads * value_dim); conv
    [channels, taps] and conv.b [channels] (channels = inner + 2 * groups * state_dim); dt_bias, A_log, D
    [heads]; norm [inner]; o [hidden, inner]."""

    @classmethod
    def _sizes(cls, spec: PartSpec):
        p = spec.params
        heads, dv, n, groups = (int(p[k]) for k in ("num_heads", "value_dim", "state_dim", "groups"))
        return heads, dv, n, groups, heads * dv + 2 * groups * n

    @classmethod
    def tensor_specs(cls, spec: PartSpec) -> list[TensorSpec]:
        hidden = int(spec.params["hidden_size"])
        heads, dv, _, _, channels = cls._sizes(spec)
        inner = heads * dv
        name = spec.tensor_name
        return [TensorSpec(name("in"), (inner + channels + heads, hidden), "matrix"),
                TensorSpec(name("conv"), (channels, int(spec.params["conv_taps"])), "taps"),
                TensorSpec(name("conv.b"), (channels,), "vector"),
                TensorSpec(name("dt_bias"), (heads,), "vector"), TensorSpec(name("A_log"), (heads,), "log_rate"),
                TensorSpec(name("D"), (heads,), "scale"), TensorSpec(name("norm"), (inner,), "scale"),
                TensorSpec(name("o"), (hidden, inner), "matrix")]

    @classmethod
    def _state_floats(cls, spec: PartSpec) -> tuple[int, int]:
        heads, dv, n, _, channels = cls._sizes(spec)
        return heads * n * dv, (int(spec.params["conv_taps"]) - 1) * channels

    @classmethod
    def state_need(cls, spec: PartSpec) -> StateNeed:
        memory, rows = cls._state_floats(spec)
        up = lambda floats: (floats + 3) // 4 * 4           # both begin on a 16-byte boundary in every slot
        return StateNeed((up(memory) + up(rows),), torch.float32)

    def __init__(self, spec, tensors, runtime):
        super().__init__(spec, tensors, runtime)
        p = spec.params
        self.num_heads, self.value_dim, self.state_dim, self.groups, self.channels = self._sizes(spec)
        if self.num_heads % self.groups:
            raise ValueError(f"state_space: {self.num_heads} heads in {self.groups} groups")
        self.inner = self.num_heads * self.value_dim
        self.norm_groups, self.norm_eps = int(p["norm_groups"]), float(p["norm_eps"])
        if self.inner % self.norm_groups:
            raise ValueError(f"state_space: {self.inner} channels do not split into {self.norm_groups} norm groups")
        name = spec.tensor_name
        self.in_weight = tensors.pop(name("in"))
        self.conv, self.conv_bias = tensors.pop(name("conv")), tensors.pop(name("conv.b"))
        self.dt_bias, self.a_log, self.skip = (tensors.pop(name(n)) for n in ("dt_bias", "A_log", "D"))
        self.norm_weight, self.o_weight = tensors.pop(name("norm")), tensors.pop(name("o"))
        self.memory_floats, self.conv_floats = self._state_floats(spec)
        self.conv_at = (self.memory_floats + 3) // 4 * 4

    def mix(self, ctx, proj, offset, cache, out, out_offset, mult):
        ops = self.ops
        heads, dv, n, groups, inner = self.num_heads, self.value_dim, self.state_dim, self.groups, self.inner
        memory = cache.state[:, : self.memory_floats]
        rows = cache.state[:, self.conv_at: self.conv_at + self.conv_floats]
        u, step, log_decay, (gate, gate_off) = ops.ssm_prepare(
            proj, offset, inner, offset + inner, self.channels, offset + inner + self.channels, heads, self.conv, self.conv_bias,
            self.dt_bias, self.a_log, rows, ctx.q_start, ctx.q_pos0, ctx.state_slot, ctx.num_seqs, ctx.max_q_len, self.runtime.dtype)
        y = ops.decay_memory((u, inner + groups * n), (u, inner), (u, 0), memory, ctx.q_start, ctx.state_slot, ctx.num_seqs, heads, groups,
                             n, dv, log_decay=log_decay, step=step, skip=self.skip, max_q_len=ctx.max_q_len,
                             num_single=ctx.num_single, multi_index=ctx.multi_index)
        ops.gated_group_norm(y, gate, gate_off, self.norm_groups, self.norm_eps, self.runtime.dtype, weight=self.norm_weight,
                             gate_first=True, mult=mult, out=out, out_off=out_offset)
