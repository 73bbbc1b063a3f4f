"""The gated delta rule: linear attention whose state forgets by a decay that each token chooses and
whose write replaces what the state already holds at the token's key.

W_in h is q | k | v | g | b | a (kv_heads x d twice, heads x dv twice, heads twice). q, k and v pass a short
causal convolution per channel (no bias) and silu; q and k are then unit vectors per head, x / sqrt(sum
x^2 + key_eps), q also times d^(-1/2); head h reads q and k of group h // (heads / kv_heads). With beta =
sigmoid(b) and the decay exp(-exp(A_log) softplus(a + dt_bias)), both per head:

    S <- decay S,    u = beta (v - S^T k),    S <- S + k u^T,    o = S^T q

Each head's o is divided by its root mean square, times a weight that the heads share and silu(g),
and projected by W_o. The request's per-request state is S [heads, d, dv] and the last taps - 1 rows
that entered the convolution, float32; unit vectors, decay, beta and recurrence are float32.
"""

from __future__ import annotations

import torch

from ..config.model_spec import PartSpec
from .base import MIXERS, ProjectedMixer, StateNeed, TensorSpec


@MIXERS.register("gated_delta")
class GatedDelta(ProjectedMixer):
    """params: hidden_size, num_heads, num_kv_heads, head_dim, value_dim, conv_taps, key_eps, norm_eps.
    tensors: q, k [kv_heads * head_dim, hidden]; v, g [heads * value_dim, hidden]; b, a [heads, hidden];
    q.conv, k.conv, v.conv [channels, taps]; A_log, dt_bias [heads]; norm [value_dim]; o [hidden, heads *
    value_dim]."""

    @classmethod
    def _sizes(cls, spec: PartSpec):
        p = spec.params
        return tuple(int(p[k]) for k in ("num_heads", "num_kv_heads", "head_dim", "value_dim"))

    @classmethod
    def _rows(cls, spec: PartSpec) -> dict[str, int]:
        """The rows of the input projections, in the order of the fused product's columns."""
        heads, groups, d, dv = cls._sizes(spec)
        return {"q": groups * d, "k": groups * d, "v": heads * dv, "g": heads * dv, "b": heads, "a": heads}

    @classmethod
    def tensor_specs(cls, spec: PartSpec) -> list[TensorSpec]:
        hidden, taps = int(spec.params["hidden_size"]), int(spec.params["conv_taps"])
        heads, _, _, dv = cls._sizes(spec)
        name, rows = spec.tensor_name, cls._rows(spec)
        return ([TensorSpec(name(n), (r, hidden), "matrix") for n, r in rows.items()]
                + [TensorSpec(name(f"{n}.conv"), (rows[n], taps), "taps") for n in ("q", "k", "v")]
                + [TensorSpec(name("A_log"), (heads,), "log_rate"), TensorSpec(name("dt_bias"), (heads,), "vector"),
                   TensorSpec(name("norm"), (dv,), "scale"), TensorSpec(name("o"), (hidden, heads * dv), "matrix")])

    @classmethod
    def _state_floats(cls, spec: PartSpec) -> tuple[int, int]:
        heads, _, d, dv = cls._sizes(spec)
        rows = cls._rows(spec)
        return heads * d * dv, (int(spec.params["conv_taps"]) - 1) * (rows["q"] + rows["k"] + rows["v"])

    @classmethod
    def state_need(cls, spec: PartSpec) -> StateNeed:
        memory, rows = cls._state_floats(spec)
        up = lambda floats: (floats + 3) // 4 * 4           # both begin on a 16-byte boundary in every slot
        return StateNeed((up(memory) + up(rows),), torch.float32)

    def __init__(self, spec, tensors, runtime):
        super().__init__(spec, tensors, runtime)
        p = spec.params
        self.num_heads, self.num_kv_heads, self.head_dim, self.value_dim = self._sizes(spec)
        if self.num_heads % self.num_kv_heads:
            raise ValueError(f"gated_delta: {self.num_heads} heads over {self.num_kv_heads} kv heads")
        self.key_eps, self.norm_eps = float(p["key_eps"]), float(p["norm_eps"])
        name, rows = spec.tensor_name, self._rows(spec)
        self.in_weight = torch.cat([tensors.pop(name(n)) for n in rows], dim=0).contiguous()
        self.conv = torch.cat([tensors.pop(name(f"{n}.conv")) for n in ("q", "k", "v")], dim=0).contiguous()
        self.a_log, self.dt_bias = tensors.pop(name("A_log")), tensors.pop(name("dt_bias"))
        # one weight for all heads: as long as the heads' channels, the way the norm's kernel reads it
        self.norm_weight = tensors.pop(name("norm")).repeat(self.num_heads).contiguous()
        self.o_weight = tensors.pop(name("o"))
        self.channels = rows["q"] + rows["k"] + rows["v"]
        self.gate_at = self.channels
        self.beta_at = self.gate_at + rows["g"]
        self.decay_at = self.beta_at + rows["b"]
        self.memory_floats, self.conv_floats = self._state_floats(spec)
        self.conv_at = (self.memory_floats + 3) // 4 * 4

    def mix(self, ctx, proj, offset, cache, out, out_offset, mult):
        ops = self.ops
        heads, groups, d, dv = self.num_heads, self.num_kv_heads, self.head_dim, self.value_dim
        memory = cache.state[:, : self.memory_floats]
        rows = cache.state[:, self.conv_at: self.conv_at + self.conv_floats]
        u, _, log_decay, (gate, gate_off), beta = ops.ssm_prepare(
            proj, offset + self.gate_at, heads * dv, offset, self.channels, offset + self.decay_at, heads, self.conv, None,
            self.dt_bias, self.a_log, rows, ctx.q_start, ctx.q_pos0, ctx.state_slot, ctx.num_seqs, ctx.max_q_len, self.runtime.dtype,
            beta_off=offset + self.beta_at)
        y = ops.gated_delta((u, 0), (u, groups * d), (u, 2 * groups * d), log_decay, beta, memory, ctx.q_start, ctx.state_slot,
                            ctx.num_seqs, heads, groups, d, dv, self.key_eps, q_scale=float(d) ** -0.5, max_q_len=ctx.max_q_len,
                            num_single=ctx.num_single, multi_index=ctx.multi_index)
        ops.gated_group_norm(y, gate, gate_off, heads, self.norm_eps, self.runtime.dtype, weight=self.norm_weight, mult=mult,
                             out=out, out_off=out_offset)
