"""A plain, slow Getozen: one function per mechanism, written from the design's equations.

Everything runs on the CPU in float64 over one whole sequence at a time, the recurrences as loops
over tokens. It shares no code with the engine: it reads a dictionary of tensors by their checkpoint
names and the config.json dictionary.

Notation: T tokens, W model width, H heads, G key/value heads or groups, d key size, n state size,
dv value size, positions p = 0..T-1.
"""

from __future__ import annotations

import math

import torch

F = torch.float64

# A function applied wherever a 16-bit engine hands numbers on as 16 bits (a sublayer's input, heads
# after rotation, channels after the convolution, an output product's operand), or None. Tests set it to
# a rounding to bfloat16 to learn how far such roundings move a model's logits.
narrow = None


def _f(t):
    return t.to(F)


def _handed(h):
    return narrow(h) if narrow is not None else h


def silu(x):
    return x / (1.0 + torch.exp(-x))


def softplus(x):
    return torch.maximum(x, torch.zeros_like(x)) + torch.log1p(torch.exp(-x.abs()))


def dynamic_tanh(x, tensors, name):
    """tanh(alpha x) * w + b: a norm without statistics. alpha is a scalar, w and b vectors."""
    return torch.tanh(_f(tensors[f"{name}.alpha"]) * x) * _f(tensors[name]) + _f(tensors[f"{name}.b"])


def unit_rms(x, eps):
    """x over the root of its mean square (eps inside the root), along the last axis."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


# --------------------------------------------------------------------------- #
# Rotation and attention
# --------------------------------------------------------------------------- #

def frequencies(rot):
    """base^(-2i / dims) for every pair i; with linear scaling each divided by the factor."""
    factor = float(rot["scaling"]["factor"]) if rot.get("scaling") else 1.0
    return [float(rot["base"]) ** (-2.0 * i / rot["dims"]) / factor for i in range(rot["dims"] // 2)]


def rotate(x, rot, neighbours, first=0):
    """Rotates the first rot.dims channels of x [T, H, d] by position * frequency. `neighbours`: pair i
    is channels (2i, 2i + 1); otherwise (i, i + dims / 2). Token t stands at position first + t."""
    out = x.clone()
    half = rot["dims"] // 2
    positions = torch.arange(first, first + x.shape[0], dtype=F)
    for i, f in enumerate(frequencies(rot)):
        a, b = (2 * i, 2 * i + 1) if neighbours else (i, i + half)
        c, s = torch.cos(positions * f)[:, None], torch.sin(positions * f)[:, None]
        out[:, :, a] = x[:, :, a] * c - x[:, :, b] * s
        out[:, :, b] = x[:, :, b] * c + x[:, :, a] * s
    return out


def causal_attention(q, k, v, scale):
    """q [T, H, d], k [T, G, d], v [T, G, dv]: softmax attention over j <= i; head h reads h // (H / G)."""
    T, H, _ = q.shape
    G = k.shape[1]
    mask = torch.ones(T, T, dtype=torch.bool).tril()
    out = torch.zeros(T, H, v.shape[2], dtype=F)
    for h in range(H):
        g = h // (H // G)
        scores = (q[:, h] @ k[:, g].T) * scale
        scores = torch.where(mask, scores, torch.tensor(-math.inf, dtype=F))
        weights = torch.exp(scores - scores.max(dim=1, keepdim=True).values)
        out[:, h] = (weights / weights.sum(dim=1, keepdim=True)) @ v[:, g]
    return out


def attention_mixer(h, tensors, name, m):
    T = h.shape[0]
    proj = lambda n: h @ _f(tensors[f"{name}.{n}"]).T
    biased = lambda n: proj(n) + _f(tensors[f"{name}.{n}.b"])
    q, k, v = (biased(n).view(T, heads, size) for n, heads, size in
               (("q", m["heads"], m["dim"]), ("k", m["kv_heads"], m["dim"]), ("v", m["kv_heads"], m["vdim"])))
    o = _handed(causal_attention(_handed(rotate(q, m["rot"], True)), _handed(rotate(k, m["rot"], True)), _handed(v), m["scale"]))
    gate = 1.0 / (1.0 + torch.exp(-proj("g")))
    return _handed(o.reshape(T, -1) * gate) @ _f(tensors[f"{name}.o"]).T


# --------------------------------------------------------------------------- #
# Recurrences
# --------------------------------------------------------------------------- #

def decayed_memory(q, k, v, keep, state=None):
    """S <- keep[t] S + k[t] v[t]^T, o[t] = S^T q[t], per head: q, k [T, H, d], v [T, H, dv], keep
    [T, H]. -> (o [T, H, dv], the last S [H, d, dv]); `state` is the S to start from (zero)."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=F) if state is None else state.clone()
    out = torch.zeros(T, H, v.shape[2], dtype=F)
    for t in range(T):
        S = keep[t][:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(dim=1)
    return out, S


def retention_mixer(h, tensors, name, m, eps):
    T, H = h.shape[0], m["heads"]
    proj = lambda n: h @ _f(tensors[f"{name}.{n}"]).T
    q, k = (_handed(rotate(proj(n).view(T, H, -1), m["rot"], False)) for n in ("q", "k"))
    k = k * float(m["dim"]) ** -0.5
    keep = torch.tensor(m["decay"], dtype=F).expand(T, H)
    o, _ = decayed_memory(q, k, _handed(proj("v").view(T, H, -1)), keep)
    return _handed(unit_rms(o, eps).reshape(T, -1) * silu(proj("g"))) @ _f(tensors[f"{name}.o"]).T


def short_convolution(u, taps, bias):
    """y[t, c] = bias[c] + sum_j taps[c, j] u[t - n + 1 + j, c] for n taps; zeros before the start."""
    n = taps.shape[1]
    padded = torch.cat([torch.zeros(n - 1, u.shape[1], dtype=F), u])
    return _f(bias) + sum(_f(taps)[:, j] * padded[j: j + u.shape[0]] for j in range(n))


def selective_memory(x, B, C, step, rate, skip):
    """x [T, H, dv], B and C [T, G, n], step [T, H], rate and skip [H]: S <- exp(-rate step) S + step B x^T,
    y = S^T C + skip x; head h reads group h // (H / G)."""
    H, G = x.shape[1], B.shape[1]
    group = [h // (H // G) for h in range(H)]
    y, _ = decayed_memory(C[:, group], step[:, :, None] * B[:, group], x, torch.exp(-rate * step))
    return y + skip[:, None] * x


def mamba2_mixer(h, tensors, name, m, eps):
    T, H, dv, n, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * dv
    z, xbc, dt = (h @ _f(tensors[f"{name}.in"]).T).split([inner, inner + 2 * G * n, H], dim=1)
    xbc = _handed(silu(short_convolution(xbc, tensors[f"{name}.conv"], tensors[f"{name}.conv.b"])))
    x, B, C = xbc.split([inner, G * n, G * n], dim=1)
    step = softplus(dt + _f(tensors[f"{name}.dt_bias"]))
    y = selective_memory(x.view(T, H, dv), B.view(T, G, n), C.view(T, G, n), step, torch.exp(_f(tensors[f"{name}.A_log"])),
                         _f(tensors[f"{name}.D"])).reshape(T, inner)
    y = unit_rms((y * silu(z)).view(T, m["norm_groups"], -1), eps).reshape(T, inner) * _f(tensors[f"{name}.norm"])
    return _handed(y) @ _f(tensors[f"{name}.o"]).T


# --------------------------------------------------------------------------- #
# The model
# --------------------------------------------------------------------------- #

def mixer(h, tensors, name, kind, m, eps):
    if kind != "parallel":
        return mamba2_mixer(h, tensors, name, m, eps)
    return (m["left_scale"] * attention_mixer(h, tensors, f"{name}.left", m["left"])
            + m["right_scale"] * retention_mixer(h, tensors, f"{name}.right", m["right"], eps))


def relu_glu(h, tensors, name):
    gate, up = h @ _f(tensors[f"{name}.gate"]).T, h @ _f(tensors[f"{name}.up"]).T
    return _handed(torch.maximum(gate, torch.zeros_like(gate)) * up) @ _f(tensors[f"{name}.down"]).T


def layer(x, tensors, name, entry, eps):
    """Both sublayers read the same x, each through a norm of its own."""
    out = mixer(_handed(dynamic_tanh(x, tensors, f"{name}.norm1")), tensors, f"{name}.mix", entry["type"], entry["mixer"], eps)
    if entry.get("mlp"):
        out = out + relu_glu(_handed(dynamic_tanh(x, tensors, f"{name}.norm2")), tensors, f"{name}.mlp")
    return x + out


def forward(config, tensors, tokens, layers_out=None):
    """float64 logits [T, vocab]. `layers_out`, a list, receives the stream after every layer."""
    x = _f(tensors["embed"])[torch.tensor(list(tokens))]
    for i, entry in enumerate(config["layers"]):
        x = layer(x, tensors, f"l{entry.get('weights_of', i)}", entry, config["norm"]["eps"])
        if layers_out is not None:
            layers_out.append(x)
    return dynamic_tanh(x, tensors, "final.norm") @ _f(tensors["head"]).T
