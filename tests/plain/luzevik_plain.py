"""A plain, slow Luzevik: one function per mechanism, written from the design's equations.

Everything runs on the CPU in float64 over one whole sequence at a time, the recurrence as a loop over
tokens, the mixture token by token. It shares no code with the engine: it reads a dictionary of
tensors by their checkpoint names and the config.json dictionary.

Notation: T tokens, W model width, H heads, G key/value heads, d key size, dv value size, positions
p = 0..T-1.
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


def product(x, tensors, name):
    return x @ _f(tensors[name]).T


def sigmoid(x):
    return 1.0 / (1.0 + torch.exp(-x))


def silu(x):
    return x * sigmoid(x)


def softplus(x):
    return torch.maximum(x, torch.zeros_like(x)) + torch.log1p(torch.exp(-x.abs()))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z * z * z)))


def rms(x, weight, eps):
    """x over the root of its mean square (eps inside the root), along the last axis, times a weight."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * _f(weight)


# --------------------------------------------------------------------------- #
# Rotation and attention
# --------------------------------------------------------------------------- #

def frequencies(rot):
    """base^(-2i / dims) for every pair i; with linear scaling each divided by the factor."""
    factor = float(rot["scaling"]["factor"]) if rot.get("scaling") else 1.0
    return [float(rot["base"]) ** (-2.0 * i / rot["dims"]) / factor for i in range(rot["dims"] // 2)]


def rotate(x, rot, first=0):
    """Rotates the first rot.dims channels of x [T, H, d] by position * frequency; pair i is channels
    (i, i + dims / 2). Token t stands at position first + t."""
    out = x.clone()
    half = rot["dims"] // 2
    positions = torch.arange(first, first + x.shape[0], dtype=F)
    for i, f in enumerate(frequencies(rot)):
        c, s = torch.cos(positions * f)[:, None], torch.sin(positions * f)[:, None]
        u, v = x[:, :, i], x[:, :, i + half]
        out[:, :, i] = u * c - v * s
        out[:, :, i + half] = v * c + u * s
    return out


def causal_attention(q, k, v, scale, sink=None):
    """q [T, H, d], k [T, G, d], v [T, G, dv]: softmax attention over j <= i; head h reads h // (H / G);
    `sink` [H]: one more term exp(sink_h) in head h's denominator, without a value."""
    T, H, _ = q.shape
    G = k.shape[1]
    mask = torch.ones(T, T, dtype=torch.bool).tril()
    out = torch.zeros(T, H, v.shape[2], dtype=F)
    for h in range(H):
        g = h // (H // G)
        scores = (q[:, h] @ k[:, g].T) * scale
        scores = torch.where(mask, scores, torch.tensor(-math.inf, dtype=F))
        top = scores.max(dim=1, keepdim=True).values
        if sink is not None:
            top = torch.maximum(top, _f(sink)[h])
        weights = torch.exp(scores - top)
        total = weights.sum(dim=1, keepdim=True)
        if sink is not None:
            total = total + torch.exp(_f(sink)[h] - top)
        out[:, h] = (weights / total) @ v[:, g]
    return out


def attention_mixer(h, tensors, name, m, eps):
    """Grouped queries, biases, a norm per head before the rotation, every earlier key. -> [T, W]"""
    T = h.shape[0]
    biased = lambda n, heads, size: (product(h, tensors, f"{name}.{n}") + _f(tensors[f"{name}.{n}.b"])).view(T, heads, size)
    q, k, v = biased("q", m["heads"], m["dim"]), biased("k", m["kv_heads"], m["dim"]), biased("v", m["kv_heads"], m["vdim"])
    q = rotate(rms(q, tensors[f"{name}.q.norm"], eps), m["rot"])
    k = rotate(rms(k, tensors[f"{name}.k.norm"], eps), m["rot"])
    o = causal_attention(_handed(q), _handed(k), _handed(v), m["scale"])
    return product(_handed(o.reshape(T, -1)), tensors, f"{name}.o")


def latent_of(h, tensors, name, m, eps):
    """The token's normed latent [T, kv_rank] and the rotated key part of all heads [T, rot_dim]."""
    down = product(h, tensors, f"{name}.dkv")
    c, shared = down[:, :m["kv_rank"]], down[:, m["kv_rank"]:]
    return _handed(rms(c, tensors[f"{name}.dkv.norm"], eps)), _handed(rotate(shared[:, None, :], m["rot"])[:, 0])


def latent_mixer(h, tensors, name, m, eps, latent):
    """`latent` = (c, shared part), this layer's own or an earlier one's. Keys and values expanded per head. -> [T, W]"""
    T, H, d, r, dv = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    c_q = _handed(rms(product(h, tensors, f"{name}.dq"), tensors[f"{name}.dq.norm"], eps))
    q = product(c_q, tensors, f"{name}.uq").view(T, H, d + r)
    q = torch.cat([q[:, :, :d], rotate(q[:, :, d:], m["rot"])], dim=2)
    c, shared = latent
    k = product(c, tensors, f"{name}.uk").view(T, H, d)
    k = torch.cat([k, shared[:, None, :].expand(T, H, r)], dim=2)
    v = product(c, tensors, f"{name}.uv").view(T, H, dv)
    o = causal_attention(_handed(q), k, v, m["scale"], tensors[f"{name}.sink"])
    return product(_handed(o.reshape(T, -1)), tensors, f"{name}.o")


# --------------------------------------------------------------------------- #
# The gated delta rule
# --------------------------------------------------------------------------- #

def short_convolution(u, taps):
    """y[t, c] = sum_j taps[c, j] u[t - n + 1 + j, c] for n taps; zeros before the start."""
    n = taps.shape[1]
    padded = torch.cat([torch.zeros(n - 1, u.shape[1], dtype=F), u])
    return sum(_f(taps)[:, j] * padded[j: j + u.shape[0]] for j in range(n))


def unit(x):
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + 1e-6)


def delta_memory(q, k, v, keep, beta, state=None):
    """Per head S <- keep S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q: q, k [T, H, d], v [T, H, dv],
    keep and beta [T, H]. -> (o [T, H, dv], the last S [H, d, dv]); `state` is the S to start from (zero)."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=F) if state is None else state.clone()
    out = torch.zeros(T, H, v.shape[2], dtype=F)
    for t in range(T):
        S = keep[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - (S * k[t][:, :, None]).sum(dim=1))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(dim=1)
    return out, S


def delta_mixer(h, tensors, name, m, eps):
    """-> [T, W]"""
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    mixed = lambda n: _handed(silu(short_convolution(product(h, tensors, f"{name}.{n}"), tensors[f"{name}.{n}.conv"])))
    group = [i // (H // G) for i in range(H)]
    q = unit(mixed("q").view(T, G, d))[:, group] * d ** -0.5
    k = unit(mixed("k").view(T, G, d))[:, group]
    beta = sigmoid(product(h, tensors, f"{name}.b"))
    keep = torch.exp(-torch.exp(_f(tensors[f"{name}.A_log"])) * softplus(product(h, tensors, f"{name}.a") + _f(tensors[f"{name}.dt_bias"])))
    o, _ = delta_memory(q, k, mixed("v").view(T, H, dv), keep, beta)
    o = rms(o, tensors[f"{name}.norm"], eps).reshape(T, H * dv) * silu(product(h, tensors, f"{name}.g"))
    return product(_handed(o), tensors, f"{name}.o")


# --------------------------------------------------------------------------- #
# Feed-forwards
# --------------------------------------------------------------------------- #

def gated(h, tensors, name, act):
    return product(_handed(act(product(h, tensors, f"{name}.gate")) * product(h, tensors, f"{name}.up")), tensors, f"{name}.down")


def choose(z, top):
    """The `top` largest logits of one token (the lower index first among equals) and the softmax over them alone."""
    order = sorted(range(z.numel()), key=lambda e: (-float(z[e]), e))[:top]
    weights = torch.exp(z[order] - z[order].max())
    return order, weights / weights.sum()


def mixture(h, tensors, name, router, margins=None):
    """`margins`, a list, receives by how much each token's last chosen logit beats the first one left out."""
    z = product(h, tensors, f"{name}.router") + _f(tensors[f"{name}.router.b"])
    if margins is not None and router["top"] < router["experts"]:
        ranked = z.sort(dim=1, descending=True).values
        margins.append(ranked[:, router["top"] - 1] - ranked[:, router["top"]])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in zip(*choose(z[t], router["top"])):
            out[t] += w * gated(h[t], tensors, f"{name}.e{e}", silu)
    return out


def feed_forward(h, tensors, name, mlp, margins=None):
    return gated(h, tensors, name, gelu_tanh) if mlp["kind"] == "dense" else mixture(h, tensors, name, mlp["router"], margins)


# --------------------------------------------------------------------------- #
# The model
# --------------------------------------------------------------------------- #

def side_by_side(h, tensors, name, m, eps):
    """Half the sum of the two mixers' outputs, each normed over the model's width first."""
    left = rms(attention_mixer(h, tensors, f"{name}.left", m["left"], eps), tensors[f"{name}.left.out"], eps)
    right = rms(delta_mixer(h, tensors, f"{name}.right", m["right"], eps), tensors[f"{name}.right.out"], eps)
    return 0.5 * (left + right)


def layer(x, tensors, i, entry, eps, latents, margins=None):
    """x + norm(mixer(x)), then the same with the feed-forward: the sublayers read x itself. `latents`: by
    layer, what the latent attentions so far keep."""
    name, m = f"l{i}", entry["mixer"]
    h = _handed(x)
    if entry["type"] == "parallel":
        y = side_by_side(h, tensors, f"{name}.mix", m, eps)
    else:
        source = m.get("kv_from")
        if source is None:
            latents[i] = latent_of(h, tensors, f"{name}.mix", m, eps)
        y = latent_mixer(h, tensors, f"{name}.mix", m, eps, latents[i if source is None else source])
    x = x + rms(y, tensors[f"{name}.norm1"], eps)
    if entry.get("mlp"):
        x = x + rms(feed_forward(_handed(x), tensors, f"{name}.mlp", entry["mlp"], margins), tensors[f"{name}.norm2"], eps)
    return x


def forward(config, tensors, tokens, layers_out=None, margins=None):
    """float64 logits [T, vocab]. `layers_out`, a list, receives the stream after every layer; `margins` as for `mixture`."""
    eps = config["norm"]["eps"]
    table = _f(tensors["embed"])
    x = table[torch.tensor(list(tokens))] * config["embedding"]["scale"]
    latents = {}
    for i, entry in enumerate(config["layers"]):
        x = layer(x, tensors, i, entry, eps, latents, margins)
        if layers_out is not None:
            layers_out.append(x)
    return _handed(rms(x, tensors["final.norm"], eps)) @ table.T
