"""Plain CPU statement of the Namizen decoder: whole sequences, no cache, one function per mechanism.

Everything is written from the equations of the model with ordinary tensor operations (float64 by default) and shares no code with the
engine: neither its configuration classes nor its loader nor its kernels.  ``config`` is the parsed ``config.json`` and ``tensors`` the
checkpoint's ``name -> tensor`` mapping.  The engine's CPU backend and the tests compare against it.

A layer computes, from one residual ``x`` of its input,

    x <- x + attention(norm1(x)) + feed_forward(norm2(x)).

The attention sees, from position ``i``, the keys ``j <= i`` of the same chunk (``i // size == j // size``, chunks counted from position
0) and a per-head sink that only enlarges the softmax denominator.
"""

from __future__ import annotations

import math

import torch


def rms_norm(x: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * weight


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z**3)))


def causal_conv(u: torch.Tensor, weight: torch.Tensor) -> torch.Tensor:
    """``u [T, channels]``, ``weight [channels, taps]``: the last tap weighs the current token, zeros stand before the start."""
    taps, total = weight.shape[1], u.shape[0]
    padded = torch.cat([torch.zeros(taps - 1, u.shape[1], dtype=u.dtype), u], dim=0)
    return sum(weight[:, j] * padded[j : j + total] for j in range(taps))


def rotate_half(x: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """``x [T, heads, dim]``: the first ``dims`` dimensions of every head turn by ``position * base**(-2i/dims)``, pair ``(i, i + dims/2)``."""
    half = dims // 2
    i = torch.arange(half, dtype=torch.float64)
    angle = torch.arange(x.shape[0], dtype=torch.float64)[:, None] * float(base) ** (-2.0 * i / dims)
    cos, sin = angle.cos().to(x.dtype)[:, None, :], angle.sin().to(x.dtype)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., dims:]], dim=-1)


def chunk_mask(total: int, size: int) -> torch.Tensor:
    """``[T, T]`` bool: may query ``i`` (row) see key ``j`` (column)?"""
    at = torch.arange(total)
    return (at[None, :] <= at[:, None]) & (at[None, :] // size == at[:, None] // size)


def sink_softmax(scores: torch.Tensor, sink: torch.Tensor, visible: torch.Tensor) -> torch.Tensor:
    """``scores [heads, T, T]``, ``sink [heads]``: weights of the visible keys; the sink takes its share and has no value."""
    scores = scores.masked_fill(~visible, float("-inf"))
    top = torch.maximum(scores.amax(dim=-1), sink[:, None])
    e = torch.exp(scores - top[..., None])
    return e / (e.sum(dim=-1) + torch.exp(sink[:, None] - top))[..., None]


def mix_values(v: torch.Tensor, first: torch.Tensor, amount: torch.Tensor) -> torch.Tensor:
    return (1.0 - amount) * v + amount * first


def attention(h: torch.Tensor, mixer: dict, weight, first_values: torch.Tensor | None):
    """``(output [T, width], values before mixing)``; ``weight(name)`` gives the mixer's tensors; ``first_values``: what the layer mixes
    its values with (``None``: nothing)."""
    heads, groups, dim, vdim = mixer["heads"], mixer["kv_heads"], mixer["dim"], mixer["vdim"]
    total = h.shape[0]
    q, k, v = (causal_conv(h @ weight(n).T, weight(n + ".conv")) for n in ("q", "k", "v"))
    q, k = q.reshape(total, heads, dim), k.reshape(total, groups, dim)
    if mixer.get("rot"):
        q, k = (rotate_half(x, mixer["rot"]["dims"], mixer["rot"]["base"]) for x in (q, k))
    v = own = v.reshape(total, groups, vdim)
    if first_values is not None:
        v = mix_values(v, first_values.reshape(total, groups, vdim), weight("vmix"))  # channel by channel, whatever the heads
    per = heads // groups
    k, v = k.repeat_interleave(per, dim=1), v.repeat_interleave(per, dim=1)
    scores = torch.einsum("ihd,jhd->hij", q, k) * mixer["scale"]
    p = sink_softmax(scores, weight("sink"), chunk_mask(total, mixer["mask"]["size"] if mixer.get("mask") else total))
    out = torch.einsum("hij,jhd->ihd", p, v).reshape(total, heads * vdim)
    return out @ weight("o").T, own


def feed_forward(h: torch.Tensor, weight) -> torch.Tensor:
    return (gelu_tanh(h @ weight("gate").T) * (h @ weight("up").T)) @ weight("down").T


def forward(config: dict, tensors: dict, tokens, *, dtype=torch.float64, layers_out: list | None = None) -> torch.Tensor:
    """Logits ``[T, vocab]`` of a sequence; ``layers_out`` collects the residual after every layer."""
    get = lambda name: tensors[name].to(dtype)  # noqa: E731
    eps = config["norm"]["eps"]
    x = get("embed")[torch.as_tensor(list(tokens), dtype=torch.long)]
    first = None
    for i, layer in enumerate(config["layers"]):
        mixes = bool(layer["mixer"].get("v_mix"))
        update, own = attention(rms_norm(x, get(f"l{i}.norm1"), eps), layer["mixer"], lambda n, i=i: get(f"l{i}.mix.{n}"), first if mixes else None)
        if mixes and first is None:
            first = own
        if layer.get("mlp") is not None:
            update = update + feed_forward(rms_norm(x, get(f"l{i}.norm2"), eps), lambda n, i=i: get(f"l{i}.mlp.{n}"))
        x = x + update
        if layers_out is not None:
            layers_out.append(x.clone())
    return rms_norm(x, get("final.norm"), eps) @ get("head").T
