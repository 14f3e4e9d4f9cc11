"""Plain CPU statement of the Zikevik decoder: whole sequences, no cache, one function per mechanism.

Everything is written from the equations of the model with ordinary tensor operations (float64 by default) and shares no code with the
engine: neither its configuration classes nor its loader nor its kernels.  ``config`` is the parsed ``config.json`` and ``tensors`` the
checkpoint's ``name -> tensor`` mapping.  The engine's CPU backend and the tests compare against it.

A layer computes ``x <- x + mixer(norm1(x))`` and then, if it has a feed-forward, ``x <- x + ff(norm2(x))``.  There are two mixers, a gated
delta rule whose decay is per key channel and attention over a shared latent, and two feed-forwards, dense and routed.
"""

from __future__ import annotations

import torch


def rms_norm(x: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * weight


def zero_centred_norm(x: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    """The weight is stored around zero."""
    return rms_norm(x, 1.0 + weight, eps)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.maximum(z, torch.zeros_like(z)) + torch.log1p(torch.exp(-z.abs()))


# ------------------------------------------------------------------------------------------------ gated delta rule
def causal_conv(u: torch.Tensor, weight: torch.Tensor) -> torch.Tensor:
    """``u [T, channels]``, ``weight [channels, taps]``: the last tap weighs the current token, zeros stand before the start."""
    taps, total = weight.shape[1], u.shape[0]
    padded = torch.cat([torch.zeros(taps - 1, u.shape[1], dtype=u.dtype), u], dim=0)
    return sum(weight[:, j] * padded[j : j + total] for j in range(taps))


def unit(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + 1e-6)


def channel_decay(h: torch.Tensor, a1: torch.Tensor, a2: torch.Tensor, dt_bias: torch.Tensor, a_log: torch.Tensor, heads: int, dim: int) -> torch.Tensor:
    """``[T, heads, dim]``: what is left of the state's row of every key channel after a token."""
    step = softplus((h @ a1.T) @ a2.T + dt_bias).reshape(-1, heads, dim)
    return torch.exp(-torch.exp(a_log)[:, None] * step)


def delta_rule(q, k, v, beta, decay, state=None):
    """``q, k, decay [T, heads, dim]``, ``v [T, heads, vdim]``, ``beta [T, heads]``; ``state [heads, dim, vdim]`` (``None``: zeros).
    Per token: decay the state, write the error of what it recalls for ``k``, read with ``q``.  Returns ``([T, heads, vdim], state)``."""
    total, heads, dim = q.shape
    S = torch.zeros(heads, dim, v.shape[-1], dtype=v.dtype) if state is None else state.clone()
    out = torch.empty_like(v)
    for t in range(total):
        S = decay[t][..., None] * S
        recalled = torch.einsum("hd,hdv->hv", k[t], S)
        write = beta[t][:, None] * (v[t] - recalled)
        S = S + k[t][..., None] * write[:, None, :]
        out[t] = torch.einsum("hd,hdv->hv", q[t], S)
    return out, S


def channel_delta(h: torch.Tensor, mixer: dict, weight, eps: float) -> torch.Tensor:
    """``weight(name)`` gives the mixer's tensors."""
    heads, groups, dim, vdim = mixer["heads"], mixer["kv_heads"], mixer["dim"], mixer["vdim"]
    total = h.shape[0]
    q, k, v = (silu(causal_conv(h @ weight(n).T, weight(n + ".conv"))) for n in ("q", "k", "v"))
    per = heads // groups
    q, k = (unit(x.reshape(total, groups, dim)).repeat_interleave(per, dim=1) for x in (q, k))
    beta = torch.sigmoid(h @ weight("b").T)
    decay = channel_decay(h, weight("a1"), weight("a2"), weight("dt_bias"), weight("A_log"), heads, dim)
    o, _ = delta_rule(q * dim**-0.5, k, v.reshape(total, heads, vdim), beta, decay)
    gate = torch.sigmoid((h @ weight("g1").T) @ weight("g2").T).reshape(total, heads, vdim)
    return (rms_norm(o, weight("norm"), eps) * gate).reshape(total, heads * vdim) @ weight("o").T


# ------------------------------------------------------------------------------------------------ latent attention
def rotate_pairs(x: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """``x [T, heads, dim]``: the first ``dims`` dimensions of every head turn by ``position * base**(-2i/dims)``, pair ``(2i, 2i + 1)``."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    angle = torch.arange(x.shape[0], dtype=torch.float64)[:, None] * float(base) ** (-2.0 * i / dims)
    cos, sin = angle.cos().to(x.dtype)[:, None, :], angle.sin().to(x.dtype)[:, None, :]
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    turned = torch.stack([u * cos - v * sin, v * cos + u * sin], dim=-1).flatten(-2)
    return torch.cat([turned, x[..., dims:]], dim=-1)


def sink_softmax(scores: torch.Tensor, sink: torch.Tensor, visible: torch.Tensor) -> torch.Tensor:
    """``scores [heads, T, T]``, ``sink [heads]``: weights of the visible keys; the sink takes its share and has no value."""
    scores = scores.masked_fill(~visible, float("-inf"))
    top = torch.maximum(scores.amax(dim=-1), sink[:, None])
    e = torch.exp(scores - top[..., None])
    return e / (e.sum(dim=-1) + torch.exp(sink[:, None] - top))[..., None]


def latent_attention(h: torch.Tensor, mixer: dict, weight, eps: float) -> torch.Tensor:
    heads, dim, rot_dim, vdim, rank = mixer["heads"], mixer["dim"], mixer["rot_dim"], mixer["vdim"], mixer["kv_rank"]
    total = h.shape[0]
    q = (rms_norm(h @ weight("dq").T, weight("dq.norm"), eps) @ weight("uq").T).reshape(total, heads, dim + rot_dim)
    joint = h @ weight("dkv").T
    latent = rms_norm(joint[:, :rank], weight("dkv.norm"), eps)
    rot = mixer["rot"]
    q_rot = rotate_pairs(q[..., dim:], rot["dims"], rot["base"])
    k_rot = rotate_pairs(joint[:, None, rank:], rot["dims"], rot["base"])[:, 0]
    k = (latent @ weight("uk").T).reshape(total, heads, dim)
    v = (latent @ weight("uv").T).reshape(total, heads, vdim)
    scores = (torch.einsum("ihd,jhd->hij", q[..., :dim], k) + torch.einsum("ihd,jd->hij", q_rot, k_rot)) * mixer["scale"]
    p = sink_softmax(scores, weight("sink"), torch.ones(total, total, dtype=torch.bool).tril())
    out = torch.einsum("hij,jhd->ihd", p, v) * torch.sigmoid(h @ weight("g").T)[..., None]
    return out.reshape(total, heads * vdim) @ weight("o").T


# ------------------------------------------------------------------------------------------------ feed-forward
def gated_ff(h: torch.Tensor, weight, prefix: str = "") -> torch.Tensor:
    return (silu(h @ weight(prefix + "gate").T) * (h @ weight(prefix + "up").T)) @ weight(prefix + "down").T


def router_margin(h: torch.Tensor, router: dict, weight) -> torch.Tensor:
    """``[T]``: how far the last expert that is chosen lies above the first that is not (in router logits; infinite if all are chosen)."""
    best = (h @ weight("router").T).sort(dim=-1, descending=True).values
    top = router["top"]
    return best[:, top - 1] - best[:, top] if top < router["experts"] else torch.full((h.shape[0],), float("inf"), dtype=h.dtype)


def routed_experts(h: torch.Tensor, router: dict, weight) -> torch.Tensor:
    """Sigmoid scores; the best ``top`` experts each take the token scaled by its own score, and their outputs are added."""
    scores = torch.sigmoid(h @ weight("router").T)
    value, chosen = scores.topk(router["top"], dim=-1)
    out = torch.zeros_like(h)
    for e in range(router["experts"]):
        rows, slot = (chosen == e).nonzero(as_tuple=True)
        if len(rows):
            out = out.index_add(0, rows, gated_ff(value[rows, slot][:, None] * h[rows], weight, f"e{e}."))
    return out


# ------------------------------------------------------------------------------------------------ the model
MIXERS = {"channel_delta": channel_delta, "latent_attention": latent_attention}


def forward(config: dict, tensors: dict, tokens, *, dtype=torch.float64, layers_out: list | None = None, margins_out: list | None = None) -> torch.Tensor:
    """Logits ``[T, vocab]`` of a sequence; ``layers_out`` collects the residual after every layer, ``margins_out`` the ``router_margin`` of every
    routed layer."""
    get = lambda name: tensors[name].to(dtype)  # noqa: E731
    eps = config["norm"]["eps"]
    x = get("embed")[torch.as_tensor(list(tokens), dtype=torch.long)] * config["embedding"]["scale"]
    for i, layer in enumerate(config["layers"]):
        j = i
        while config["layers"][j].get("weights_of") is not None:
            j = config["layers"][j]["weights_of"]
        x = x + MIXERS[layer["type"]](zero_centred_norm(x, get(f"l{j}.norm1"), eps), layer["mixer"], lambda n, j=j: get(f"l{j}.mix.{n}"), eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            h, weight = zero_centred_norm(x, get(f"l{j}.norm2"), eps), lambda n, j=j: get(f"l{j}.mlp.{n}")
            if margins_out is not None and mlp["kind"] != "dense":
                margins_out.append(router_margin(h, mlp["router"], weight))
            x = x + (gated_ff(h, weight) if mlp["kind"] == "dense" else routed_experts(h, mlp["router"], weight))
        if layers_out is not None:
            layers_out.append(x.clone())
    return zero_centred_norm(x, get("final.norm"), eps) @ get("head").T
