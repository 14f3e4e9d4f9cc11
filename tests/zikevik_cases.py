"""Model configurations and weights for the Zikevik tests, and helpers that compare logits."""

from __future__ import annotations

import torch

from glm_tpu_b200.config.zikevik import DeltaSpec, DenseSpec, LatentSpec, LayerSpec, RoutedSpec, ZikevikGeometry, tiny_zikevik
from glm_tpu_b200.models.zikevik.weights import random_checkpoint
from glm_tpu_b200.oracle import zikevik as oracle
from tests.namizen_cases import row_errors, tokens_for  # noqa: F401 - the same helpers for every family

MARGIN = 0.15  # of router logits: several times what bf16 activations can move them


def delta(heads, kv_heads, dim, vdim, conv=4, decay_rank=16, gate_rank=16):
    return DeltaSpec(heads, kv_heads, dim, vdim, conv, decay_rank, gate_rank)


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale=None, base=10000.0):
    return LatentSpec(heads, dim, rot_dim, vdim, q_rank, kv_rank, (dim + rot_dim) ** -0.5 if scale is None else scale, base)


def geometries() -> dict[str, ZikevikGeometry]:
    """Sizes that differ in every layer, that are not multiples of anything, and that take each kernel."""
    return {
        "tiny": tiny_zikevik(),
        # nothing is a multiple of 8; one tap and more taps than the strips hold; every expert chosen; three value heads per key head
        "odd": ZikevikGeometry(vocab_size=301, hidden_size=100, norm_eps=1e-3, embedding_scale=0.7, layers=(
            LayerSpec(delta(3, 1, 21, 13, 1, 5, 7), DenseSpec(51)), LayerSpec(latent(5, 19, 6, 11, 33, 27, scale=0.31, base=777.0), RoutedSpec(3, 3, 29)),
            LayerSpec(delta(2, 2, 36, 44, 6, 9, 3), RoutedSpec(7, 2, 20)), LayerSpec(latent(3, 30, 10, 36, 50, 90), None))),
        # tensor-core sizes: full tiles, more than one block of query heads, two value heads per key head
        "tiles": ZikevikGeometry(vocab_size=512, hidden_size=256, norm_eps=1e-6, embedding_scale=2.0, layers=(
            LayerSpec(delta(4, 2, 128, 128, 4, 64, 32), RoutedSpec(8, 3, 96)), LayerSpec(latent(40, 64, 64, 128, 128, 512, base=500000.0), DenseSpec(384)),
            LayerSpec(delta(2, 1, 64, 96, 3, 32, 16), DenseSpec(256)), LayerSpec(latent(16, 32, 32, 64, 96, 192), RoutedSpec(16, 1, 128)))),
        # key channels beyond the chunked kernels, heads beyond 128 (no tcgen05) and beyond 256 (no tensor cores), latents beyond 512
        "wide": ZikevikGeometry(vocab_size=320, hidden_size=192, norm_eps=1e-5, embedding_scale=1.0, layers=(
            LayerSpec(delta(2, 1, 200, 72, 4, 24, 24), DenseSpec(96)), LayerSpec(latent(4, 120, 48, 200, 64, 304), RoutedSpec(5, 2, 40)),
            LayerSpec(latent(2, 200, 64, 272, 80, 544), DenseSpec(64)), LayerSpec(delta(2, 2, 96, 264, 2, 8, 8), None))),
        # the smallest sizes, one expert, and layers that run again with their own caches: both mixers, both feed-forwards, one of them three times
        "again": ZikevikGeometry(vocab_size=288, hidden_size=64, norm_eps=1e-5, embedding_scale=8.0, layers=(
            LayerSpec(latent(1, 2, 2, 3, 8, 6), RoutedSpec(1, 1, 24)), LayerSpec(delta(1, 1, 8, 8, 2, 1, 1), DenseSpec(48)),
            LayerSpec(latent(1, 2, 2, 3, 8, 6), RoutedSpec(1, 1, 24), weights_of=0), LayerSpec(delta(1, 1, 8, 8, 2, 1, 1), DenseSpec(48), weights_of=1),
            LayerSpec(delta(1, 1, 8, 8, 2, 1, 1), DenseSpec(48), weights_of=3), LayerSpec(delta(6, 2, 40, 24, 3), RoutedSpec(4, 2, 32)))),
    }


def sharp_checkpoint(g: ZikevikGeometry, seed: int = 0, factor: float = 3.0) -> dict[str, torch.Tensor]:
    """Random weights under which small faults show: attention is peaked on a handful of keys, wherever they are; sinks carry weight; key
    channels forget at every speed, from hardly ever (a state that is lost moves every later token) to within a token; and the router's
    scores differ, so that the weight on an expert's input matters."""
    out = random_checkpoint(g, seed)
    gen = torch.Generator().manual_seed(seed + 1000)
    for name, t in list(out.items()):
        leaf = name.rsplit(".", 1)[-1]
        if leaf in ("uq", "router"):
            out[name] = (t.float() * factor).to(torch.bfloat16)
        elif leaf == "sink":
            out[name] = (t.float() + factor).to(torch.bfloat16)
        elif leaf == "dt_bias":
            out[name] = (-4.0 + 4.0 * torch.randn(t.shape, generator=gen)).to(torch.bfloat16)
        elif leaf == "A_log":
            out[name] = (1.0 + 0.8 * torch.randn(t.shape, generator=gen)).to(torch.bfloat16)
    return out


def expected(g: ZikevikGeometry, checkpoint: dict, tokens, **kw) -> torch.Tensor:
    return oracle.forward(g.to_config(), checkpoint, tokens, **kw)


def settled_tokens(g: ZikevikGeometry, checkpoint: dict, n: int, seed: int = 0, keep=()) -> list[int]:
    """Random tokens none of which leaves the router a close call (which rounding could decide either way); positions in ``keep`` repeat
    the token at another position: ``(position, position of the original)``."""
    gen = torch.Generator().manual_seed(seed)
    tokens = torch.randint(0, g.vocab_size, (n,), generator=gen)
    for _ in range(60):
        for at, back in keep:
            tokens[at] = tokens[back]
        margins: list = []
        expected(g, checkpoint, tokens.tolist(), dtype=torch.float32, margins_out=margins)
        close = torch.stack(margins).amin(0) < MARGIN if margins else torch.zeros(n, dtype=torch.bool)
        for at, back in keep:
            close[back] |= close[at]
        if not close.any():
            return tokens.tolist()
        tokens[close] = torch.randint(0, g.vocab_size, (int(close.sum()),), generator=gen)
    raise AssertionError("no tokens without a close call found")
