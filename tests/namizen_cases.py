"""Model configurations and weights for the Namizen tests, and helpers that compare logits."""

from __future__ import annotations

import torch

from glm_tpu_b200.config.namizen import AttentionSpec, LayerSpec, NamizenGeometry, tiny_namizen
from glm_tpu_b200.models.namizen.weights import random_checkpoint
from glm_tpu_b200.oracle import namizen as oracle


def attention(heads, kv_heads, dim, vdim, conv, rot_dims, base, chunk, v_mix=False, scale=None):
    return AttentionSpec(heads, kv_heads, dim, vdim, dim**-0.5 if scale is None else scale, conv, rot_dims, base, chunk, v_mix)


def geometries() -> dict[str, NamizenGeometry]:
    """Sizes that differ in every layer, that are not multiples of anything, and that take each kernel."""
    return {
        "tiny": tiny_namizen(),
        # nothing is a multiple of 8; one tap, no rotation, equal query and key heads; a layer over the whole sequence
        "odd": NamizenGeometry(vocab_size=301, hidden_size=100, norm_eps=1e-3, layers=(
            LayerSpec(attention(3, 3, 21, 13, 1, 0, 10000.0, 7, True), 51),
            LayerSpec(attention(5, 1, 36, 44, 5, 36, 777.0, None, False, scale=0.3), 0),
            LayerSpec(attention(6, 3, 30, 13, 3, 10, 10000.0, 19, True), 70))),
        # tensor-core sizes: full tiles of 64 columns, eight query heads per key head, chunks around the tile sizes
        "tiles": NamizenGeometry(vocab_size=512, hidden_size=256, norm_eps=1e-6, layers=(
            LayerSpec(attention(8, 1, 128, 128, 4, 64, 500000.0, 96, True), 384),
            LayerSpec(attention(4, 2, 64, 64, 4, 32, 10000.0, 130, True), 320),
            LayerSpec(attention(20, 1, 48, 64, 2, 48, 10000.0, 64, False), 128))),
        # heads beyond 128 (no tcgen05) and beyond 256 (no tensor cores)
        "wide": NamizenGeometry(vocab_size=320, hidden_size=192, norm_eps=1e-5, layers=(
            LayerSpec(attention(4, 2, 160, 200, 3, 80, 10000.0, 40, True), 96),
            LayerSpec(attention(2, 1, 264, 272, 4, 128, 10000.0, 33, False), 64),
            LayerSpec(attention(2, 2, 256, 200, 3, 100, 10000.0, 50, True), 64))),
        # chunks of one and two tokens, and one that no sequence of the tests leaves
        "edges": NamizenGeometry(vocab_size=288, hidden_size=64, norm_eps=1e-5, layers=(
            LayerSpec(attention(2, 1, 32, 32, 4, 32, 10000.0, 1, False), 96),
            LayerSpec(attention(4, 2, 32, 16, 2, 16, 100.0, 2, True), 64),
            LayerSpec(attention(2, 2, 16, 16, 6, 16, 10000.0, 100000, True), 64))),
    }


def sharp_checkpoint(g: NamizenGeometry, seed: int = 0, factor: float = 3.0) -> dict[str, torch.Tensor]:
    """Random weights whose attention is peaked: a handful of keys per query carry the weight, wherever they are in the chunk, so a key
    that is missing, one too many, or a sink that is left out moves the logits visibly."""
    out = random_checkpoint(g, seed)
    for i in range(g.num_layers):
        out[f"l{i}.mix.q"] = (out[f"l{i}.mix.q"].float() * factor).to(torch.bfloat16)
        out[f"l{i}.mix.sink"] = (out[f"l{i}.mix.sink"].float() + factor).to(torch.bfloat16)
    return out


def tokens_for(g: NamizenGeometry, n: int, seed: int = 0) -> list[int]:
    return torch.randint(0, g.vocab_size, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def expected(g: NamizenGeometry, checkpoint: dict, tokens, **kw) -> torch.Tensor:
    return oracle.forward(g.to_config(), checkpoint, tokens, **kw)


def row_errors(got: torch.Tensor, want: torch.Tensor) -> torch.Tensor:
    """Per row: root mean square of the difference (mean taken off) over the root mean square of the expected logits."""
    got, want = got.double(), want.double()
    d = got - want
    d = d - d.mean(dim=-1, keepdim=True)
    return d.square().mean(dim=-1).sqrt() / want.std(dim=-1).clamp_min(1e-6)
