"""Configuration of the Namizen decoder, read from its ``config.json``.

Namizen is a small decoder-only model: parallel attention and feed-forward from one residual (two norms), grouped-query attention inside
chunks of the sequence with a learned sink per head, a short causal convolution on q, k and v, partial rotary positions, values mixed with
those of an earlier layer, and a GELU-gated feed-forward.  ``layers`` lists every layer with its own sizes; nothing is shared between layers
but the width.  Sizes and constants all come from the file; what the design fixes (the activation, the pairing of the rotation, eps inside
the root) is in the code.
"""

from __future__ import annotations

import dataclasses
import hashlib
from dataclasses import dataclass
from typing import Any, Mapping

from glm_tpu_b200.exceptions import ConfigValidationError
from glm_tpu_b200.utils.json_utils import canonical_hash_bytes

ARCHITECTURE = "Namizen"


@dataclass(frozen=True)
class AttentionSpec:
    """Sizes and constants of one attention layer; the mechanisms are parameters, so a layer may leave out any of them."""

    heads: int
    kv_heads: int
    dim: int  # per-head size of queries and keys
    vdim: int  # per-head size of values
    scale: float
    conv: int = 1  # taps of the causal convolution on q, k and v (1 without a table: none)
    rot_dims: int = 0  # leading dimensions of every q and k head that are rotated
    rot_base: float = 10000.0
    chunk: int | None = None  # attention stays inside chunks of this many positions (None: the whole sequence)
    v_mix: bool = False

    def __post_init__(self) -> None:
        if min(self.heads, self.kv_heads, self.dim, self.vdim, self.conv) < 1 or self.heads % self.kv_heads:
            raise ConfigValidationError("attention sizes must be positive and heads a multiple of kv_heads")
        if self.rot_dims < 0 or self.rot_dims % 2 or self.rot_dims > self.dim:
            raise ConfigValidationError("rotated dimensions must be even and fit the head")
        if self.chunk is not None and self.chunk < 1:
            raise ConfigValidationError("a chunk has at least one position")

    @property
    def q_width(self) -> int:
        return self.heads * self.dim

    @property
    def k_width(self) -> int:
        return self.kv_heads * self.dim

    @property
    def v_width(self) -> int:
        return self.kv_heads * self.vdim

    @property
    def qkv_width(self) -> int:
        return self.q_width + self.k_width + self.v_width

    @property
    def out_width(self) -> int:
        return self.heads * self.vdim


@dataclass(frozen=True)
class LayerSpec:
    mixer: AttentionSpec
    ff: int = 0  # 0: no feed-forward


@dataclass(frozen=True)
class NamizenGeometry:
    vocab_size: int
    hidden_size: int
    layers: tuple[LayerSpec, ...]
    norm_eps: float
    eos_ids: tuple[int, ...] = ()

    def __post_init__(self) -> None:
        if self.vocab_size < 1 or self.hidden_size < 1 or not self.layers:
            raise ConfigValidationError("a Namizen model has a vocabulary, a width and at least one layer")
        mixing = [layer.mixer for layer in self.layers if layer.mixer.v_mix]
        if any(m.v_width != mixing[0].v_width for m in mixing):
            raise ConfigValidationError("layers that mix values need as many value channels as the first such layer")

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @property
    def first_mixing_layer(self) -> int | None:
        return next((i for i, layer in enumerate(self.layers) if layer.mixer.v_mix), None)

    @classmethod
    def from_config(cls, config: Mapping[str, Any]) -> "NamizenGeometry":
        if config.get("architecture") != ARCHITECTURE:
            raise ConfigValidationError("not a Namizen config")
        try:
            layers = []
            for entry in config["layers"]:
                if entry["type"] != "attention":
                    raise ConfigValidationError(f"layer type {entry['type']!r} is not part of Namizen")
                m = entry["mixer"]
                rot, mask, mlp = m.get("rot"), m.get("mask"), entry.get("mlp")
                if mlp is not None and mlp["kind"] != "dense":
                    raise ConfigValidationError(f"feed-forward kind {mlp['kind']!r} is not part of Namizen")
                layers.append(LayerSpec(
                    AttentionSpec(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), scale=float(m["scale"]),
                                  conv=int(m.get("conv") or 1), rot_dims=int(rot["dims"]) if rot else 0, rot_base=float(rot["base"]) if rot else 10000.0,
                                  chunk=int(mask["size"]) if mask else None, v_mix=bool(m.get("v_mix", False))),
                    ff=int(mlp["ff"]) if mlp is not None else 0))
            eos = config.get("eos_token_id", ())
            eos = (eos,) if isinstance(eos, int) else tuple(eos or ())
            return cls(vocab_size=int(config["vocab"]), hidden_size=int(config["width"]), layers=tuple(layers), norm_eps=float(config["norm"]["eps"]),
                       eos_ids=eos)
        except (KeyError, TypeError) as exc:
            raise ConfigValidationError(f"the Namizen config is incomplete: {exc}") from exc

    def to_config(self) -> dict:
        """The ``config.json`` that ``from_config`` reads back."""
        layers = []
        for layer in self.layers:
            m = layer.mixer
            mixer = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale, "conv": m.conv, "v_mix": m.v_mix}
            if m.rot_dims:
                mixer["rot"] = {"dims": m.rot_dims, "base": m.rot_base}
            if m.chunk is not None:
                mixer["mask"] = {"size": m.chunk}
            layers.append({"type": "attention", "mixer": mixer, "mlp": {"kind": "dense", "ff": layer.ff} if layer.ff else None})
        out = {"architecture": ARCHITECTURE, "vocab": self.vocab_size, "width": self.hidden_size, "norm": {"eps": self.norm_eps}, "layers": layers}
        if self.eos_ids:
            out["eos_token_id"] = list(self.eos_ids)
        return out

    def truncated(self, num_layers: int) -> "NamizenGeometry":
        if not 1 <= num_layers <= self.num_layers:
            raise ValueError("truncation must keep between 1 and num_layers layers")
        return dataclasses.replace(self, layers=self.layers[:num_layers])

    def tensor_shapes(self) -> dict[str, tuple[int, ...]]:
        """Every tensor of the checkpoint by name."""
        out: dict[str, tuple[int, ...]] = {"embed": (self.vocab_size, self.hidden_size)}
        width = self.hidden_size
        for i, layer in enumerate(self.layers):
            m, p = layer.mixer, f"l{i}"
            out[p + ".norm1"] = (width,)
            if layer.ff:
                out[p + ".norm2"] = (width,)
            for name, rows in (("q", m.q_width), ("k", m.k_width), ("v", m.v_width)):
                out[f"{p}.mix.{name}"] = (rows, width)
                out[f"{p}.mix.{name}.conv"] = (rows, m.conv)
            if m.v_mix:
                out[p + ".mix.vmix"] = ()
            out[p + ".mix.sink"] = (m.heads,)
            out[p + ".mix.o"] = (width, m.out_width)
            if layer.ff:
                out[p + ".mlp.gate"] = out[p + ".mlp.up"] = (layer.ff, width)
                out[p + ".mlp.down"] = (width, layer.ff)
        out["final.norm"] = (width,)
        out["head"] = (self.vocab_size, width)
        return out

    def as_dict(self) -> dict[str, Any]:
        return self.to_config()

    @property
    def geometry_hash(self) -> str:
        return hashlib.sha256(canonical_hash_bytes(self.as_dict())).hexdigest()


def tiny_namizen() -> NamizenGeometry:
    """CPU-sized fixture: three layers of unequal sizes, one without a feed-forward, two that mix values."""
    def attention(heads, kv_heads, dim, vdim, conv, rot_dims, base, chunk, v_mix):
        return AttentionSpec(heads, kv_heads, dim, vdim, dim**-0.5, conv, rot_dims, base, chunk, v_mix)

    return NamizenGeometry(
        vocab_size=640, hidden_size=128, norm_eps=1e-5, eos_ids=(637, 638, 639),
        layers=(LayerSpec(attention(6, 2, 32, 24, 4, 16, 10000.0, 48, False), 192),
                LayerSpec(attention(4, 2, 40, 32, 3, 40, 50000.0, 32, True), 0),
                LayerSpec(attention(8, 2, 24, 32, 2, 8, 10000.0, 64, True), 160)))


def bench_namizen(layers: int, *, width: int, heads: int, kv_heads: int, head_dim: int, ff: int, vocab: int, chunk: int) -> NamizenGeometry:
    """A model of equal layers at sizes that resemble a real model's (speed measurements)."""
    spec = LayerSpec(AttentionSpec(heads, kv_heads, head_dim, head_dim, head_dim**-0.5, 4, head_dim // 2, 500000.0, chunk, True), ff)
    return NamizenGeometry(vocab_size=vocab, hidden_size=width, layers=(spec,) * layers, norm_eps=1e-5)
