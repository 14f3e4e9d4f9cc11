"""Configuration of the Zikevik decoder, read from its ``config.json``.

Zikevik is a small decoder-only model whose layers are of two kinds, in any order: a gated delta rule with one decay per head and key channel
(a recurrent state per head, nothing per token), and attention over a shared low-rank latent (one latent and one rotated key part per
token, a sink and an output gate per head).  A layer may be followed by a dense or a routed feed-forward, or none, and may use the weights of
an earlier layer.  Norm weights are stored around zero and the embedding is scaled.  Every size and constant comes from the file; the two ranks
it does not name (of the decay's and the gate's projections) come from the tensors' shapes.  What the design fixes is in the code.
"""

from __future__ import annotations

import dataclasses
import hashlib
from dataclasses import dataclass
from typing import Any, Mapping

from glm_tpu_b200.exceptions import ConfigValidationError
from glm_tpu_b200.utils.json_utils import canonical_hash_bytes

ARCHITECTURE = "Zikevik"


@dataclass(frozen=True)
class DeltaSpec:
    """A gated delta rule: ``kv_heads`` query and key heads of ``dim`` channels, ``heads`` value heads of ``vdim``."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int  # taps of the causal convolution on q, k and v
    decay_rank: int
    gate_rank: int
    kind = "channel_delta"

    def __post_init__(self) -> None:
        if min(self.heads, self.kv_heads, self.dim, self.vdim, self.conv, self.decay_rank, self.gate_rank) < 1 or self.heads % self.kv_heads:
            raise ConfigValidationError("delta-rule sizes must be positive and heads a multiple of kv_heads")

    @property
    def k_width(self) -> int:
        return self.kv_heads * self.dim

    @property
    def v_width(self) -> int:
        return self.heads * self.vdim

    @property
    def conv_width(self) -> int:
        return 2 * self.k_width + self.v_width

    @property
    def out_width(self) -> int:
        return self.v_width

    def tensors(self, width: int) -> dict[str, tuple[int, ...]]:
        out: dict[str, tuple[int, ...]] = {}
        for name, rows in (("q", self.k_width), ("k", self.k_width), ("v", self.v_width)):
            out[name], out[name + ".conv"] = (rows, width), (rows, self.conv)
        out |= {"b": (self.heads, width), "A_log": (self.heads,), "norm": (self.vdim,), "a1": (self.decay_rank, width),
                "a2": (self.heads * self.dim, self.decay_rank), "dt_bias": (self.heads * self.dim,), "g1": (self.gate_rank, width),
                "g2": (self.v_width, self.gate_rank), "o": (width, self.v_width)}
        return out

    def to_config(self) -> dict:
        return dataclasses.asdict(self)


@dataclass(frozen=True)
class LatentSpec:
    """Attention whose keys and values are projections of one normalized latent per token, beside one rotated key part all heads share."""

    heads: int
    dim: int  # unrotated query / key dimensions per head
    rot_dim: int  # rotated ones
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot_base: float
    kind = "latent_attention"

    def __post_init__(self) -> None:
        if min(self.heads, self.dim, self.rot_dim, self.vdim, self.q_rank, self.kv_rank) < 1:
            raise ConfigValidationError("latent attention sizes must be positive")
        if self.rot_dim % 2:
            raise ConfigValidationError("the rotated part has an even number of dimensions")

    @property
    def out_width(self) -> int:
        return self.heads * self.vdim

    def tensors(self, width: int) -> dict[str, tuple[int, ...]]:
        return {"dq": (self.q_rank, width), "dq.norm": (self.q_rank,), "uq": (self.heads * (self.dim + self.rot_dim), self.q_rank),
                "dkv": (self.kv_rank + self.rot_dim, width), "dkv.norm": (self.kv_rank,), "uk": (self.heads * self.dim, self.kv_rank),
                "uv": (self.heads * self.vdim, self.kv_rank), "sink": (self.heads,), "g": (self.heads, width), "o": (width, self.out_width)}

    def to_config(self) -> dict:
        out = {name: value for name, value in dataclasses.asdict(self).items() if name != "rot_base"}
        return out | {"rot": {"base": self.rot_base, "dims": self.rot_dim}}


@dataclass(frozen=True)
class DenseSpec:
    ff: int
    kind = "dense"

    def __post_init__(self) -> None:
        if self.ff < 1:
            raise ConfigValidationError("a feed-forward has at least one channel")

    def tensors(self, width: int) -> dict[str, tuple[int, ...]]:
        return {"gate": (self.ff, width), "up": (self.ff, width), "down": (width, self.ff)}

    def to_config(self) -> dict:
        return {"kind": self.kind, "ff": self.ff}


@dataclass(frozen=True)
class RoutedSpec:
    experts: int
    top: int
    ff: int
    kind = "moe"

    def __post_init__(self) -> None:
        if self.ff < 1 or not 1 <= self.top <= self.experts:
            raise ConfigValidationError("a routed feed-forward chooses between one expert and all of them")

    def tensors(self, width: int) -> dict[str, tuple[int, ...]]:
        out = {f"e{e}.{name}": shape for e in range(self.experts) for name, shape in DenseSpec(self.ff).tensors(width).items()}
        return out | {"router": (self.experts, width)}

    def to_config(self) -> dict:
        return {"kind": self.kind, "expert": {"ff": self.ff}, "router": {"experts": self.experts, "top": self.top}}


@dataclass(frozen=True)
class LayerSpec:
    mixer: DeltaSpec | LatentSpec
    mlp: DenseSpec | RoutedSpec | None = None
    weights_of: int | None = None  # the layer whose tensors this one uses (its cache or state is its own)


def _mixer(kind: str, m: Mapping, name: str, shapes: Mapping | None):
    if kind == DeltaSpec.kind:
        ranks = {}
        for key, tensor in (("decay_rank", "a1"), ("gate_rank", "g1")):
            shape = (shapes or {}).get(f"{name}.mix.{tensor}")
            if key not in m and shape is None:
                raise ConfigValidationError(f"neither the config nor a tensor gives the {key} of {name}")
            ranks[key] = int(m[key] if key in m else shape[0])
        return DeltaSpec(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), conv=int(m["conv"]), **ranks)
    if kind == LatentSpec.kind:
        if int(m["rot"]["dims"]) != int(m["rot_dim"]):
            raise ConfigValidationError("the rotation covers the rotated part of a head, no more and no less")
        return LatentSpec(heads=int(m["heads"]), dim=int(m["dim"]), rot_dim=int(m["rot_dim"]), vdim=int(m["vdim"]), q_rank=int(m["q_rank"]),
                          kv_rank=int(m["kv_rank"]), scale=float(m["scale"]), rot_base=float(m["rot"]["base"]))
    raise ConfigValidationError(f"layer type {kind!r} is not part of {ARCHITECTURE}")


def _mlp(m: Mapping | None):
    if m is None:
        return None
    if m["kind"] == DenseSpec.kind:
        return DenseSpec(int(m["ff"]))
    if m["kind"] == RoutedSpec.kind:
        return RoutedSpec(experts=int(m["router"]["experts"]), top=int(m["router"]["top"]), ff=int(m["expert"]["ff"]))
    raise ConfigValidationError(f"feed-forward kind {m['kind']!r} is not part of {ARCHITECTURE}")


@dataclass(frozen=True)
class ZikevikGeometry:
    vocab_size: int
    hidden_size: int
    layers: tuple[LayerSpec, ...]
    norm_eps: float
    embedding_scale: float = 1.0
    eos_ids: tuple[int, ...] = ()

    def __post_init__(self) -> None:
        if self.vocab_size < 1 or self.hidden_size < 1 or not self.layers:
            raise ConfigValidationError(f"a {ARCHITECTURE} model has a vocabulary, a width and at least one layer")
        for i, layer in enumerate(self.layers):
            owner = self.owner(i)
            if (layer.mixer, layer.mlp) != (self.layers[owner].mixer, self.layers[owner].mlp):
                raise ConfigValidationError(f"layer {i} uses the weights of layer {owner} but differs from it")

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    def owner(self, layer: int) -> int:
        """The layer whose tensors ``layer`` uses (itself, unless it says otherwise)."""
        seen = set()
        while self.layers[layer].weights_of is not None:
            seen.add(layer)
            layer = self.layers[layer].weights_of
            if layer in seen or not 0 <= layer < len(self.layers):
                raise ConfigValidationError("the layers' weights_of do not end at a layer that has weights")
        return layer

    @classmethod
    def from_config(cls, config: Mapping[str, Any], shapes: Mapping | None = None) -> "ZikevikGeometry":
        """``shapes``: tensor name -> shape, for the sizes that only the tensors give."""
        if config.get("architecture") != ARCHITECTURE:
            raise ConfigValidationError(f"not a {ARCHITECTURE} config")
        try:
            layers = []
            for i, entry in enumerate(config["layers"]):
                j, hops = i, 0
                while config["layers"][j].get("weights_of") is not None and hops <= len(config["layers"]):
                    j, hops = int(config["layers"][j]["weights_of"]), hops + 1
                of = entry.get("weights_of")
                layers.append(LayerSpec(_mixer(entry["type"], entry["mixer"], f"l{j}", shapes), _mlp(entry.get("mlp")), None if of is None else int(of)))
            eos = config.get("eos_token_id", ())
            eos = (eos,) if isinstance(eos, int) else tuple(eos or ())
            return cls(vocab_size=int(config["vocab"]), hidden_size=int(config["width"]), layers=tuple(layers), norm_eps=float(config["norm"]["eps"]),
                       embedding_scale=float(config["embedding"]["scale"]), eos_ids=eos)
        except (KeyError, TypeError, IndexError) as exc:
            raise ConfigValidationError(f"the {ARCHITECTURE} config is incomplete: {exc}") from exc

    def to_config(self) -> dict:
        """The ``config.json`` that ``from_config`` reads back (with the ranks written out)."""
        layers = []
        for layer in self.layers:
            entry = {"type": layer.mixer.kind, "mixer": layer.mixer.to_config(), "mlp": layer.mlp.to_config() if layer.mlp else None}
            if layer.weights_of is not None:
                entry["weights_of"] = layer.weights_of
            layers.append(entry)
        out = {"architecture": ARCHITECTURE, "vocab": self.vocab_size, "width": self.hidden_size, "norm": {"eps": self.norm_eps},
               "embedding": {"scale": self.embedding_scale}, "layers": layers}
        if self.eos_ids:
            out["eos_token_id"] = list(self.eos_ids)
        return out

    def truncated(self, num_layers: int) -> "ZikevikGeometry":
        if not 1 <= num_layers <= self.num_layers:
            raise ValueError("truncation must keep between 1 and num_layers layers")
        return dataclasses.replace(self, layers=self.layers[:num_layers])

    def tensor_shapes(self) -> dict[str, tuple[int, ...]]:
        """Every tensor of the checkpoint by name."""
        width = self.hidden_size
        out: dict[str, tuple[int, ...]] = {"embed": (self.vocab_size, width)}
        for i, layer in enumerate(self.layers):
            if self.owner(i) != i:
                continue
            out[f"l{i}.norm1"] = (width,)
            out |= {f"l{i}.mix.{name}": shape for name, shape in layer.mixer.tensors(width).items()}
            if layer.mlp is not None:
                out[f"l{i}.norm2"] = (width,)
                out |= {f"l{i}.mlp.{name}": shape for name, shape in layer.mlp.tensors(width).items()}
        out["final.norm"] = (width,)
        out["head"] = (self.vocab_size, width)
        return out

    def as_dict(self) -> dict[str, Any]:
        return self.to_config()

    @property
    def geometry_hash(self) -> str:
        return hashlib.sha256(canonical_hash_bytes(self.as_dict())).hexdigest()


def tiny_zikevik() -> ZikevikGeometry:
    """CPU-sized fixture: both mixers, both feed-forwards and none, unequal sizes, a layer that runs twice."""
    delta = DeltaSpec(heads=4, kv_heads=2, dim=24, vdim=40, conv=4, decay_rank=16, gate_rank=12)
    latent = LatentSpec(heads=6, dim=24, rot_dim=12, vdim=20, q_rank=48, kv_rank=56, scale=36**-0.5, rot_base=10000.0)
    return ZikevikGeometry(
        vocab_size=640, hidden_size=128, norm_eps=1e-5, embedding_scale=3.0, eos_ids=(637, 638, 639),
        layers=(LayerSpec(delta, DenseSpec(160)), LayerSpec(latent, RoutedSpec(6, 2, 64)), LayerSpec(delta, None), LayerSpec(latent, DenseSpec(96)),
                LayerSpec(delta, DenseSpec(160), weights_of=0)))


def bench_zikevik(layers: int, *, width: int, heads: int, head_dim: int, ff: int, vocab: int, q_rank: int = 1536, kv_rank: int = 512, kinds=None,
                  routed: RoutedSpec | None = None) -> ZikevikGeometry:
    """Sizes that resemble a real model's layers (speed measurements): every third layer attends unless ``kinds`` says otherwise."""
    half = head_dim // 2
    delta = DeltaSpec(heads, heads, head_dim, head_dim, 4, head_dim, head_dim)
    latent = LatentSpec(heads, half, half, head_dim, q_rank, kv_rank, head_dim**-0.5, 500000.0)
    kinds = kinds or [LatentSpec.kind if i % 3 == 2 else DeltaSpec.kind for i in range(layers)]
    mlp = routed or DenseSpec(ff)
    return ZikevikGeometry(vocab_size=vocab, hidden_size=width, norm_eps=1e-5, embedding_scale=1.0,
                           layers=tuple(LayerSpec(latent if kind == LatentSpec.kind else delta, mlp) for kind in kinds))
