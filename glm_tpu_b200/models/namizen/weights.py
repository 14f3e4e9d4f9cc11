"""Namizen weights: the checkpoint mapping, random fixtures, and the tables one GPU keeps.

The checkpoint is a flat ``name -> tensor`` mapping (``NamizenGeometry.tensor_shapes``), e.g. ``model_loader.directory.SourceTensors``.

Resident tables are laid out for the kernels: every row is padded to a multiple of 8 columns (zeros), so any width, head size or
feed-forward size meets the alignment of the tensor-core and streaming kernels; q, k and v are one table, gate and up are one table, and the
two output projections of a parallel layer lie side by side in one table ``[width, attention | feed-forward]`` -- the sum of the two
branches is then the sum over the columns of one product.  Tables are bf16 for serving and fp32 for the 32-bit path.
"""

from __future__ import annotations

from collections.abc import Mapping
from dataclasses import dataclass

import torch

from glm_tpu_b200.config.namizen import NamizenGeometry
from glm_tpu_b200.exceptions import CheckpointValidationError
from glm_tpu_b200.model_loader.directory import pad8, padded


def check_tensors(g: NamizenGeometry, tensors: Mapping, shape_of=None) -> None:
    """Every tensor of the geometry is there with its shape (a one-tap convolution and an unused mixing amount may be left out)."""
    first = g.first_mixing_layer
    optional = {f"l{first}.mix.vmix"} | {f"l{i}.mix.{n}.conv" for i, layer in enumerate(g.layers) if layer.mixer.conv == 1 for n in "qkv"}
    missing = [name for name in g.tensor_shapes() if name not in tensors and name not in optional]
    if missing:
        raise CheckpointValidationError(f"the checkpoint misses {len(missing)} tensors, e.g. {missing[0]!r}")
    if shape_of is not None:
        for name, shape in g.tensor_shapes().items():
            if name in tensors and tuple(shape_of(name)) != shape:
                raise CheckpointValidationError(f"{name!r} has shape {tuple(shape_of(name))}, the configuration says {shape}")


def random_checkpoint(g: NamizenGeometry, seed: int = 0) -> dict[str, torch.Tensor]:
    """Random bf16 weights on the CPU (fixtures): projections ``N(0, 1/fan_in)``, norms around one, sinks and mixing amounts spread."""
    gen = torch.Generator().manual_seed(seed)
    out: dict[str, torch.Tensor] = {}
    for name, shape in g.tensor_shapes().items():
        z = torch.randn(shape, generator=gen)
        if name.endswith("norm1") or name.endswith("norm2") or name == "final.norm":
            z = 1.0 + 0.1 * z
        elif name.endswith(".conv"):
            z = z * 0.4
            z[:, -1] += 0.8
        elif name.endswith(".vmix"):
            z = 0.4 + 0.1 * z
        elif name.endswith(".sink"):
            z = 0.5 + z
        elif name != "embed":
            z = z * shape[-1] ** -0.5
        out[name] = z.to(torch.bfloat16)
    return out


@dataclass
class NamizenLayer:
    norm1: torch.Tensor
    norm2: torch.Tensor | None
    qkv: torch.Tensor  # [pad8(q | k | v), width']
    conv: torch.Tensor  # [taps, q | k | v] fp32
    gate_up: torch.Tensor | None  # [2 ff', width']: gate rows, then up rows
    out: torch.Tensor  # [width', heads * vdim' + ff']
    sink: torch.Tensor  # [heads] fp32
    mix: float  # how much of the first mixing layer's values this layer takes
    attn_cols: int  # columns of `out` that belong to the attention
    ff_cols: int


@dataclass
class NamizenWeights:
    geometry: NamizenGeometry
    dtype: torch.dtype
    embed: torch.Tensor  # [vocab, width']
    layers: list[NamizenLayer]
    final_norm: torch.Tensor
    head: torch.Tensor  # [vocab', width']
    bytes_resident: int = 0

    def __post_init__(self) -> None:
        tables = [self.embed, self.final_norm, self.head]
        for layer in self.layers:
            tables += [value for value in vars(layer).values() if isinstance(value, torch.Tensor)]
        self.bytes_resident = sum(t.numel() * t.element_size() for t in tables)


def resident_weights(g: NamizenGeometry, tensors: Mapping, device, dtype: torch.dtype = torch.bfloat16) -> NamizenWeights:
    """The tables of one GPU from a checkpoint mapping (each tensor is asked for once)."""
    check_tensors(g, tensors)
    dev, W, Wp = torch.device(device), g.hidden_size, pad8(g.hidden_size)
    shapes = g.tensor_shapes()

    def get(name: str) -> torch.Tensor:
        t = tensors[name]
        if tuple(t.shape) != shapes[name]:
            raise CheckpointValidationError(f"{name!r} has shape {tuple(t.shape)}, the configuration says {shapes[name]}")
        return t

    def row(name: str) -> torch.Tensor:
        return padded(get(name)[None, :], 1, Wp, dtype, dev)[0]

    layers = []
    for i, spec in enumerate(g.layers):
        m, p = spec.mixer, f"l{i}"
        qkv = torch.zeros((pad8(m.qkv_width), Wp), dtype=dtype, device=dev)
        conv = torch.ones((m.conv, m.qkv_width), dtype=torch.float32, device=dev)
        at = 0
        for name, rows in (("q", m.q_width), ("k", m.k_width), ("v", m.v_width)):
            qkv[at : at + rows, :W] = get(f"{p}.mix.{name}").to(device=dev, dtype=dtype)
            if f"{p}.mix.{name}.conv" in tensors:
                conv[:, at : at + rows] = get(f"{p}.mix.{name}.conv").to(device=dev, dtype=torch.float32).T
            at += rows
        attn_cols, ff_cols = pad8(m.out_width), pad8(spec.ff)
        out = torch.zeros((Wp, attn_cols + ff_cols), dtype=dtype, device=dev)
        out[:W, : m.out_width] = get(p + ".mix.o").to(device=dev, dtype=dtype)
        gate_up = None
        if spec.ff:
            gate_up = torch.zeros((2 * ff_cols, Wp), dtype=dtype, device=dev)
            gate_up[: spec.ff, :W] = get(p + ".mlp.gate").to(device=dev, dtype=dtype)
            gate_up[ff_cols : ff_cols + spec.ff, :W] = get(p + ".mlp.up").to(device=dev, dtype=dtype)
            out[:W, attn_cols : attn_cols + spec.ff] = get(p + ".mlp.down").to(device=dev, dtype=dtype)
        mixes = m.v_mix and i != g.first_mixing_layer
        layers.append(NamizenLayer(
            norm1=row(p + ".norm1"), norm2=row(p + ".norm2") if spec.ff else None, qkv=qkv, conv=conv.contiguous(), gate_up=gate_up, out=out,
            sink=get(p + ".mix.sink").to(device=dev, dtype=torch.float32).contiguous(), mix=float(get(p + ".mix.vmix")) if mixes else 0.0,
            attn_cols=attn_cols, ff_cols=ff_cols))
    return NamizenWeights(g, dtype, embed=padded(get("embed"), g.vocab_size, Wp, dtype, dev), layers=layers, final_norm=row("final.norm"),
                          head=padded(get("head"), pad8(g.vocab_size), Wp, dtype, dev))


def random_spread(name: str, shape) -> tuple[float, float]:
    """Mean and standard deviation of the tensors that are made on the device (``DeviceRandomTensors``)."""
    if "norm" in name:
        return 1.0, 0.1
    if not shape:
        return 0.5, 0.0
    return 0.0, 1.0 if name == "embed" else shape[-1] ** -0.5
