"""Zikevik weights: random fixtures, and the tables one GPU keeps.

The checkpoint is a flat ``name -> tensor`` mapping (``ZikevikGeometry.tensor_shapes``), e.g. ``model_loader.directory.SourceTensors``.
Resident tables are laid out for the kernels.  Everything a mixer reads from its input is one table: query, key, value, beta and the first
halves of the two low-rank projections of a delta-rule layer; both latents, the rotated key part and the output gate of a latent layer.
Sections start at multiples of 8 rows, rows are padded to multiples of 8 columns (zeros).  Vectors that enter fp32 arithmetic are fp32.  A
layer that uses another layer's weights shares its tables.  Tables are bf16 for serving and fp32 for the 32-bit path.
"""

from __future__ import annotations

from collections.abc import Mapping
from dataclasses import dataclass

import torch

from glm_tpu_b200.config.zikevik import DeltaSpec, LatentSpec, RoutedSpec, ZikevikGeometry
from glm_tpu_b200.model_loader.directory import ShapedTensors, pad8, pad16, pad_to, padded


def random_checkpoint(g: ZikevikGeometry, seed: int = 0) -> dict[str, torch.Tensor]:
    """Random bf16 weights on the CPU (fixtures): projections ``N(0, 1/fan_in)``, norms around their neutral value, decays from slow to fast."""
    gen = torch.Generator().manual_seed(seed)
    out: dict[str, torch.Tensor] = {}
    for name, shape in g.tensor_shapes().items():
        mean, std = random_spread(name, shape)
        z = mean + std * torch.randn(shape, generator=gen)
        if name.endswith(".conv"):
            z[:, -1] += 0.8
        out[name] = z.to(torch.bfloat16)
    return out


def random_spread(name: str, shape) -> tuple[float, float]:
    """Mean and standard deviation of a random tensor."""
    leaf = name.rsplit(".", 1)[-1]
    if leaf in ("norm1", "norm2") or name == "final.norm":
        return 0.0, 0.1  # stored around zero
    if leaf == "norm":
        return 1.0, 0.1
    if leaf == "conv":
        return 0.0, 0.4
    if leaf == "A_log":
        return 0.0, 0.7
    if leaf == "dt_bias":
        return -3.0, 1.0
    if leaf == "sink":
        return 0.5, 1.0
    return 0.0, 1.0 if name == "embed" else shape[-1] ** -0.5


# ------------------------------------------------------------------------------------------------ resident tables
@dataclass
class DeltaTables:
    proj: torch.Tensor  # [q | k | v (channels of the convolution) | beta | decay rank | gate rank, width']
    conv: torch.Tensor  # [taps, channels] fp32
    a2: torch.Tensor  # [heads * dim', decay rank']
    g2: torch.Tensor  # [heads * vdim', gate rank']
    a_rate: torch.Tensor  # [heads] fp32: exp(A_log)
    dt_bias: torch.Tensor  # [heads * dim] fp32
    norm: torch.Tensor  # [vdim] fp32
    out: torch.Tensor  # [width', (heads * vdim)']
    off_b: int
    off_a: int
    off_g: int


@dataclass
class LatentTables:
    proj: torch.Tensor  # [query latent | key/value latent, rotated key part | gate, width']
    uq: torch.Tensor  # [heads * dimp, q_rank']: a head's dim unrotated rows, its rotated rows, zero rows
    uk: torch.Tensor  # [heads, dim, lat]
    uv: torch.Tensor  # [heads, vdim, lat]
    expand_k: torch.Tensor  # [heads * dimp, lat + pe]: cache row -> the keys of every head (the rotated part is copied)
    expand_v: torch.Tensor  # [heads * vdimp, lat]
    q_norm: torch.Tensor  # fp32
    kv_norm: torch.Tensor  # fp32
    sink: torch.Tensor  # [heads] fp32
    out: torch.Tensor  # [width', (heads * vdim)']
    off_kv: int
    off_gate: int
    dimp: int
    vdimp: int


@dataclass
class DenseTables:
    gate_up: torch.Tensor  # [2 ff', width']: gate rows, then up rows
    down: torch.Tensor  # [width', ff']

    @property
    def ff_cols(self) -> int:
        return self.down.shape[-1]


@dataclass
class RoutedTables:
    router: torch.Tensor  # [experts', width']
    gate_up: torch.Tensor  # [experts, 2 ff', width']
    down: torch.Tensor  # [experts, width', ff']

    @property
    def ff_cols(self) -> int:
        return self.down.shape[-1]


@dataclass
class ZikevikLayer:
    norm1: torch.Tensor
    mixer: DeltaTables | LatentTables
    norm2: torch.Tensor | None
    mlp: DenseTables | RoutedTables | None


@dataclass
class ZikevikWeights:
    geometry: ZikevikGeometry
    dtype: torch.dtype
    embed: torch.Tensor  # [vocab, width']
    layers: list[ZikevikLayer]  # one per layer; layers that share weights share the object
    final_norm: torch.Tensor
    head: torch.Tensor  # [vocab', width']
    bytes_resident: int = 0

    def __post_init__(self) -> None:
        tables = {id(t): t for t in (self.embed, self.final_norm, self.head)}
        for layer in self.layers:
            for part in (layer, layer.mixer, layer.mlp):
                if part is not None:
                    tables |= {id(t): t for t in vars(part).values() if isinstance(t, torch.Tensor)}
        self.bytes_resident = sum(t.numel() * t.element_size() for t in tables.values())


class _Maker:
    """Tables of one precision on one device."""

    def __init__(self, g: ZikevikGeometry, get: ShapedTensors, dtype, device):
        self.g, self.get, self.dtype, self.device = g, get, dtype, device
        self.W, self.Wp = g.hidden_size, pad8(g.hidden_size)

    def table(self, name: str, rows: int | None = None) -> torch.Tensor:
        t = self.get(name)
        return padded(t, t.shape[0] if rows is None else rows, pad8(t.shape[1]), self.dtype, self.device)

    def vector(self, name: str) -> torch.Tensor:
        return self.get(name).to(device=self.device, dtype=torch.float32).contiguous()

    def row(self, name: str) -> torch.Tensor:
        return padded(self.get(name)[None, :], 1, self.Wp, self.dtype, self.device)[0]

    def stacked(self, names) -> tuple[torch.Tensor, list[int]]:
        """Tables one under the other, each from a multiple of 8 rows on; ``names`` are groups whose members follow without a gap."""
        sizes = [sum(self.get.shapes[n][0] for n in group) for group in names]
        starts = [sum(pad8(s) for s in sizes[:i]) for i in range(len(sizes))]
        out = torch.zeros((sum(pad8(s) for s in sizes), self.Wp), dtype=self.dtype, device=self.device)
        for group, at in zip(names, starts):
            for name in group:
                t = self.get(name)
                out[at : at + t.shape[0], : self.W] = t.to(device=self.device, dtype=self.dtype)
                at += t.shape[0]
        return out, starts

    def delta(self, p: str, m: DeltaSpec) -> DeltaTables:
        proj, (_, off_b, off_a, off_g) = self.stacked([[p + "q", p + "k", p + "v"], [p + "b"], [p + "a1"], [p + "g1"]])
        conv = torch.cat([self.vector(f"{p}{n}.conv").T for n in "qkv"], dim=1).contiguous()
        return DeltaTables(proj=proj, conv=conv, a2=self.table(p + "a2", pad8(m.heads * m.dim)), g2=self.table(p + "g2", pad8(m.v_width)),
                           a_rate=self.vector(p + "A_log").exp(), dt_bias=self.vector(p + "dt_bias"), norm=self.vector(p + "norm"),
                           out=self.table(p + "o", self.Wp), off_b=off_b, off_a=off_a, off_g=off_g)

    def latent(self, p: str, m: LatentSpec) -> LatentTables:
        proj, (_, off_kv, off_gate) = self.stacked([[p + "dq"], [p + "dkv"], [p + "g"]])
        lat, pe, dimp, vdimp = pad16(m.kv_rank), pad16(m.rot_dim), pad16(m.dim + m.rot_dim), pad16(m.vdim)
        kw = dict(dtype=self.dtype, device=self.device)

        def per_head(name: str, rows: int, cols: int) -> torch.Tensor:
            t = self.get(name)
            return t.to(**kw).view(m.heads, t.shape[0] // m.heads, t.shape[1]), torch.zeros((m.heads, rows, cols), **kw)

        src, uq = per_head(p + "uq", dimp, pad8(m.q_rank))
        uq[:, : m.dim + m.rot_dim, : m.q_rank] = src
        src, uk = per_head(p + "uk", m.dim, lat)
        uk[:, :, : m.kv_rank] = src
        expand_k = torch.zeros((m.heads, dimp, lat + pe), **kw)
        expand_k[:, : m.dim, : m.kv_rank] = src
        i = torch.arange(m.rot_dim, device=self.device)
        expand_k[:, m.dim + i, lat + i] = 1.0
        src, uv = per_head(p + "uv", m.vdim, lat)
        uv[:, :, : m.kv_rank] = src
        expand_v = uv
        if vdimp != m.vdim:
            expand_v = torch.zeros((m.heads, vdimp, lat), **kw)
            expand_v[:, : m.vdim] = uv
        return LatentTables(proj=proj, uq=uq.view(m.heads * dimp, -1), uk=uk, uv=uv, expand_k=expand_k.view(m.heads * dimp, -1),
                            expand_v=expand_v.view(m.heads * vdimp, -1), q_norm=self.vector(p + "dq.norm"), kv_norm=self.vector(p + "dkv.norm"),
                            sink=self.vector(p + "sink"), out=self.table(p + "o", self.Wp), off_kv=off_kv, off_gate=off_gate, dimp=dimp, vdimp=vdimp)

    def _gate_up(self, p: str, ff: int, out: torch.Tensor) -> None:
        F = pad8(ff)
        for at, name in ((0, "gate"), (F, "up")):
            out[at : at + ff, : self.W] = self.get(p + name).to(device=self.device, dtype=self.dtype)

    def mlp(self, p: str, m) -> DenseTables | RoutedTables | None:
        if m is None:
            return None
        F, kw = pad8(m.ff), dict(dtype=self.dtype, device=self.device)
        if not isinstance(m, RoutedSpec):
            gate_up = torch.zeros((2 * F, self.Wp), **kw)
            self._gate_up(p, m.ff, gate_up)
            return DenseTables(gate_up, self.table(p + "down", self.Wp))
        gate_up, down = torch.zeros((m.experts, 2 * F, self.Wp), **kw), torch.zeros((m.experts, self.Wp, F), **kw)
        for e in range(m.experts):
            self._gate_up(f"{p}e{e}.", m.ff, gate_up[e])
            down[e, : self.W, : m.ff] = self.get(f"{p}e{e}.down").to(**kw)
        return RoutedTables(self.table(p + "router", pad8(m.experts)), gate_up, down)


def resident_weights(g: ZikevikGeometry, tensors: Mapping, device, dtype: torch.dtype = torch.bfloat16) -> ZikevikWeights:
    """The tables of one GPU from a checkpoint mapping."""
    make = _Maker(g, ShapedTensors(tensors, g.tensor_shapes()), dtype, torch.device(device))
    layers: list[ZikevikLayer | None] = [None] * g.num_layers
    for i, spec in enumerate(g.layers):
        if g.owner(i) == i:
            mixer = (make.delta if isinstance(spec.mixer, DeltaSpec) else make.latent)(f"l{i}.mix.", spec.mixer)
            layers[i] = ZikevikLayer(norm1=make.row(f"l{i}.norm1"), mixer=mixer, norm2=make.row(f"l{i}.norm2") if spec.mlp else None,
                                     mlp=make.mlp(f"l{i}.mlp.", spec.mlp))
    layers = [layers[g.owner(i)] for i in range(g.num_layers)]
    return ZikevikWeights(g, dtype, embed=padded(make.get("embed"), g.vocab_size, make.Wp, dtype, make.device), layers=layers,
                          final_norm=make.row("final.norm"), head=make.table("head", pad8(g.vocab_size)))
