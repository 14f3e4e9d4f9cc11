"""Checkpoints that are a plain directory (``config.json`` and safetensors files), and helpers to lay their tensors out for the kernels.

``SourceTensors`` reads the files through the same streaming reader the packed checkpoints use.  Resident tables are padded: every row to a
multiple of 8 columns (zeros), so any width, head size or feed-forward size meets the alignment of the tensor-core and streaming kernels.
"""

from __future__ import annotations

from collections.abc import Mapping
from pathlib import Path

import torch

from glm_tpu_b200.exceptions import CheckpointValidationError
from glm_tpu_b200.model_loader.sharded_state import format as fmt


def pad_to(n: int, multiple: int) -> int:
    return -(-n // multiple) * multiple


def pad8(n: int) -> int:
    return pad_to(n, 8)


def pad16(n: int) -> int:
    return pad_to(n, 16)


def padded(t: torch.Tensor, rows: int, cols: int, dtype, device) -> torch.Tensor:
    out = torch.zeros((rows, cols), dtype=dtype, device=device)
    out[: t.shape[0], : t.shape[1]] = t.to(device=device, dtype=dtype)
    return out


class SourceTensors(Mapping):
    """``name -> tensor`` over the ``*.safetensors`` files of a directory; a tensor is streamed to ``device`` when it is looked up."""

    def __init__(self, root: Path, device=None):
        from glm_tpu_b200.model_loader.source_inventory import read_source_inventory

        self.device = device
        tensors = read_source_inventory(root).tensors
        self.shapes = {name: tuple(t.shape) for name, t in tensors.items()}
        self._where = {name: t.shard for name, t in tensors.items()}
        self._readers = {shard: fmt.TensorReader(Path(root) / shard) for shard in sorted(set(self._where.values()))}

    def __getitem__(self, name: str) -> torch.Tensor:
        return self._readers[self._where[name]].read(name, device=self.device)

    def __iter__(self):
        return iter(self._where)

    def __len__(self) -> int:
        return len(self._where)


class ShapedTensors:
    """Looks tensors up by name and checks them against the shapes the configuration asks for."""

    def __init__(self, tensors: Mapping, shapes: Mapping, optional=()):
        self.tensors, self.shapes = tensors, shapes
        missing = [name for name in shapes if name not in tensors and name not in optional]
        if missing:
            raise CheckpointValidationError(f"the checkpoint misses {len(missing)} tensors, e.g. {missing[0]!r}")

    def __contains__(self, name: str) -> bool:
        return name in self.tensors

    def __call__(self, name: str) -> torch.Tensor:
        t = self.tensors[name]
        if tuple(t.shape) != self.shapes[name]:
            raise CheckpointValidationError(f"{name!r} has shape {tuple(t.shape)}, the configuration says {self.shapes[name]}")
        return t


class DeviceRandomTensors(Mapping):
    """Random bf16 tensors made on the GPU one at a time (speed measurements at full size: nothing passes through host memory).
    ``spread(name, shape)`` gives mean and standard deviation."""

    def __init__(self, shapes: Mapping, spread, device, seed: int = 0):
        self.shapes, self.spread, self.device, self.seed = dict(shapes), spread, torch.device(device), seed
        self._index = {name: i for i, name in enumerate(self.shapes)}

    def __getitem__(self, name: str) -> torch.Tensor:
        from glm_tpu_b200.ops import native

        out = torch.empty(self.shapes[name], dtype=torch.bfloat16, device=self.device)
        mean, std = self.spread(name, self.shapes[name])
        native.fill_random_bf16(out, self.seed * 4096 + self._index[name], mean, std)
        return out

    def __iter__(self):
        return iter(self.shapes)

    def __len__(self) -> int:
        return len(self.shapes)
