"""The model families the engine serves.

A family says how its configuration is recognised and read, where its weights come from, which kernels it needs and how its runner and its
CPU oracle are made.  Everything above (worker, engine, command line, replay of traces) asks the registry and never names a family.
Modules of a family are imported when they are needed, so reading a configuration imports no kernels.
"""

from __future__ import annotations

import json
from dataclasses import dataclass
from pathlib import Path
from typing import Any, Callable, Mapping

from glm_tpu_b200.config import model as glm_config
from glm_tpu_b200.config import namizen as namizen_config
from glm_tpu_b200.config import zikevik as zikevik_config
from glm_tpu_b200.exceptions import ConfigValidationError


@dataclass(frozen=True)
class Family:
    name: str
    architecture: str
    geometry_type: type
    presets: Mapping[str, Callable[[], Any]]  # `random:<preset>` models
    library_component: str | None  # kernels it needs when the complete library is not built (None: the complete library)
    dtypes: tuple[str, ...]
    from_config: Callable[[Mapping], Any]
    matches: Callable[[Mapping], bool]
    is_checkpoint: Callable[[Path], bool]  # is this directory one of its checkpoints?
    read_geometry: Callable[[Path], Any]
    load_checkpoint: Callable[..., Mapping]  # (path, rank, world, *, pins, device) -> name -> tensor
    load_full_checkpoint: Callable[[Path], Mapping]  # the same on the CPU (oracle)
    random_checkpoint: Callable[..., Mapping]  # (geometry, seed) -> name -> tensor, the bits the oracle uses too
    small_enough_for_host: Callable[[Any], bool]  # random weights are made on the host (same bits as the oracle) up to this size
    next_token: Callable[..., Callable]  # (geometry, checkpoint, capacity) -> sequence -> greedy next token, on the CPU
    build_runner: Callable[..., Any] | None = None
    multi_gpu: bool = True


def _read_config(path: Path) -> dict:
    try:
        return json.loads((Path(path) / "config.json").read_text(encoding="utf-8"))
    except (OSError, ValueError) as exc:
        raise ConfigValidationError(f"{path} has no readable config.json") from exc


# ------------------------------------------------------------------------------------------------ GLM-MoE-DSA
def _glm_geometry(path: Path):
    from glm_tpu_b200.model_loader.sharded_state import loader

    return loader.read_geometry(path)


def _glm_load(path: Path, rank: int, world: int, *, pins=None, device=None):
    from glm_tpu_b200.model_loader.sharded_state import loader

    return loader.load_rank_checkpoint(path, rank, world, pins=pins, device=device)


def _glm_load_full(path: Path):
    from glm_tpu_b200.model_loader.sharded_state import loader

    return loader.load_full_checkpoint(path)


def _glm_random(geometry, seed: int = 0):
    from glm_tpu_b200.models.glm_moe_dsa.weights import random_checkpoint

    return random_checkpoint(geometry, seed=seed)


def _glm_next_token(geometry, checkpoint, capacity: int):
    from glm_tpu_b200.oracle import contract

    weights = contract.OracleWeights.from_checkpoint(geometry, checkpoint)
    return lambda sequence: int(contract.forward(weights, sequence, capacity=capacity).tokens[-1])


def _glm_is_checkpoint(path: Path) -> bool:
    from glm_tpu_b200.model_loader.sharded_state.format import GEOMETRY_FILE

    return (Path(path) / GEOMETRY_FILE).exists()


GLM = Family(
    name="glm_moe_dsa", architecture="GlmMoeDsaForCausalLM", geometry_type=glm_config.ModelGeometry,
    presets={"tiny": glm_config.tiny_geometry, "small": glm_config.small_geometry, "glm53": glm_config.glm53_geometry},
    library_component=None, dtypes=("bfloat16",), from_config=glm_config.ModelGeometry.from_hf_config,
    matches=lambda config: config.get("model_type") == "glm_moe_dsa", is_checkpoint=_glm_is_checkpoint, read_geometry=_glm_geometry,
    load_checkpoint=_glm_load, load_full_checkpoint=_glm_load_full, random_checkpoint=_glm_random,
    small_enough_for_host=lambda g: g.num_layers <= 8 and g.hidden_size <= 1024, next_token=_glm_next_token)


# ------------------------------------------------------------------------------------------------ one-GPU families read from a directory
def _load_directory(architecture: str):
    def load(path: Path, rank: int = 0, world: int = 1, *, pins=None, device=None):
        from glm_tpu_b200.exceptions import CheckpointValidationError
        from glm_tpu_b200.model_loader.directory import SourceTensors

        if any((pins or {}).values()):
            raise CheckpointValidationError(f"the site pins a packed checkpoint; a {architecture} directory has no manifest to pin")
        return SourceTensors(path, device=device)

    return load


def _matches(architecture: str):
    return lambda config: config.get("architecture") == architecture


def _is_directory_of(architecture: str):
    def is_checkpoint(path: Path) -> bool:
        try:
            return _matches(architecture)(_read_config(path))
        except ConfigValidationError:
            return False

    return is_checkpoint


def _random_weights(package: str):
    def random(geometry, seed: int = 0):
        import importlib

        return importlib.import_module(f"glm_tpu_b200.models.{package}.weights").random_checkpoint(geometry, seed=seed)

    return random


def _oracle_next_token(module: str):
    def next_token(geometry, checkpoint, capacity: int):
        import importlib

        import torch

        oracle = importlib.import_module(f"glm_tpu_b200.oracle.{module}")
        config, tensors = geometry.to_config(), dict(checkpoint.items())
        return lambda sequence: int(torch.argmax(oracle.forward(config, tensors, sequence, dtype=torch.float32)[-1]))

    return next_token


def _runner_of(module: str):
    def build(geometry, **kwargs):
        import importlib

        return importlib.import_module(f"glm_tpu_b200.runner.{module}").build(geometry, **kwargs)

    return build


def _directory_family(name: str, architecture: str, geometry_type: type, presets: Mapping, read_geometry: Callable[[Path], Any]) -> Family:
    """A family that runs on one GPU, from ``config.json`` and safetensors, with modules called after it."""
    load = _load_directory(architecture)
    return Family(
        name=name, architecture=architecture, geometry_type=geometry_type, presets=presets, library_component=name, dtypes=("bfloat16", "float32"),
        from_config=geometry_type.from_config, matches=_matches(architecture), is_checkpoint=_is_directory_of(architecture),
        read_geometry=read_geometry, load_checkpoint=load, load_full_checkpoint=load, random_checkpoint=_random_weights(name),
        small_enough_for_host=lambda g: g.num_layers <= 16 and g.hidden_size <= 1024, next_token=_oracle_next_token(name),
        build_runner=_runner_of(f"{name}_runner"), multi_gpu=False)


NAMIZEN = _directory_family("namizen", namizen_config.ARCHITECTURE, namizen_config.NamizenGeometry, {"namizen-tiny": namizen_config.tiny_namizen},
                            lambda path: namizen_config.NamizenGeometry.from_config(_read_config(path)))


def _zikevik_geometry(path: Path):
    from glm_tpu_b200.model_loader.directory import SourceTensors

    return zikevik_config.ZikevikGeometry.from_config(_read_config(path), SourceTensors(path).shapes)


ZIKEVIK = _directory_family("zikevik", zikevik_config.ARCHITECTURE, zikevik_config.ZikevikGeometry, {"zikevik-tiny": zikevik_config.tiny_zikevik},
                            _zikevik_geometry)

FAMILIES = (GLM, NAMIZEN, ZIKEVIK)


def family_of(geometry) -> Family:
    for family in FAMILIES:
        if isinstance(geometry, family.geometry_type):
            return family
    raise ConfigValidationError(f"no model family takes a {type(geometry).__name__}")


def family_of_config(config: Mapping) -> Family:
    for family in FAMILIES:
        if family.matches(config):
            return family
    raise ConfigValidationError("no model family takes this config.json")


def resolve_model(spec: str):
    """``(geometry, source)`` of ``random:<preset>[:layers]`` or of a checkpoint directory; source is ``('random', None)`` or
    ``('checkpoint', Path)``."""
    if spec.startswith("random:"):
        parts = spec.split(":")
        presets = {name: make for family in FAMILIES for name, make in family.presets.items()}
        if parts[1] not in presets:
            raise ConfigValidationError(f"random models are {', '.join(presets)}")
        base = presets[parts[1]]()
        return (base.truncated(int(parts[2])) if len(parts) > 2 else base), ("random", None)
    path = Path(spec)
    for family in FAMILIES:
        if family is not GLM and family.is_checkpoint(path):
            return family.read_geometry(path), ("checkpoint", path)
    return GLM.read_geometry(path), ("checkpoint", path)
