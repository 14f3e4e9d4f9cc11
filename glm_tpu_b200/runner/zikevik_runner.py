"""The Zikevik runner of one GPU: resident weights, latent caches and recurrent states, and the programs of ``LaneRunner`` over ``ZikevikModel``."""

from __future__ import annotations

import torch

from glm_tpu_b200.config.cache import HybridCacheConfig
from glm_tpu_b200.model_loader.directory import pad8
from glm_tpu_b200.models.zikevik.model import HybridState, ZikevikModel, ZikevikWorkspace, workspace_elements
from glm_tpu_b200.models.zikevik.weights import random_spread, resident_weights
from glm_tpu_b200.runner.local_runner import LocalRunner, build_local


class ZikevikRunner(LocalRunner):
    def _make_cache(self, context_capacity: int, element_bytes: int) -> HybridCacheConfig:
        return HybridCacheConfig(self.g, context_capacity, lanes=self.lanes, element_bytes=element_bytes)

    def _make_model(self) -> ZikevikModel:
        return ZikevikModel(self.weights, self.cache, self.peer)

    def _make_state(self) -> HybridState:
        return HybridState.allocate(self.cache, self.device, self.weights.dtype)

    def _make_workspace(self, rows: int, *, prefill: bool) -> ZikevikWorkspace:
        return ZikevikWorkspace(self.model, rows, prefill=prefill)

    def _workspace_bytes(self) -> int:
        g, item, is_f32 = self.g, self.cache.element_bytes, self.weights.dtype == torch.float32
        total = self.lanes * pad8(g.vocab_size) * 4
        for rows, prefill in ((self.lanes, False), (self.prefill_chunk, True)):
            sizes = workspace_elements(g, self.cache, rows, prefill=prefill, is_f32=is_f32)
            total += sum(sizes["model"].values()) * item + sum(sizes["f32"].values()) * 4 + rows * pad8(g.hidden_size) * (8 + item)
        rot = {(layer.mixer.rot_dim, layer.mixer.rot_base) for i, layer in enumerate(g.layers) if self.cache.is_latent(i)}
        return total + sum(dims * 4 * self.cache.context_capacity for dims, _ in rot)

    def _random_state(self) -> list:
        st = self.state
        return [(t, 0.0, 0.5) for group in (st.latent, st.conv) for t in group if t is not None] + [(t, 0.0, 0.1) for t in st.state if t is not None]


def build(geometry, **kwargs) -> ZikevikRunner:
    return build_local(ZikevikRunner, resident_weights, random_spread, geometry, **kwargs)
