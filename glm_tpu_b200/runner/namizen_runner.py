"""The Namizen runner of one GPU: resident weights, ring caches, and the programs of ``LaneRunner`` over ``NamizenModel``."""

from __future__ import annotations

from glm_tpu_b200.config.cache import RingCacheConfig
from glm_tpu_b200.model_loader.directory import pad8, pad16
from glm_tpu_b200.models.namizen.model import NamizenModel, NamizenWorkspace, RingState
from glm_tpu_b200.models.namizen.weights import random_spread, resident_weights
from glm_tpu_b200.runner.local_runner import LocalRunner, build_local


class NamizenRunner(LocalRunner):
    def _make_cache(self, context_capacity: int, element_bytes: int) -> RingCacheConfig:
        return RingCacheConfig(self.g, context_capacity, lanes=self.lanes, element_bytes=element_bytes)

    def _make_model(self) -> NamizenModel:
        return NamizenModel(self.weights, self.cache, self.peer)

    def _make_state(self) -> RingState:
        return RingState.allocate(self.cache, self.device, self.weights.dtype)

    def _make_workspace(self, rows: int, *, prefill: bool) -> NamizenWorkspace:
        return NamizenWorkspace(self.model, rows, prefill=prefill)

    def _workspace_bytes(self) -> int:
        g, item = self.g, self.cache.element_bytes
        rows = self.lanes + self.prefill_chunk
        widest = max(pad8(m.qkv_width) + m.heads * pad16(m.dim) + m.kv_heads * pad16(m.vdim) + pad8(m.out_width) + 3 * pad8(layer.ff)
                     for layer in g.layers for m in (layer.mixer,))
        linear = max(self.cache.linear_rows(i, self.prefill_chunk) * m.kv_heads * (pad16(m.dim) + pad16(m.vdim))
                     for i, layer in enumerate(g.layers) for m in (layer.mixer,))
        workspace = rows * (pad8(g.hidden_size) * (8 + 2 * item) + widest * item) + linear * item + self.lanes * pad8(g.vocab_size) * 4
        rot = {(layer.mixer.rot_dims, layer.mixer.rot_base) for layer in g.layers}
        return workspace + sum(dims * 4 * self.cache.context_capacity for dims, _ in rot)

    def _random_state(self) -> list:
        return [(t, 0.0, 0.5) for group in (self.state.k, self.state.v, self.state.conv) for t in group]


def build(geometry, **kwargs) -> NamizenRunner:
    return build_local(NamizenRunner, resident_weights, random_spread, geometry, **kwargs)
