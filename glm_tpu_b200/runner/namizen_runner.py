"""The Namizen runner of one GPU: resident weights, ring caches, and the programs of ``LaneRunner`` over ``NamizenModel``."""

from __future__ import annotations

import time

import torch

from glm_tpu_b200.config.cache import RingCacheConfig
from glm_tpu_b200.exceptions import PlanValidationError
from glm_tpu_b200.models.namizen.model import NamizenModel, NamizenWorkspace, RingState
from glm_tpu_b200.models.namizen.weights import DeviceRandomTensors, NamizenWeights, pad8, pad16, resident_weights
from glm_tpu_b200.parallel.peer import PeerGroup
from glm_tpu_b200.runner.admission import project_live, project_ring_memory, require_admitted
from glm_tpu_b200.runner.lane_runner import LaneRunner, RunnerReport


class NamizenRunner(LaneRunner):
    kv_layout = "local"

    def __init__(self, weights: NamizenWeights, *, context_capacity: int, lanes: int = 1, prefill_chunk: int = 512, use_graphs: bool | None = None,
                 wait_limit: int | None = None):
        from glm_tpu_b200 import envs

        self.use_graphs = envs.GLM_B200_CUDA_GRAPHS if use_graphs is None else use_graphs
        wait_limit = envs.GLM_B200_WAIT_LIMIT if wait_limit is None else wait_limit
        self.weights, self.g = weights, weights.geometry
        self.device = weights.embed.device
        self.world, self.rank, self.lanes = 1, 0, lanes
        self.prefill_chunk = max(1, min(prefill_chunk, context_capacity))
        self.cache = RingCacheConfig(self.g, context_capacity, lanes=lanes, element_bytes=torch.empty((), dtype=weights.dtype).element_size())
        self.report = RunnerReport()
        t0 = time.perf_counter()
        self.report.memory = self._project(already_resident=weights.bytes_resident)
        require_admitted(self.report.memory)
        with torch.cuda.device(self.device):
            self.peer = PeerGroup(1, 0, staging_bytes=0, wait_limit=wait_limit, device=self.device)
            self.model = NamizenModel(weights, self.cache, self.peer)
            self.state = RingState.allocate(self.cache, self.device, weights.dtype)
            self.decode_ws = NamizenWorkspace(self.model, lanes, prefill=False)
        self._ready()
        self.report.phases["allocate"] = time.perf_counter() - t0

    def _project(self, *, already_resident: int, mem_info=None) -> dict:
        g, item = self.g, self.cache.element_bytes
        rows = self.lanes + self.prefill_chunk
        widest = max(pad8(m.qkv_width) + m.heads * pad16(m.dim) + m.kv_heads * pad16(m.vdim) + pad8(m.out_width) + 3 * pad8(layer.ff)
                     for layer in g.layers for m in (layer.mixer,))
        linear = max(self.cache.linear_rows(i, self.prefill_chunk) * m.kv_heads * (pad16(m.dim) + pad16(m.vdim))
                     for i, layer in enumerate(g.layers) for m in (layer.mixer,))
        workspace = rows * (pad8(g.hidden_size) * (8 + 2 * item) + widest * item) + linear * item + self.lanes * pad8(g.vocab_size) * 4
        rot = {(layer.mixer.rot_dims, layer.mixer.rot_base) for layer in g.layers}
        workspace += sum(dims * 4 * self.cache.context_capacity for dims, _ in rot)
        projection = project_ring_memory(self.cache, self.weights.bytes_resident, workspace)
        free, total = mem_info if mem_info is not None else torch.cuda.mem_get_info(self.device)
        return project_live(projection, free, total, already_resident=already_resident)

    def admit_request(self, mem_info=None) -> dict:
        """Before every request: everything projected is resident by now, so the reserve must still be free on the device."""
        admitted = self._project(already_resident=1 << 62, mem_info=mem_info)
        require_admitted(admitted)
        self.report.memory["last_request"] = {"device_free": admitted["device_free"], "reserve": admitted["reserve"]}
        return admitted

    def _prefill_workspace(self) -> NamizenWorkspace:
        return NamizenWorkspace(self.model, self.prefill_chunk, prefill=True)

    def memory_stats(self) -> dict:
        free, total = torch.cuda.mem_get_info(self.device)
        return {
            "device_total_bytes": int(total), "device_free_bytes": int(free),
            "torch_allocated_bytes": int(torch.cuda.memory_allocated(self.device)),
            "torch_peak_allocated_bytes": int(torch.cuda.max_memory_allocated(self.device)),
            "weights_bytes": int(self.weights.bytes_resident),
            "kv_cache_bytes": int(self.cache.cache_bytes_per_gpu()),
            "kv_layout": self.kv_layout,
            "fallbacks": dict(self.model.fallbacks),
        }

    def synthetic_context(self, lane: int, depth: int, seed: int = 0) -> None:
        """Benchmarks only: make ``lane`` look ``depth`` tokens deep without running a prefill (random cache rows and convolution state)."""
        from glm_tpu_b200.ops import native

        if not 0 < depth < self.cache.context_capacity:
            raise ValueError("depth does not fit the context capacity")
        st = self.state
        with torch.cuda.device(self.device):
            for i, tensor in enumerate(t for group in (st.k, st.v, st.conv) for t in group):
                if tensor[lane].numel():
                    native.fill_random_bf16(tensor[lane], seed * 4096 + i, 0.0, 0.5)
            st.tokens[lane] = 1 + seed % max(self.g.vocab_size - 1, 1)
            st.positions[lane] = depth
            st.active[lane] = 1
            torch.cuda.synchronize(self.device)


def build(geometry, *, world: int = 1, rank: int = 0, device=None, checkpoint=None, seed: int = 0, dtype: torch.dtype = torch.bfloat16,
          comm: str | None = None, kv_layout: str = "auto", stripe: int = 0, decode_path: str = "auto", **kwargs) -> NamizenRunner:
    """``checkpoint``: a tensor mapping, or ``None`` for random weights made on the device.  The layout arguments of the multi-GPU family are
    accepted where they mean nothing here; more than one GPU is refused."""
    if world != 1:
        raise PlanValidationError("Namizen runs on one GPU")
    if comm not in (None, "fused", "nccl") or kv_layout not in ("auto", "replicated") or decode_path not in ("auto", "kernels"):
        raise PlanValidationError("Namizen has one cache layout and one decode path")
    device = torch.device(device if device is not None else f"cuda:{torch.cuda.current_device()}")
    with torch.cuda.device(device):
        tensors = checkpoint if checkpoint is not None else DeviceRandomTensors(geometry, device, seed)
        weights = resident_weights(geometry, tensors, device, dtype)
    return NamizenRunner(weights, **kwargs)
