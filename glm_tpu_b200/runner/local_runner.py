"""What the runners of the one-GPU families share: construction with memory admission, per-request admission, memory report, random contexts.

A family's runner says how its cache configuration, model, state and workspaces are made and how large its scratch memory is; lanes, the
captured decode step, prefill and replay come from ``LaneRunner``.
"""

from __future__ import annotations

import time

import torch

from glm_tpu_b200.exceptions import PlanValidationError
from glm_tpu_b200.model_loader.directory import DeviceRandomTensors
from glm_tpu_b200.parallel.peer import PeerGroup
from glm_tpu_b200.runner.admission import project_live, project_local_memory, require_admitted
from glm_tpu_b200.runner.lane_runner import LaneRunner, RunnerReport


class LocalRunner(LaneRunner):
    """``weights`` brings ``geometry``, ``dtype``, ``embed`` and ``bytes_resident``."""

    kv_layout = "local"

    # ------------------------------------------------------------------ what a family provides
    def _make_cache(self, context_capacity: int, element_bytes: int):
        raise NotImplementedError

    def _make_model(self):
        raise NotImplementedError

    def _make_state(self):
        raise NotImplementedError

    def _make_workspace(self, rows: int, *, prefill: bool):
        raise NotImplementedError

    def _workspace_bytes(self) -> int:
        """Scratch memory of the decode and the prefill workspace and the tables made at construction."""
        raise NotImplementedError

    def _random_state(self) -> list:
        """``[(per-lane tensor, mean, standard deviation), ...]``: what ``synthetic_context`` fills."""
        raise NotImplementedError

    # ------------------------------------------------------------------ construction
    def __init__(self, weights, *, context_capacity: int, lanes: int = 1, prefill_chunk: int = 512, use_graphs: bool | None = None,
                 wait_limit: int | None = None):
        from glm_tpu_b200 import envs

        self.use_graphs = envs.GLM_B200_CUDA_GRAPHS if use_graphs is None else use_graphs
        wait_limit = envs.GLM_B200_WAIT_LIMIT if wait_limit is None else wait_limit
        self.weights, self.g = weights, weights.geometry
        self.device = weights.embed.device
        self.world, self.rank, self.lanes = 1, 0, lanes
        self.prefill_chunk = max(1, min(prefill_chunk, context_capacity))
        self.cache = self._make_cache(context_capacity, torch.empty((), dtype=weights.dtype).element_size())
        self.report = RunnerReport()
        t0 = time.perf_counter()
        self.report.memory = self._project(already_resident=weights.bytes_resident)
        require_admitted(self.report.memory)
        with torch.cuda.device(self.device):
            self.peer = PeerGroup(1, 0, staging_bytes=0, wait_limit=wait_limit, device=self.device)
            self.model = self._make_model()
            self.state = self._make_state()
            self.decode_ws = self._make_workspace(lanes, prefill=False)
        self._ready()
        self.report.phases["allocate"] = time.perf_counter() - t0

    def _prefill_workspace(self):
        return self._make_workspace(self.prefill_chunk, prefill=True)

    def _project(self, *, already_resident: int, mem_info=None) -> dict:
        projection = project_local_memory(self.cache, self.weights.bytes_resident, self._workspace_bytes())
        free, total = mem_info if mem_info is not None else torch.cuda.mem_get_info(self.device)
        return project_live(projection, free, total, already_resident=already_resident)

    # ------------------------------------------------------------------ requests
    def admit_request(self, mem_info=None) -> dict:
        """Before every request: everything projected is resident by now, so the reserve must still be free on the device."""
        admitted = self._project(already_resident=1 << 62, mem_info=mem_info)
        require_admitted(admitted)
        self.report.memory["last_request"] = {"device_free": admitted["device_free"], "reserve": admitted["reserve"]}
        return admitted

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
        """Benchmarks only: make ``lane`` look ``depth`` tokens deep without running a prefill (random cache rows and state)."""
        from glm_tpu_b200.ops import native

        if not 0 < depth < self.cache.context_capacity:
            raise ValueError("depth does not fit the context capacity")
        st = self.state
        with torch.cuda.device(self.device):
            for i, (tensor, mean, std) in enumerate(self._random_state()):
                if not tensor[lane].numel():
                    continue
                if tensor.dtype == torch.float32 and self.weights.dtype != torch.float32:
                    tensor[lane].normal_(mean, std, generator=torch.Generator(self.device).manual_seed(seed * 4096 + i))
                else:
                    native.fill_random_bf16(tensor[lane], seed * 4096 + i, mean, std)
            st.tokens[lane] = 1 + seed % max(self.g.vocab_size - 1, 1)
            st.positions[lane] = depth
            st.active[lane] = 1
            torch.cuda.synchronize(self.device)


def build_local(runner_type, resident_weights, random_spread, geometry, *, world: int = 1, rank: int = 0, device=None, checkpoint=None, seed: int = 0,
                dtype: torch.dtype = torch.bfloat16, comm: str | None = None, kv_layout: str = "auto", stripe: int = 0, decode_path: str = "auto",
                **kwargs) -> LocalRunner:
    """``checkpoint``: a tensor mapping, or ``None`` for random weights made on the device.  The layout arguments of the multi-GPU family are
    accepted where they mean nothing here; more than one GPU is refused."""
    name = geometry.to_config()["architecture"]
    if world != 1:
        raise PlanValidationError(f"{name} runs on one GPU")
    if comm not in (None, "fused", "nccl") or kv_layout not in ("auto", "replicated") or decode_path not in ("auto", "kernels"):
        raise PlanValidationError(f"{name} has one cache layout and one decode path")
    device = torch.device(device if device is not None else f"cuda:{torch.cuda.current_device()}")
    with torch.cuda.device(device):
        tensors = checkpoint if checkpoint is not None else DeviceRandomTensors(geometry.tensor_shapes(), random_spread, device, seed)
        weights = resident_weights(geometry, tensors, device, dtype)
    return runner_type(weights, **kwargs)
