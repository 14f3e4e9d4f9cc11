"""The GLM-MoE-DSA runner of one GPU: resident weights, caches, the prefill program and the CUDA-graph decode program.

The runner is what the engine drives (``LaneRunner`` is the part it shares with the other model families).  It owns

* the resident weights (``DeviceWeights``) and the peer-buffer registry,
* the device state for ``lanes`` concurrent chats (striped KV/index caches, token/position registers),
* the *decode program*: one token for every lane, captured once in a CUDA graph and replayed per step
  (positions and tokens live in device memory, so the graph is static),
* the *prefill program*: chunks of one lane's prompt, launched eagerly.

Parity: reference ``glm_tpu/runner/tpu_runner.py:29-289`` (load phases, program set, batch programs),
``runner/programs.py:80-118``, ``runner/kv_cache_manager.py:15-57``, ``runner/compilation_manager.py:28-69``
(here a program is a captured CUDA graph instead of a compiled XLA executable).
"""

from __future__ import annotations

import os
import time

import torch

from glm_tpu_b200.config.cache import CacheConfig
from glm_tpu_b200.config.parallel import ParallelLayout, default_expert_split
from glm_tpu_b200.models.glm_moe_dsa.model import DecoderState, GlmMoeDsaModel, Workspace
from glm_tpu_b200.models.glm_moe_dsa.weights import DeviceWeights
from glm_tpu_b200.ops import native
from glm_tpu_b200.parallel.peer import PeerGroup
from glm_tpu_b200.runner.admission import project_live, project_memory, require_admitted
from glm_tpu_b200.runner.lane_runner import LaneRunner, ProgramRecord, RunnerReport


class GpuModelRunner(LaneRunner):
    def __init__(self, weights: DeviceWeights, *, context_capacity: int, lanes: int = 1, stripe: int = 64, comm: str | None = None,
                 group=None, prefill_chunk: int = 512, use_graphs: bool | None = None, wait_limit: int | None = None,
                 staging_bytes: int | None = None, kv_layout: str = "auto", replica_budget_bytes: int = 32 << 30,
                 decode_path: str = "auto", mega_compat_ksplit: bool | None = None, emulate_shard: bool = False):
        from glm_tpu_b200 import envs

        # what the caller leaves open comes from the environment registry (GLM_B200_COMM, GLM_B200_CUDA_GRAPHS, GLM_B200_WAIT_LIMIT)
        comm = envs.GLM_B200_COMM if comm is None else comm
        use_graphs = envs.GLM_B200_CUDA_GRAPHS if use_graphs is None else use_graphs
        wait_limit = envs.GLM_B200_WAIT_LIMIT if wait_limit is None else wait_limit
        if comm not in ("fused", "nccl"):
            raise ValueError("comm is 'fused' or 'nccl'")
        self.weights = weights
        self.g, self.layout = weights.geometry, weights.layout
        self.device = weights.embed.device
        self.world, self.rank = self.layout.world, self.layout.rank
        # KV layout: a full replica of the latent cache on every GPU removes all attention exchanges; stripe the caches
        # by position over the GPUs once a replica would not fit the budget (long contexts, many lanes).
        if kv_layout not in ("auto", "striped", "replicated"):
            raise ValueError("kv_layout is 'auto', 'striped' or 'replicated'")
        replica = CacheConfig(self.g, context_capacity, world=1, stripe=stripe, lanes=lanes)
        if kv_layout == "auto":
            kv_layout = "replicated" if replica.cache_bytes_per_gpu() <= replica_budget_bytes else "striped"
        self.kv_layout = kv_layout if self.world > 1 else "local"
        self.cache = replica if kv_layout == "replicated" else CacheConfig(self.g, context_capacity, world=self.world, stripe=stripe,
                                                                          lanes=lanes)
        self.lanes = lanes
        self.report = RunnerReport()
        self.use_graphs = use_graphs
        self.prefill_chunk = prefill_chunk
        t0 = time.perf_counter()
        if staging_bytes is None:
            g = self.g
            staging_bytes = lanes * (g.attention_heads * g.kv_row_width * 2 + context_capacity * 4
                                     + self.world * self.layout.heads_local * (g.kv_lora_rank + 2) * 4 + self.world * 8) + (1 << 20)
            if self.world > 1 and prefill_chunk > 8:  # output + partial-tile slots of the prefill GEMM with the fused all-reduce
                staging_bytes += prefill_chunk * g.hidden_size * 2 + native.gemm_allreduce_part_bytes(prefill_chunk, g.hidden_size, self.world) + 8192
        # memory admission BEFORE anything large is allocated: the projection (weights already resident + caches of every lane
        # + staging + workspaces) against the device's size and against what the driver reports as free right now
        self.report.memory = self._project(weights.bytes_resident, staging_bytes, already_resident=weights.bytes_resident)
        require_admitted(self.report.memory)
        self._staging_bytes = staging_bytes
        with torch.cuda.device(self.device):
            # emulate_shard (measurements only): this process holds rank `rank`'s shard of a `world`-GPU layout but runs alone:
            # every exchange is skipped, so the outputs mean nothing and the decode step costs what one GPU of the box spends
            # outside the exchanges (persistent decode kernel only)
            self.emulate_shard = bool(emulate_shard) and self.world > 1
            if self.emulate_shard:
                self.peer = PeerGroup(1, 0, staging_bytes=0, wait_limit=wait_limit, group=None, device=self.device)
            else:
                self.peer = PeerGroup(self.world, self.rank, staging_bytes=staging_bytes if self.world > 1 else 0,
                                      wait_limit=wait_limit, group=group, device=self.device)
            self.model = GlmMoeDsaModel(weights, self.cache, self.peer, comm=comm, group=group)
            self.model.emulated_shard = self.emulate_shard
            self.state = DecoderState.allocate(self.cache, self.device)
            self.decode_ws = Workspace(self.model, lanes, "decode")
            # decode program: 'kernels' (default) is the per-kernel sequence; 'phases' runs the fused phases of
            # csrc/decode_mega.cu as 11 kernels per layer, 'mega' as stretches of one persistent cooperative kernel.  Both fused
            # forms agree with 'kernels' bit for bit and are slower on B200 as measured (they give up occupancy, the L1 and a
            # small instruction footprint for fewer launches), so 'auto' means 'kernels'.  GLM_B200_DECODE overrides 'auto'.
            import os

            if decode_path == "auto":
                decode_path = os.environ.get("GLM_B200_DECODE", "kernels")
            if decode_path not in ("auto", "phases", "mega", "kernels"):
                raise ValueError("decode_path is 'auto', 'phases', 'mega' or 'kernels'")
            if mega_compat_ksplit is None and "GLM_B200_MEGA_KSPLIT" in os.environ:
                mega_compat_ksplit = os.environ["GLM_B200_MEGA_KSPLIT"] == "compat"
            self.mega = None
            if decode_path != "kernels":
                from glm_tpu_b200.models.glm_moe_dsa.mega import MegaDecoder

                mega = MegaDecoder(self.model, self.decode_ws, self.state, compat_ksplit=mega_compat_ksplit,
                                   mode="persistent" if decode_path == "mega" else "phases")
                if mega.supported:
                    self.mega = mega
                elif decode_path != "auto":
                    raise ValueError(f"the fused decode phases do not take this configuration (code {mega.supported_code})")
            self.decode_path = ("mega" if self.mega.mode == "persistent" else "phases") if self.mega is not None else "kernels"
        self._ready()
        self.report.phases["allocate"] = time.perf_counter() - t0

    # ------------------------------------------------------------------ admission
    def _project(self, weight_bytes: int, staging_bytes: int, *, already_resident: int, mem_info=None) -> dict:
        projection = project_memory(self.g, self.layout, self.cache, weight_bytes, staging_bytes)
        free, total = mem_info if mem_info is not None else torch.cuda.mem_get_info(self.device)
        return project_live(projection, free, total, already_resident=already_resident)

    def admit_request(self, mem_info=None) -> dict:
        """Before every request: everything this runner projected is resident by now, so the device must still have the reserve
        free (another process on the GPU, a leak) and the status word must be clean.  Raises ``PlanValidationError``."""
        admitted = self._project(self.weights.bytes_resident, self._staging_bytes, already_resident=1 << 62, mem_info=mem_info)
        require_admitted(admitted)
        self.report.memory["last_request"] = {"device_free": admitted["device_free"], "reserve": admitted["reserve"]}
        return admitted

    # ------------------------------------------------------------------ decode program
    def _decode_body(self) -> None:
        if self.mega is not None:
            self.mega.step()
            return
        super()._decode_body()

    def _captures_graphs(self) -> bool:
        return self.use_graphs and (self.model.comm_mode == "fused" or self.world == 1)

    def _capture_decode(self) -> torch.cuda.CUDAGraph:
        try:
            return super()._capture_decode()
        except RuntimeError:
            if self.mega is None:
                raise
            # a driver that will not record a cooperative launch: the same grid as an ordinary launch (it fits the GPU
            # and nothing else runs beside it, so every CTA is resident all the same)
            torch.cuda.synchronize(self.device)
            native.set_mega_cooperative(0)
            self.report.phases["mega_cooperative_capture"] = "refused: ordinary launch"
            return super()._capture_decode()

    # ------------------------------------------------------------------ prefill program
    def _prefill_workspace(self) -> Workspace:
        return Workspace(self.model, self.prefill_chunk, "prefill", attn_rows=min(self.prefill_chunk, 64),
                         score_stride=self.cache.context_capacity, peer_visible=False)

    def memory_stats(self) -> dict:
        """Device memory as the allocator and the driver see it, plus what this runner knows it holds (per-request records)."""
        free, total = torch.cuda.mem_get_info(self.device)
        st = self.state
        return {
            "device_total_bytes": int(total), "device_free_bytes": int(free),
            "torch_allocated_bytes": int(torch.cuda.memory_allocated(self.device)),
            "torch_peak_allocated_bytes": int(torch.cuda.max_memory_allocated(self.device)),
            "weights_bytes": int(self.model.w.bytes_resident),
            "kv_cache_bytes": int(st.kv_cache.numel() * st.kv_cache.element_size()),
            "index_cache_bytes": int(st.index_cache.numel() * st.index_cache.element_size()),
            "staging_bytes": int(self.peer._total) if self.peer.world > 1 else 0,
            "kv_layout": self.kv_layout,
            "fallbacks": dict(self.model.fallbacks),  # library routines taken in place of the hand-written kernels, with counts
        }

    def synthetic_context(self, lane: int, depth: int, seed: int = 0) -> None:
        """Benchmarks only: make ``lane`` look ``depth`` tokens deep without running a prefill.

        The lane's cache rows are filled with random bf16 values (a normalized latent and a rotated key have this
        scale), its position is set to ``depth`` and it is activated; decode steps then cost what they cost at that
        depth (indexer scoring over ``depth`` keys, top-k, 2,048 selected rows), which a short prompt does not show.
        """
        if not 0 < depth < self.cache.context_capacity:
            raise ValueError("depth does not fit the context capacity")
        st = self.state
        with torch.cuda.device(self.device):
            native.fill_random_bf16(st.kv_cache[lane], seed * 2 + 1, 0.0, 0.5)
            native.fill_random_bf16(st.index_cache[lane], seed * 2 + 2, 0.0, 0.5)
            st.tokens[lane] = 1 + (seed % 1000)
            st.positions[lane] = depth
            st.active[lane] = 1
            torch.cuda.synchronize(self.device)

def build_runner(geometry, *, world: int = 1, rank: int = 0, device=None, checkpoint=None, seed: int = 0, expert_split: str | None = None,
                 **kwargs) -> LaneRunner:
    """Convenience constructor: shard ``checkpoint`` (a runtime-layout mapping) or random-init on the device.  The geometry says which
    model family it is."""
    from glm_tpu_b200.models import registry

    family = registry.family_of(geometry)
    if family.name != registry.GLM.name:
        return family.build_runner(geometry, world=world, rank=rank, device=device, checkpoint=checkpoint, seed=seed, **kwargs)
    from glm_tpu_b200.models.glm_moe_dsa.weights import random_device_weights, shard_checkpoint

    device = torch.device(device if device is not None else f"cuda:{torch.cuda.current_device()}")
    if expert_split is None and checkpoint is not None and "__expert_split__" in checkpoint:
        expert_split = checkpoint["__expert_split__"]  # a packed checkpoint was cut one way: the layout follows it
    layout = ParallelLayout(geometry, world, rank, expert_split or default_expert_split(geometry, world))
    with torch.cuda.device(device):
        weights = shard_checkpoint(checkpoint, layout, device) if checkpoint is not None else random_device_weights(layout, device, seed)
    return GpuModelRunner(weights, **kwargs)
