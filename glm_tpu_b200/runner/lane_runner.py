"""What every model runner shares: lanes, the CUDA-graph decode program, the prefill program, feeding and reading tokens.

A family's runner (``GpuModelRunner`` for GLM-MoE-DSA, ``NamizenRunner``) builds the model, the caches and the workspaces; the engine drives
the interface below and never sees a difference.  The model object has two entry points,

    run_rows(ws, state, tokens, row_pos, row_lane, row_active, rows, decode=..., max_ctx=..., head_rows=..., head=..., lane_of_rows=...)
    sample(ws, state, logits, rows, row_active, advance=..., ...)

the state begins with ``LaneRegisters``, and the cache configuration knows its ``context_capacity``.

Parity: reference ``glm_tpu/runner/tpu_runner.py:29-289`` (load phases, program set, batch programs), ``runner/programs.py:80-118``,
``runner/compilation_manager.py:28-69`` (here a program is a captured CUDA graph instead of a compiled XLA executable).
"""

from __future__ import annotations

import time
from dataclasses import dataclass, field

import torch

from glm_tpu_b200.runner.admission import check_collective_plan
from glm_tpu_b200.runner.lane_state import RING


@dataclass
class ProgramRecord:
    name: str
    kind: str  # 'cuda_graph' or 'eager'
    rows: int
    launches: int
    capture_seconds: float = 0.0


@dataclass
class RunnerReport:
    phases: dict = field(default_factory=dict)
    programs: list = field(default_factory=list)
    memory: dict = field(default_factory=dict)


class _LaunchCounter:
    """Counts kernel launches issued through the native library while a program is being recorded."""

    def __init__(self):
        self.count = 0

    def __enter__(self):
        from glm_tpu_b200.ops import native

        self._native = native
        self._orig = native._check

        def counting(code, what):
            self.count += 1
            self._orig(code, what)

        native._check = counting
        return self

    def __exit__(self, *exc):
        self._native._check = self._orig


class LaneRunner:
    """Set by the family's constructor before ``_ready``: ``model``, ``state``, ``cache``, ``peer``, ``decode_ws``, ``device``, ``world``,
    ``rank``, ``lanes``, ``prefill_chunk``, ``use_graphs``, ``report``."""

    decode_path = "kernels"

    def _ready(self) -> None:
        """The part of the construction that follows the model: program slots, counters, the prefill's output register."""
        with torch.cuda.device(self.device):
            self.prefill_ws = None
            self._prefill_out = torch.zeros(1, dtype=torch.int32, device=self.device)
            self._graph = None
            self._graph_stream = torch.cuda.Stream(device=self.device)
        self.decode_launches = 0
        self.steps_issued = 0
        self._feed_host = None
        self.fed_bytes_per_step = 0
        self.lengths = [0] * self.lanes  # tokens each lane has cached, as far as ``open_lane`` / ``extend`` / ``decode_logits`` drove it

    # ------------------------------------------------------------------ decode program
    def _decode_body(self) -> None:
        st, ws, m = self.state, self.decode_ws, self.model
        logits = m.run_rows(ws, st, st.tokens, st.positions, st.lane_ids, st.active, self.lanes, decode=True,
                            max_ctx=self.cache.context_capacity, head="argmax")
        m.sample(ws, st, logits, self.lanes, st.active, advance=3)

    def _captures_graphs(self) -> bool:
        return self.use_graphs

    def _capture_decode(self) -> torch.cuda.CUDAGraph:
        graph = torch.cuda.CUDAGraph()
        with torch.cuda.graph(graph, stream=self._graph_stream):
            self._decode_body()
        return graph

    def build_decode_program(self) -> ProgramRecord:
        """Warm up eagerly (lanes inactive: no cache write, no advance), then capture the step in a CUDA graph."""
        t0 = time.perf_counter()
        with torch.cuda.device(self.device):
            saved = self.state.active.clone()
            self.state.active.zero_()
            from glm_tpu_b200.ops import native

            with _LaunchCounter() as counter, native.record_exchanges() as plan:
                self._decode_body()
            self.decode_launches = counter.count
            # the cross-GPU exchanges of the step, in launch order, against the rules the in-kernel protocol rests on (alternating
            # all-reduce channels, a signal at most once between two all-reduces, payloads within the slots): refused before capture
            check_collective_plan(plan, world=self.peer.world)
            self.report.phases["collective_plan"] = {"exchanges": len(plan), "allreduces": sum(1 for op in plan if op["kind"] == "allreduce")}
            torch.cuda.synchronize(self.device)
            kind = "eager"
            if self._captures_graphs():
                self._graph = self._capture_decode()
                kind = "cuda_graph"
            self.state.active.copy_(saved)
            self.state.step_counter.zero_()
            self.steps_issued = 0
            torch.cuda.synchronize(self.device)
            self.peer.check_status()
        rec = ProgramRecord("decode:" + self.decode_path, kind, self.lanes, self.decode_launches, time.perf_counter() - t0)
        self.report.programs.append(rec)
        return rec

    def decode_step(self) -> None:
        """Enqueue one decode step for every active lane (asynchronous)."""
        if self._graph is None and not self.report.programs:
            self.build_decode_program()
        if self._graph is not None:
            self._graph.replay()
        else:
            self._decode_body()
        self.steps_issued += 1

    def feed_tokens(self, tokens: dict) -> None:
        """Copy the committed tokens of the given lanes (``lane -> token``) from pinned host memory into the device's token
        registers (asynchronous, on the current stream: the next decode step reads them).  4 bytes per lane; a lane that is not
        named keeps being fed what it was fed last, which a frozen lane never uses."""
        if self._feed_host is None:
            self._feed_host = torch.zeros(self.lanes, dtype=torch.int32).pin_memory()
        for lane, token in tokens.items():
            self._feed_host[lane] = int(token)
        with torch.cuda.device(self.device):
            self.state.tokens.copy_(self._feed_host, non_blocking=True)
        self.fed_bytes_per_step = 4 * self.lanes

    def read_last_tokens(self) -> list[int]:
        """Tokens of the most recent decode step, one per lane (-1 for a frozen lane).  Synchronizes."""
        return self.read_step_tokens(self.steps_issued - 1)

    def read_status(self) -> int:
        """The device status word (0 = clean); reading clears it."""
        return self.peer.read_status()

    def read_step_tokens(self, step_index: int) -> list[int]:
        """Tokens produced by decode step ``step_index`` (synchronizes; one small D2H copy)."""
        row = self.state.out_tokens[step_index % RING].cpu()
        return [int(v) for v in row]

    # ------------------------------------------------------------------ prefill program
    def _prefill_workspace(self):
        """The family's workspace for ``prefill_chunk`` rows of one lane."""
        raise NotImplementedError

    def _ensure_prefill_ws(self):
        if self.prefill_ws is None:
            with torch.cuda.device(self.device):
                self.prefill_ws = self._prefill_workspace()
        return self.prefill_ws

    def _chunks(self, lane: int, token_ids, first: int, head_rows):
        """Push ``token_ids`` through ``lane`` from position ``first`` on, ``prefill_chunk`` rows at a time.  ``head_rows(start, rows)``
        names the rows of a chunk (counted from ``first``) whose logits are computed; yields ``(start, logits)`` per chunk."""
        n = len(token_ids)
        ws, st, m = self._ensure_prefill_ws(), self.state, self.model
        ids = torch.as_tensor(list(token_ids), dtype=torch.int32).pin_memory().to(self.device, non_blocking=True)
        lane_t = torch.full((self.prefill_chunk,), lane, dtype=torch.int32, device=self.device)
        for start in range(0, n, self.prefill_chunk):
            rows = min(self.prefill_chunk, n - start)
            pos = torch.arange(first + start, first + start + rows, dtype=torch.int32, device=self.device)
            yield start, m.run_rows(ws, st, ids[start : start + rows], pos, lane_t, None, rows, decode=False, max_ctx=first + start + rows,
                                    head_rows=head_rows(start, rows), lane_of_rows=lane)

    def prefill(self, lane: int, token_ids) -> int:
        """Run a prompt through ``lane`` with a fresh cache; returns the first generated token.

        After the call the lane is active, its position is ``len(token_ids)`` and its next input is that token.
        """
        n = len(token_ids)
        if not 0 < n < self.cache.context_capacity:
            raise ValueError("prompt does not fit the context capacity")
        st, m = self.state, self.model
        with torch.cuda.device(self.device):
            st.reset_lane(lane)
            logits = None
            for _, logits in self._chunks(lane, token_ids, 0, lambda start, rows: slice(rows - 1, rows) if start + rows == n else slice(0, 1)):
                pass
            m.sample(self.prefill_ws, st, logits, 1, None, advance=1, tokens_out=st.tokens[lane : lane + 1],
                     positions=st.positions[lane : lane + 1], out=self._prefill_out)
            st.positions[lane] = n
            st.active[lane] = 1
            self.lengths[lane] = n
            token = int(self._prefill_out.cpu()[0])
            self.peer.check_status()
        return token

    # ------------------------------------------------------------------ given tokens, logits out
    def open_lane(self, lane: int) -> None:
        """A new request on ``lane`` whose tokens will be given to ``extend`` and ``decode_logits``."""
        with torch.cuda.device(self.device):
            self.state.reset_lane(lane)
        self.lengths[lane] = 0

    def extend(self, lane: int, token_ids, want=()) -> torch.Tensor:
        """Run the next tokens of ``lane`` through the prefill program, from the cache that earlier calls left.  Returns the logits at
        the places ``want`` (indices into ``token_ids``) as fp32 ``[len(want), vocab]`` on the CPU, in the order of ``want``."""
        n, first = len(token_ids), self.lengths[lane]
        want = [int(w) for w in want]
        if not n or first + n > self.cache.context_capacity or any(not 0 <= w < n for w in want):
            raise ValueError("the tokens do not fit the context capacity, or a wanted place is not among them")
        out = [None] * len(want)

        def rows_of(start, rows):
            picked = [w - start for w in want if start <= w < start + rows]
            return torch.as_tensor(picked, dtype=torch.int64, device=self.device) if picked else slice(0, 1)

        with torch.cuda.device(self.device):
            for start, logits in self._chunks(lane, token_ids, first, rows_of):
                slots = [i for i, w in enumerate(want) if start <= w < start + self.prefill_chunk]
                if slots:
                    rows = logits.float().cpu()
                    for row, i in enumerate(slots):
                        out[i] = rows[row]
            self.lengths[lane] = first + n
            self.state.positions[lane] = first + n
            self.peer.check_status()
        return torch.stack(out) if out else torch.empty((0, self.g.vocab_size))

    def decode_logits(self, tokens: dict) -> dict:
        """One step of the decode program's kernels for the lanes of ``tokens`` (``lane -> its next token``; every other lane is frozen),
        with the logits kept: ``lane -> fp32 [vocab]`` on the CPU."""
        if any(self.lengths[lane] >= self.cache.context_capacity for lane in tokens):
            raise ValueError("a lane is at the end of its context")
        st, m = self.state, self.model
        with torch.cuda.device(self.device):
            st.active.copy_(torch.tensor([1 if lane in tokens else 0 for lane in range(self.lanes)], dtype=torch.int32))
            self.feed_tokens(tokens)
            logits = m.run_rows(self.decode_ws, st, st.tokens, st.positions, st.lane_ids, st.active, self.lanes, decode=True,
                                max_ctx=self.cache.context_capacity, head="logits")
            rows = logits.float().cpu()
            m.sample(self.decode_ws, st, logits, self.lanes, st.active, advance=2)
            self.steps_issued += 1  # the step took its place in the ring of produced tokens
            self.peer.check_status()
        for lane in tokens:
            self.lengths[lane] += 1
        return {lane: rows[lane] for lane in tokens}

    def deactivate(self, lane: int) -> None:
        self.state.active[lane] = 0

    def close(self) -> None:
        self._graph = None
        if self.peer.world > 1:
            torch.cuda.synchronize(self.device)
            self.peer.check_canaries()  # a kernel (of any rank) that overran a staging region wrote into its guard band
        self.peer.close()
