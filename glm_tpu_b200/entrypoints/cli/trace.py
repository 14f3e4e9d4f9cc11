"""``trace``: replay given token ids through a model, step by step, and write the logits.  Nothing is sampled.

Steps are read from standard input, one JSON object a line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": ["b"]}

Every entry brings the next tokens of a request; ``want`` lists the places among them whose logits are written, ``end`` the requests that
are over after the step (their lane is given back).  The logits of a step go to ``<out>/<step>.f32``: little-endian fp32, ``[wanted, vocab]``,
in the order of the entries and of ``want``; a step in which nothing is wanted writes no file.  After every step a line ``done <step>``
is printed.

The requests run on the engine's own lanes: a request's later single tokens go through the decode program's kernels (those of one step
together, one lane each), everything else through the prefill program, both from the cache that earlier steps left.

Exit status 3: the model has no path in the asked-for number format.
"""

from __future__ import annotations

import json
import sys
from pathlib import Path

from glm_tpu_b200.exceptions import RequestValidationError

LANES = 4
PREFILL_CHUNK = 2048


class TraceReplay:
    """Requests by name on the lanes of a runner.  The runner needs ``lanes``, ``lengths``, ``open_lane``, ``extend`` and ``decode_logits``."""

    def __init__(self, runner):
        self.runner = runner
        self.free = list(range(runner.lanes))
        self.lane_of: dict[str, int] = {}

    def _lane(self, name: str) -> int:
        if name not in self.lane_of:
            if not self.free:
                raise RequestValidationError(f"more than {self.runner.lanes} requests are live")
            self.lane_of[name] = self.free.pop(0)
            self.runner.open_lane(self.lane_of[name])
        return self.lane_of[name]

    def step(self, command: dict) -> list:
        """Run one step; returns the wanted logits as a list of fp32 rows."""
        entries = command["entries"]
        names = [e["id"] for e in entries]
        if len(set(names)) != len(names):
            raise RequestValidationError("a request has two entries in one step")
        lanes = [self._lane(name) for name in names]
        single = {lane: e["tokens"][0] for lane, e in zip(lanes, entries) if len(e["tokens"]) == 1 and self.runner.lengths[lane] > 0}
        decoded = self.runner.decode_logits(single) if single else {}
        rows = []
        for lane, entry in zip(lanes, entries):
            if lane in decoded:
                rows += [decoded[lane] for _ in entry["want"]]
            else:
                rows += list(self.runner.extend(lane, entry["tokens"], entry["want"]))
        for name in command.get("end", ()):
            self.free.append(self.lane_of.pop(name))
        return rows


def write_rows(path: Path, rows) -> None:
    import torch

    torch.stack(list(rows)).contiguous().numpy().astype("<f4", copy=False).tofile(path)


def replay(runner, lines, out: Path, emit=print) -> None:
    session = TraceReplay(runner)
    for line in lines:
        if not line.strip():
            continue
        command = json.loads(line)
        rows = session.step(command)
        if rows:
            write_rows(out / f"{int(command['step'])}.f32", rows)
        emit(f"done {int(command['step'])}", flush=True)


def main(args) -> int:
    from glm_tpu_b200.models import registry

    geometry, (kind, path) = registry.resolve_model(str(args.model))
    family = registry.family_of(geometry)
    if args.dtype not in family.dtypes:
        print(f"{family.architecture} runs in {', '.join(family.dtypes)} only", file=sys.stderr)
        return 3
    import torch

    from glm_tpu_b200.csrc.build import build
    from glm_tpu_b200.ops import native
    from glm_tpu_b200.runner.gpu_runner import build_runner

    native.select_library(build(component=family.library_component))
    device = torch.device("cuda", 0)
    capacity = -(-max(args.max_tokens, 1) // 64) * 64
    options = {"dtype": torch.float32} if args.dtype == "float32" else {}
    checkpoint = family.load_checkpoint(path, 0, 1, device=device) if kind == "checkpoint" else None
    runner = build_runner(geometry, device=device, checkpoint=checkpoint, context_capacity=capacity, lanes=LANES,
                          prefill_chunk=min(PREFILL_CHUNK, capacity), **options)
    try:
        replay(runner, sys.stdin, Path(args.out))
    finally:
        runner.close()
    return 0
