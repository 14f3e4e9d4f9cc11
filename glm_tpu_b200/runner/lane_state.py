"""The lane registers every model family's device state begins with.

A lane is one live request.  Its registers live in device memory so that a captured decode step replays unchanged: the token each lane feeds
next, its position (= tokens already cached), whether it is active, and a ring of the tokens produced by the last steps.

Parity: reference ``glm_tpu/models/glm_moe_dsa/state.py:23-69``.
"""

from __future__ import annotations

from dataclasses import dataclass

import torch

RING = 64


@dataclass
class LaneRegisters:
    tokens: torch.Tensor  # [lanes] int32: the token each lane feeds next
    positions: torch.Tensor  # [lanes] int32: its position (= tokens already cached)
    active: torch.Tensor  # [lanes] int32
    lane_ids: torch.Tensor  # [lanes] int32 arange
    out_tokens: torch.Tensor  # [RING, lanes] int32
    step_counter: torch.Tensor  # [1] int32

    @staticmethod
    def registers(lanes: int, device) -> dict:
        z = lambda *s: torch.zeros(s, dtype=torch.int32, device=device)  # noqa: E731
        return dict(tokens=z(lanes), positions=z(lanes), active=z(lanes), lane_ids=torch.arange(lanes, dtype=torch.int32, device=device),
                    out_tokens=torch.full((RING, lanes), -1, dtype=torch.int32, device=device), step_counter=z(1))

    def reset_lane(self, lane: int) -> None:
        """Fresh cache for a new request on ``lane`` (stale rows are never read: reads are bounded by the position)."""
        self.positions[lane] = 0
        self.tokens[lane] = 0
        self.active[lane] = 0
