"""Recurrent state of a lane: everything a layer carries from token to token besides keys and values (scan states, the last
inputs of causal convolutions), in two versions per lane.

A step reads a lane's current version and writes the other one, so the kernels of a step see the state before it wherever
they read it, a repeated launch gives the same result, and the latest step of a lane can be undone: when a sequence continues
at a position inside that step (rejected speculative rows), the rows before the position are run again from the version the
step started with.  A lane that starts at position 0 reads no version at all (zeros), so freed lanes need no clearing.
"""
from __future__ import annotations

from dataclasses import dataclass, field

import torch


@dataclass
class _Lane:
    rows: int = 0                 # positions the current version stands for
    version: int = 0
    start: int = 0                # where the latest step began ...
    start_slot: int = -1          # ... and the version slot it read (-1: zeros)
    tokens: list[int] = field(default_factory=list)      # ... and the tokens it ran


@dataclass
class Advance:
    """One segment's part in a step: read slot ``src``, write slot ``dst``, after running ``replay`` tokens again first."""
    lane: int
    start: int
    src: int
    dst: int
    version: int
    replay: list[int]


class StateSlots:
    def __init__(self, lanes: int, device):
        self.lanes, self.device = [_Lane() for _ in range(lanes)], device
        self.tensors: dict[str, torch.Tensor] = {}

    def add(self, name: str, shape: tuple[int, ...], dtype: torch.dtype) -> torch.Tensor:
        t = torch.zeros((2 * len(self.lanes), *shape), dtype=dtype, device=self.device)
        self.tensors[name] = t
        return t

    def rows(self, lane: int) -> int:
        return self.lanes[lane].rows

    def plan(self, lane: int, pos: int) -> Advance:
        """How a step that begins at ``pos`` continues this lane."""
        s = self.lanes[lane]
        if pos == 0:
            return Advance(lane, 0, -1, 2 * lane + (s.version ^ 1), s.version ^ 1, [])
        if pos == s.rows:
            return Advance(lane, pos, 2 * lane + s.version, 2 * lane + (s.version ^ 1), s.version ^ 1, [])
        if s.start <= pos < s.rows:
            return Advance(lane, s.start, s.start_slot, 2 * lane + s.version, s.version, s.tokens[:pos - s.start])
        raise ValueError(f"lane {lane} holds {s.rows} positions (latest step from {s.start}): a recurrent state cannot continue at {pos}")

    def commit(self, adv: Advance, tokens: list[int]) -> None:
        """``tokens``: all that the step ran for the lane, from ``adv.start`` on."""
        s = self.lanes[adv.lane]
        s.start, s.start_slot, s.tokens = adv.start, adv.src, list(tokens)
        s.rows, s.version = adv.start + len(tokens), adv.version

    def reset(self, lane: int) -> None:
        self.lanes[lane] = _Lane(version=self.lanes[lane].version)

    def nbytes(self) -> int:
        return sum(t.numel() * t.element_size() for t in self.tensors.values())
