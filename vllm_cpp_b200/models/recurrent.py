"""Recurrent state of models with stateful layers: one row per request slot in every tensor."""
from __future__ import annotations

import torch


class RecurrentState:
    """Tensors ``[slots, ...]`` that a step advances in place. A step that verifies draft tokens advances the
    state over all of them; when some are rejected there is nothing to subtract, so the runner restores
    the copy taken before the step and has the kept tokens run again."""

    def __init__(self):
        self.tensors: list[torch.Tensor] = []
        self._saved: list[torch.Tensor] | None = None

    def add(self, shape, dtype, device) -> torch.Tensor:
        t = torch.zeros(shape, dtype=dtype, device=device)
        self.tensors.append(t)
        return t

    def snapshot(self, slots: list) -> None:
        if not slots or not self.tensors:
            return
        if self._saved is None or len(self._saved) != len(self.tensors):
            self._saved = [torch.empty_like(t) for t in self.tensors]
        idx = torch.tensor(slots, dtype=torch.long, device=self.tensors[0].device)
        for t, s in zip(self.tensors, self._saved):
            s.index_copy_(0, idx, t.index_select(0, idx))

    def restore(self, slots: list) -> None:
        if not slots or not self.tensors:
            return
        idx = torch.tensor(slots, dtype=torch.long, device=self.tensors[0].device)
        for t, s in zip(self.tensors, self._saved):
            t.index_copy_(0, idx, s.index_select(0, idx))
