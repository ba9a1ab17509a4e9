"""Per-sequence state of recurrent layers: tensors with one slot per engine batch row.

The engine zeroes a slot when a sequence opens on its row, saves and restores all slots around graph capture (a step cannot be
run twice on them), and moves single slots in and out of session snapshots.
"""

from __future__ import annotations

import torch


class RecurrentState:
    slot_dim = 0

    def __init__(self, tensors: list[torch.Tensor]) -> None:
        """``tensors``: any number, each with the slots along :attr:`slot_dim`."""
        self.tensors = list(tensors)

    def _slot(self, t: torch.Tensor, slot: int) -> torch.Tensor:
        return t.select(self.slot_dim, slot)

    def reset(self, slot: int) -> None:
        for t in self.tensors:
            self._slot(t, slot).zero_()

    def save(self) -> list[torch.Tensor]:
        return [t.clone() for t in self.tensors]

    def load(self, saved: list[torch.Tensor]) -> None:
        for t, s in zip(self.tensors, saved):
            t.copy_(s)

    def export_slot(self, slot: int) -> tuple[torch.Tensor, ...]:
        """Host copies of one slot."""
        return tuple(self._slot(t, slot).detach().cpu().clone() for t in self.tensors)

    def import_slot(self, slot: int, saved) -> None:
        for t, s in zip(self.tensors, saved):
            self._slot(t, slot).copy_(s)

    def bytes_per_slot(self) -> int:
        return sum(t.numel() // t.shape[self.slot_dim] * t.element_size() for t in self.tensors)


class LayerStates(RecurrentState):
    """fp32 state ``[slots, *shape]`` of each entry of ``shapes``: layer index, or (layer index, part) where a layer keeps several
    things, -> shape of one sequence's state."""

    def __init__(self, shapes: dict, slots: int, device) -> None:
        self.by_layer = {i: torch.zeros((slots, *shape), dtype=torch.float32, device=device) for i, shape in shapes.items()}
        super().__init__(list(self.by_layer.values()))

    def layer(self, i) -> torch.Tensor:
        return self.by_layer[i]
