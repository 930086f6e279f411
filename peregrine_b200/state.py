"""What live sequences carry from step to step: slots, and the tensors that hold every slot's part of a layer's cache or
state.  A layer asks for its tensors once (`SlotPool.tensor`), the engine hands slots out and takes them back.

A slot is not cleared when it changes hands: kernels take the recurrent state and the convolution inputs of a sequence
as zero at position 0, and attention reads no position that the sequence has not written."""
from __future__ import annotations

from typing import List


class OutOfSlots(RuntimeError):
    pass


class SlotPool:
    def __init__(self, slots: int, capacity: int, device):
        """slots: most sequences alive at once; capacity: most positions of one sequence."""
        self.slots, self.capacity, self.device = int(slots), int(capacity), device
        self._free: List[int] = list(range(self.slots))
        self._live = set()
        self.bytes = 0

    def tensor(self, shape, dtype):
        """A zeroed tensor with one entry per slot in front: [slots, *shape]."""
        import torch

        t = torch.zeros((self.slots, *shape), dtype=dtype, device=self.device)
        self.bytes += t.numel() * t.element_size()
        return t

    def take(self) -> int:
        if not self._free:
            raise OutOfSlots(f"all {self.slots} slots are in use")
        s = self._free.pop(0)
        self._live.add(s)
        return s

    def give_back(self, slot: int) -> None:
        self._live.remove(slot)
        self._free.append(slot)

    @property
    def free(self) -> int:
        return len(self._free)
