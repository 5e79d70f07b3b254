"""Per-request state of recurrent layers: fixed-size slots in HBM plus the allocator that hands them out.

A slot holds everything a request carries from step to step in every recurrent layer (32-bit matrix states, the
normaliser and running maximum of mLSTM, the last inputs of a short convolution, the last input of time mixing).  Nothing is cleared when a slot
changes hands: the kernels take a segment that starts at position 0 as having a zero state.  Slot 0 is the padding
slot (graph warm-up and padded rows write there), like block 0 of the paged pools.
"""

from __future__ import annotations

from dataclasses import dataclass

import torch

from ...metal.hybrid_ops import RECURRENCE_TILE_V


class StateSlots:
    """Slot ids 1..n by request id."""

    def __init__(self, num_slots: int) -> None:
        self.num_slots = num_slots
        self._free = list(range(num_slots, 0, -1))
        self._of: dict[str, int] = {}

    def acquire(self, req_id: str) -> int:
        slot = self._of.get(req_id)
        if slot is None:
            if not self._free:
                raise RuntimeError(f"all {self.num_slots} state slots are in use")
            slot = self._of[req_id] = self._free.pop()
        return slot

    def release(self, req_id: str) -> None:
        slot = self._of.pop(req_id, None)
        if slot is not None:
            self._free.append(slot)

    def __contains__(self, req_id: str) -> bool:
        return req_id in self._of

    @property
    def num_free(self) -> int:
        return len(self._free)


@dataclass
class RecurrentState:
    """The slots of one layer (row 0 is the padding slot); fields a mixer does not use are ``None``."""

    matrix: torch.Tensor                    # fp32 [slots, heads, key_dim, value_dim]
    normaliser: torch.Tensor | None = None  # fp32 [slots, heads, value tiles, key_dim]
    maximum: torch.Tensor | None = None     # fp32 [slots, heads, value tiles]
    conv: torch.Tensor | None = None        # [slots, taps - 1, channels], the activation type
    last: torch.Tensor | None = None        # fp32 [slots, width]

    @classmethod
    def allocate(cls, num_slots: int, heads: int, key_dim: int, value_dim: int, device, *, normalised: bool = False,
                 conv_taps: int = 0, conv_channels: int = 0, dtype: torch.dtype = torch.bfloat16,
                 last: int = 0) -> RecurrentState:
        n = num_slots + 1
        f32 = dict(dtype=torch.float32, device=device)
        tiles = -(-value_dim // RECURRENCE_TILE_V)
        return cls(torch.zeros((n, heads, key_dim, value_dim), **f32),
                   torch.zeros((n, heads, tiles, key_dim), **f32) if normalised else None,
                   torch.zeros((n, heads, tiles), **f32) if normalised else None,
                   torch.zeros((n, conv_taps - 1, conv_channels), dtype=dtype, device=device) if conv_taps else None,
                   torch.zeros((n, last), **f32) if last else None)

    @property
    def nbytes(self) -> int:
        return sum(t.numel() * t.element_size() for t in (self.matrix, self.normaliser, self.maximum, self.conv, self.last)
                   if t is not None)
