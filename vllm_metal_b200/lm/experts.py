"""Feed-forward of routed experts, where the design has it with a gated shared one beside them, over the C-ABI kernels: router product -> choice ->
sort of the (row, place) pairs -> ONE launch for the way in of all experts and the shared one -> ONE for their way out.
The weighted sum is left to whoever reads the result (the step to the next sublayer).  Nothing is read back to the host, so
the block runs under CUDA graphs."""

from __future__ import annotations

import torch

from ..metal import get_ops
from ..metal.hybrid_ops import EXPERT_TILES
from .dense import StackedLinear
from .hybrid_config import RoutedArgs


def _pad8(n: int) -> int:
    return -(-n // 8) * 8


class RoutedExperts:
    def __init__(self, r: RoutedArgs, width: int, get, dtype, device) -> None:
        """``get(name, shape)``: the block's tensors by their own names (``e0.gate`` ..., ``router``, ``shared.sg`` ...)."""
        self.r, self.width, self.dtype = r, width, dtype
        self.correction = get("router.b" if r.over_chosen else "correction", (r.experts,)).to(device=device, dtype=torch.float32).contiguous()
        heads = {"router": get("router", (r.experts, width))}
        self.way_in = torch.empty((r.experts, 2 * r.ff, width), dtype=dtype, device=device)
        self.way_out = torch.zeros((r.experts, width, _pad8(r.ff)), dtype=dtype, device=device)
        for e in range(r.experts):
            self._fill(get, f"e{e}.", r.ff, self.way_in[e], self.way_out[e])
        self.shared_in = self.shared_out = None
        if r.shared_ff:
            heads["gate"] = get("shared.sg", (1, width))
            self.shared_in = torch.empty((2 * r.shared_ff, width), dtype=dtype, device=device)
            self.shared_out = torch.zeros((width, _pad8(r.shared_ff)), dtype=dtype, device=device)
            self._fill(get, "shared.", r.shared_ff, self.shared_in, self.shared_out)
        self.router = StackedLinear(heads, dtype, device)
        # the tensor-core products take whole 16-byte units
        self.any_size = dtype != torch.bfloat16 or width % 8 != 0 or r.ff % 8 != 0 or r.shared_ff % 8 != 0

    def _fill(self, get, name: str, ff: int, way_in: torch.Tensor, way_out: torch.Tensor) -> None:
        way_in[:ff].copy_(get(name + "gate", (ff, self.width)))
        way_in[ff:].copy_(get(name + "up", (ff, self.width)))
        way_out[:, :ff].copy_(get(name + "down", (self.width, ff)))

    def tile_rows(self, rows: int) -> int:
        """Pairs per tile: few experts should need a second pass over their weights."""
        if self.any_size:
            return EXPERT_TILES[0]
        per_expert = rows * self.r.top / self.r.experts
        return next((t for t in EXPERT_TILES if t >= 2 * per_expert), EXPERT_TILES[-1])

    def __call__(self, h: torch.Tensor) -> dict:
        """``h [T, width]``: ``y [T * top, width]`` with ``part_weight [T, top]`` and the shared ``extra`` with its gate's
        logits, as ``residual_step`` takes them."""
        r, ops, t = self.r, get_ops(), h.shape[0]
        heads = self.router.split(self.router.wide(h))
        chosen, weights = ops.expert_route(heads["router"], self.correction, r.experts, r.top, r.scale, r.over_chosen)
        plan = ops.expert_plan(chosen, r.experts, self.tile_rows(t))
        act, shared_act = ops.expert_product(h, self.way_in, plan, r.top, t, gated=True, shared_weight=self.shared_in)
        y, extra = ops.expert_product(act, self.way_out, plan, r.top, t, gated=False, k=r.ff, shared_x=shared_act,
                                      shared_weight=self.shared_out, shared_k=r.shared_ff)
        out = {"y": y, "part_weight": weights}
        if extra is not None:
            out |= {"extra": extra, "extra_gate": heads["gate"][:, 0]}
        return out
