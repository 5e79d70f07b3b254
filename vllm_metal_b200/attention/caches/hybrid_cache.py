"""What a hybrid decoder keeps between steps: one paged pool of latent rows per latent-attention layer (one row
``[latent | rotated key part]`` per token instead of keys and values per head), paged keys and values per layer with
softmax attention, one set of state slots per recurrent layer and, where a convolution or a token shift stands before
the mixer, the last inputs of every layer per slot.  Layers that share weights still have a pool or slots of their own."""

from __future__ import annotations

from collections.abc import Sequence

import torch

from ...lm.hybrid_config import (HybridArgs, LatentAttentionArgs, LightningArgs, Mamba2Args, MLSTMArgs,
                                SideBySideArgs, TimeMixArgs, cached_heads)
from .state_cache import RecurrentState


def _esize(dtype: torch.dtype) -> int:
    return torch.empty((), dtype=dtype).element_size()


def paged_bytes_per_token(args: HybridArgs, dtype: torch.dtype) -> int:
    return sum(args.paged_layers().values()) * _esize(dtype)


class HybridCache:
    def __init__(self, args: HybridArgs, num_blocks: int, block_size: int, num_slots: int,
                 dtype: torch.dtype = torch.bfloat16, device: torch.device | str = "cuda") -> None:
        self.args, self.num_blocks, self.block_size, self.num_slots = args, num_blocks, block_size, num_slots
        self.dtype, self.device = dtype, torch.device(device)
        self.latent: dict[int, torch.Tensor] = {}
        self.kv: dict[int, tuple[torch.Tensor, torch.Tensor]] = {}  # [blocks, block_size, kv heads, dim / vdim]
        self.states: dict[int, RecurrentState] = {}
        self.previous: dict[int, torch.Tensor] = {}                 # [slots, taps - 1, width], the activation type
        for i, layer in enumerate(args.layers):
            m = layer.mixer
            if isinstance(m, LatentAttentionArgs):
                self.latent[i] = torch.zeros((num_blocks * block_size, m.kv_rank + m.rot_dim), dtype=dtype,
                                             device=self.device)
            elif isinstance(m, Mamba2Args):
                self.states[i] = RecurrentState.allocate(num_slots, m.heads, m.state, m.vdim, self.device,
                                                         conv_taps=m.conv, conv_channels=m.conv_channels, dtype=dtype)
            elif isinstance(m, MLSTMArgs):
                self.states[i] = RecurrentState.allocate(num_slots, m.heads, m.dim, m.vdim, self.device,
                                                         normalised=True)
            elif isinstance(m, (LightningArgs, SideBySideArgs)):
                r = m.right if isinstance(m, SideBySideArgs) else m
                self.states[i] = RecurrentState.allocate(num_slots, r.heads, r.dim, r.vdim, self.device)
            elif isinstance(m, TimeMixArgs):
                self.states[i] = RecurrentState.allocate(num_slots, m.heads, m.dim, m.dim, self.device, last=args.width)
            a = cached_heads(m)
            if a is not None:
                self.kv[i] = tuple(torch.zeros((num_blocks, block_size, a.kv_heads, d), dtype=dtype, device=self.device)
                                   for d in (a.dim, a.vdim))
            if args.input_taps:
                self.previous[i] = torch.zeros((num_slots + 1, args.input_taps - 1, args.width), dtype=dtype,
                                               device=self.device)

    @staticmethod
    def state_bytes_per_slot(args: HybridArgs, dtype: torch.dtype) -> int:
        meta = HybridCache(args, 0, 1, 0, dtype, "meta")  # slot 0 alone
        return sum(s.nbytes for s in meta.states.values()) + sum(t.numel() * t.element_size() for t in meta.previous.values())

    def block_size_for_layer(self, layer_idx: int) -> int:
        return self.block_size

    def group_index_for_layer(self, layer_idx: int) -> int:
        return 0

    def copy_blocks(self, block_copies: Sequence[tuple[int, int]]) -> None:
        """Copy-on-write of pages: every source is read before any destination is written."""
        if not block_copies:
            return
        src, dst = zip(*block_copies, strict=True)
        if any(b < 0 or b >= self.num_blocks for b in (*src, *dst)) or len(set(dst)) != len(dst):
            raise RuntimeError("block copy names an out-of-range or a repeated destination block")
        s = torch.tensor(src, dtype=torch.int64, device=self.device)
        d = torch.tensor(dst, dtype=torch.int64, device=self.device)
        for pool in (*self.latent.values(), *(t for kv in self.kv.values() for t in kv)):
            pages = pool.view(self.num_blocks, self.block_size, -1)
            pages.index_copy_(0, d, pages.index_select(0, s))

    @property
    def nbytes(self) -> int:
        tensors = (*self.latent.values(), *self.previous.values(), *(t for kv in self.kv.values() for t in kv))
        return sum(t.numel() * t.element_size() for t in tensors) + sum(s.nbytes for s in self.states.values())
