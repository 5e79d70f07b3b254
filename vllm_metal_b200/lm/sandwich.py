"""Decoder of sublayers between two norms (architecture "Kerolorn"): a layer is rotary attention over a window with kept first
tokens, fed through a short convolution, and routed experts beside a gated shared one; every sublayer's result passes a norm
of its own before it joins the fp32 residual stream.

On the device, per sublayer: one launch for everything between two sublayers (``residual_step``: the result's norm and sum,
the next norm, for single rows also the convolution) -> the sublayer's products and kernels.  A sublayer therefore hands on what
is still to be added instead of adding it."""

from __future__ import annotations

import torch

from ..attention.impls.segments import segment_metadata
from ..metal import get_ops
from .dense import SideBySideLinear, StackedLinear
from .experts import RoutedExperts
from .hybrid import HybridModel
from .hybrid_config import HybridArgs
from .mixers import MIXERS


class SandwichLayer:
    """The weights of one layer."""

    def __init__(self, args: HybridArgs, index: int, get, dtype, device) -> None:
        layer, w = args.owners()[index], args.width
        own = f"l{index}."
        f32 = lambda name, *shape: get(own + name, shape).to(device=device, dtype=torch.float32)  # noqa: E731
        self.eps, self.dtype = args.eps, dtype
        self.norm1, self.norm1b = f32("norm1", w), f32("norm1b", w)
        self.conv = f32("canon1", w, args.input_taps).t().contiguous()
        self.conv_and_input = self.conv.clone()  # of portions: the input itself is one more unit of the current tap
        self.conv_and_input[-1] += 1.0
        self.mixer = MIXERS[type(layer.mixer)](layer.mixer, w, args.eps,
                                               lambda name, shape: get(f"{own}mix.{name}", tuple(shape)), dtype, device)
        ins, out = self.mixer.take_weights()
        self.input = StackedLinear(ins, dtype, device)
        self.output = SideBySideLinear({"mix": out}, dtype, device)
        self.experts = None
        if layer.routed is not None:
            self.norm2, self.norm2b = f32("norm2", w), f32("norm2b", w)
            self.experts = RoutedExperts(layer.routed, w, lambda name, shape: get(f"{own}mlp.{name}", tuple(shape)), dtype,
                                         device)

    def run_mixer(self, x: torch.Tensor, result, meta, cache, index: int) -> dict:
        ops, previous = get_ops(), cache.previous[index]
        single = meta.max_q_len == 1  # one row a request: the convolution is part of the step
        h = ops.residual_step(x, result, self.norm1, eps=self.eps, dtype=self.dtype,
                              conv=(self.conv, previous) if single else None, seg=meta)
        if not single:
            h = ops.causal_conv(h, self.conv_and_input, None, previous, meta, silu=False)
        y = self.output.operand(h.shape[0])
        self.mixer.run(self.input.split(self.input(h)), None, meta, cache, index, y, 0)
        return {"y": self.output(y), "norm": self.norm1b}

    def run_feed_forward(self, x: torch.Tensor, result) -> dict:
        h = get_ops().residual_step(x, result, self.norm2, eps=self.eps, dtype=self.dtype)
        return self.experts(h) | {"norm": self.norm2b}


class SandwichModel(HybridModel):
    layer_class = SandwichLayer

    def __init__(self, args: HybridArgs, get, dtype: torch.dtype = torch.bfloat16, device="cuda") -> None:
        super().__init__(args, get, dtype, device)
        self.final_norm = self.final_norm * args.logit_scale  # the head is linear

    def forward(self, input_ids: torch.Tensor, ctx, cache, meta=None, logits_rows=None) -> torch.Tensor:
        if meta is None:
            meta = segment_metadata(ctx, cache.block_size, self.device)
        ops, a = get_ops(), self.args
        x = ops.embed_rows(input_ids, self.embed)
        result = None
        for i, layer in enumerate(self.layers):
            result = layer.run_mixer(x, result, meta, cache, i)
            if layer.experts is not None:
                result = layer.run_feed_forward(x, result)
            if self.residual_hook is not None:
                ops.residual_step(x, result, eps=a.eps, dtype=self.dtype)
                self.residual_hook(i, x)
                result = None
        if logits_rows is not None and logits_rows.shape[0] == 0:
            return torch.empty((0, a.vocab), dtype=torch.float32, device=self.device)
        return self.head(ops.residual_step(x, result, self.final_norm, eps=a.eps, dtype=self.dtype, rows=logits_rows))

    __call__ = forward
