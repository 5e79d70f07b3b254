"""Decoder of pre-norm sublayers (architecture "Retuvik"): a layer is RWKV-style time mixing, or attention with a distance bias
over a window, and a dense xIELU or routed feed-forward, or none; norms work on groups of a row.  A stretch of layers may
run several times: every pass takes the embedding in again (but the first) and a vector of its own.

On the device, per sublayer: one launch for everything between two sublayers (``residual_step``: the result's sum, at the
start of a pass the embedding and the pass's vector, the next norm, for single rows also the mixes with the row before) -> the
sublayer's products and kernels.  A sublayer therefore hands on what is still to be added instead of adding it; the first
step also is the embedding."""

from __future__ import annotations

import torch

from ..attention.impls.segments import segment_metadata
from ..metal import get_ops
from .dense import SideBySideLinear, StackedLinear
from .experts import RoutedExperts
from .hybrid import HybridModel
from .hybrid_config import HybridArgs
from .mixers import MIXERS


class XieluFeedForward:
    def __init__(self, ff: int, width: int, get, dtype, device) -> None:
        self.up = StackedLinear({"up": get("up", (ff, width))}, dtype, device, bias=get("up.b", (ff,)))
        self.down = SideBySideLinear({"down": get("down", (width, ff))}, dtype, device)
        self.down_bias = get("down.b", (width,)).to(device=device, dtype=torch.float32)
        p, q = torch.nn.functional.softplus(get("act", (2,)).to(device="cpu", dtype=torch.float64)).tolist()
        self.act = (p, 0.5 + q)

    def __call__(self, h: torch.Tensor) -> dict:
        y = self.down.operand(h.shape[0])
        get_ops().mixer_finish(y, 0, self.up.split(self.up(h))["up"], act="xielu", act_weights=self.act)
        return {"y": self.down(y), "bias": self.down_bias}


class PreNormLayer:
    """The weights of one layer."""

    def __init__(self, args: HybridArgs, index: int, get, dtype, device) -> None:
        layer, w = args.owners()[index], args.width
        own = f"l{index}."
        f32 = lambda name, *shape: get(own + name, shape).to(device=device, dtype=torch.float32)  # noqa: E731
        mlp = lambda name, shape: get(f"{own}mlp.{name}", tuple(shape))  # noqa: E731
        self.step = dict(eps=args.eps, dtype=dtype, groups=args.norm_groups)
        self.dtype = dtype
        self.norm1 = f32("norm1", w)
        self.mixer = MIXERS[type(layer.mixer)](layer.mixer, w, args.eps,
                                               lambda name, shape: get(f"{own}mix.{name}", tuple(shape)), dtype, device)
        ins, out = self.mixer.take_weights()
        self.input = StackedLinear(ins, dtype, device) if ins else None
        self.output = SideBySideLinear({"mix": out}, dtype, device)
        self.feed = None
        if layer.routed is not None:
            self.feed = RoutedExperts(layer.routed, w, mlp, dtype, device)
        elif layer.ff:
            self.feed = XieluFeedForward(layer.ff, w, mlp, dtype, device)
        self.norm2 = f32("norm2", w) if self.feed is not None else None

    def _parts(self, x: torch.Tensor, result, taken_in: dict, meta, cache, index: int) -> dict[str, torch.Tensor]:
        ops, mu = get_ops(), self.mixer.mix_weight
        step = self.step | taken_in
        if mu is None:
            return self.input.split(self.input(ops.residual_step(x, result, self.norm1, **step)))
        last = cache.states[index].last
        if meta.max_q_len == 1:  # one row a request: the mixes are part of the step
            return self.mixer.project(ops.residual_step(x, result, self.norm1, mix=(mu, last), seg=meta, **step))
        h = ops.residual_step(x, result, self.norm1, wide=True, **step)
        return self.mixer.project(ops.token_mix(h, mu, last, meta, self.dtype))

    def run_mixer(self, x: torch.Tensor, result, taken_in: dict, meta, cache, index: int) -> dict:
        """``taken_in``: what joins the stream ahead of the layer."""
        parts = self._parts(x, result, taken_in, meta, cache, index)
        y = self.output.operand(x.shape[0])
        self.mixer.run(parts, None, meta, cache, index, y, 0)
        return {"y": self.output(y)}

    def run_feed_forward(self, x: torch.Tensor, result) -> dict:
        return self.feed(get_ops().residual_step(x, result, self.norm2, **self.step))


class PreNormModel(HybridModel):
    layer_class = PreNormLayer

    def __init__(self, args: HybridArgs, get, dtype: torch.dtype = torch.bfloat16, device="cuda") -> None:
        super().__init__(args, get, dtype, device)
        self.passes = dict(args.passes)
        self.loop_step = None
        if self.passes:
            self.loop_step = get("loop.step", (args.loop_times, args.width)).to(device=device, dtype=torch.float32).contiguous()

    def taken_in(self, index: int, input_ids: torch.Tensor) -> dict:
        """What joins the stream ahead of a layer run: the embedding, of which the stream starts, and again with every later
        pass of the loop; a pass's vector."""
        number = self.passes.get(index)
        out = {}
        if index == 0 or (number or 0) > 0:
            out["embed"] = (input_ids, self.embed, self.args.embedding_scale, index == 0)
        if number is not None:
            out["add"] = self.loop_step[number]
        return out

    def forward(self, input_ids: torch.Tensor, ctx, cache, meta=None, logits_rows=None) -> torch.Tensor:
        if meta is None:
            meta = segment_metadata(ctx, cache.block_size, self.device)
        ops, a = get_ops(), self.args
        x = torch.empty((input_ids.shape[0], a.width), dtype=torch.float32, device=self.device)
        result = None
        for i, layer in enumerate(self.layers):
            result = layer.run_mixer(x, result, self.taken_in(i, input_ids), meta, cache, i)
            if layer.feed is not None:
                result = layer.run_feed_forward(x, result)
            if self.residual_hook is not None:
                ops.residual_step(x, result, eps=a.eps, dtype=self.dtype)
                self.residual_hook(i, x)
                result = None
        if logits_rows is not None and logits_rows.shape[0] == 0:
            return torch.empty((0, a.vocab), dtype=torch.float32, device=self.device)
        return self.head(ops.residual_step(x, result, self.final_norm, eps=a.eps, dtype=self.dtype, rows=logits_rows,
                                           groups=a.norm_groups))

    __call__ = forward
