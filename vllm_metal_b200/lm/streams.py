"""Decoder of hyper-connected sublayers (architecture "Tatazen"): several copies of the residual stream, read by every
sublayer through one vector of weights and written back through a mixing matrix.  A layer is a mixer sublayer -- lightning
attention, or softmax attention and lightning attention side by side -- and a gated feed-forward; the mixer sees a
token-shifted input and every sublayer's result passes a gate of its own.

On the device, per sublayer: one launch for everything between two sublayers (``stream_step``) -> ONE product for all
projections of the sublayer's input -> the mixer's kernels -> the output product, whose result the next ``stream_step``
takes in.  A sublayer therefore hands on what is still to be added instead of adding it."""

from __future__ import annotations

import torch

from ..attention.impls.segments import segment_metadata
from ..metal import get_ops
from .dense import SideBySideLinear, StackedLinear
from .hybrid import HybridModel
from .hybrid_config import HybridArgs, SideBySideArgs
from .mixers import MIXERS


class HyperConnection:
    """How a sublayer reads the streams and what its result does to them, with the sublayer's norm and residual gate."""

    def __init__(self, args: HybridArgs, own: str, q: int, get, device) -> None:
        s, w = args.streams, args.width
        f32 = lambda name, *shape: get(own + name, shape).to(device=device, dtype=torch.float32).contiguous()  # noqa: E731
        self.reader = (f32(f"hc{q}.in", s), f32(f"norm{q}", w))
        self.writer = {"mix": f32(f"hc{q}.mix", s, s), "out_weight": f32(f"hc{q}.out", s), "gate_bias": f32(f"rg{q}.b", w)}
        self.gate_weight = get(f"{own}rg{q}", (w, w))  # belongs to a product of the layer


class Branch:
    """A mixer with its output product and, beside another one, the norm of its result."""

    def __init__(self, prefix: str, m, args: HybridArgs, own: str, get, dtype, device) -> None:
        self.prefix = prefix
        self.mixer = MIXERS[type(m)](m, args.width, args.eps,
                                     lambda name, shape: get(f"{own}mix.{prefix}{name}", tuple(shape)), dtype, device)
        ins, out = self.mixer.take_weights()
        self.weights = {prefix + name: w for name, w in ins.items()}
        self.output = SideBySideLinear({"mix": out}, dtype, device)
        self.norm = None
        if prefix:
            self.norm = get(f"{own}mix.{prefix}out", (args.width,)).to(device=device, dtype=torch.float32)

    def run(self, input_: StackedLinear, stacked: torch.Tensor, parts, meta, cache, index: int) -> torch.Tensor:
        n = len(self.prefix)
        mine = {name[n:]: t for name, t in parts.items() if name.startswith(self.prefix)}
        for name, (first, last) in self.mixer.spans.items():
            mine[name] = input_.span(stacked, self.prefix + first, self.prefix + last)
        y = self.output.operand(stacked.shape[0])
        self.mixer.run(mine, None, meta, cache, index, y, 0)
        return self.output(y)


class StreamLayer:
    """The weights of one layer."""

    def __init__(self, args: HybridArgs, index: int, get, dtype, device) -> None:
        layer = args.owners()[index]
        own = f"l{index}."
        m, w = layer.mixer, args.width
        self.eps, self.dtype = args.eps, dtype
        self.shift = get(own + "shift", (w,)).to(device=device, dtype=torch.float32)
        self.shift_taps = torch.stack([self.shift, 1.0 - self.shift]).contiguous()
        pairs = (("left.", m.left), ("right.", m.right)) if isinstance(m, SideBySideArgs) else (("", m),)
        self.branches = [Branch(prefix, b, args, own, get, dtype, device) for prefix, b in pairs]
        self.input = StackedLinear({k: t for b in self.branches for k, t in b.weights.items()}, dtype, device)
        for b in self.branches:
            b.weights = {}
        self.mix = HyperConnection(args, own, 1, get, device)
        self.gate = StackedLinear({"gate": self._take_gate(self.mix)}, dtype, device)
        self.feed = None
        if layer.ff:
            self.feed = HyperConnection(args, own, 2, get, device)
            self.up = StackedLinear({"gate": get(own + "mlp.gate", (layer.ff, w)), "up": get(own + "mlp.up", (layer.ff, w)),
                                     "rg": self._take_gate(self.feed)}, dtype, device)
            self.down = SideBySideLinear({"down": get(own + "mlp.down", (w, layer.ff))}, dtype, device)

    @staticmethod
    def _take_gate(c: HyperConnection) -> torch.Tensor:
        weight, c.gate_weight = c.gate_weight, None
        return weight

    def run_mixer(self, streams: torch.Tensor, result, meta, cache, index: int) -> dict:
        ops = get_ops()
        step = dict(eps=self.eps, dtype=self.dtype)
        previous = cache.previous[index]
        if meta.max_q_len == 1:  # one row a request: the shift is part of the step
            h, shifted = ops.stream_step(streams, result, self.mix.reader, shift=self.shift, previous=previous, seg=meta,
                                         **step)
        else:
            h, _ = ops.stream_step(streams, result, self.mix.reader, **step)
            shifted = ops.causal_conv(h, self.shift_taps, None, previous, meta, silu=False)
        stacked = self.input(shifted)
        parts = self.input.split(stacked)
        out = dict(self.mix.writer, gate=self.gate.split(self.gate(h))["gate"])
        for name, b in zip(("y", "y2"), self.branches):
            out[name] = b.run(self.input, stacked, parts, meta, cache, index)
            out[name + "_norm"] = b.norm
        return out

    def run_feed_forward(self, streams: torch.Tensor, result) -> dict:
        ops = get_ops()
        h, _ = ops.stream_step(streams, result, self.feed.reader, eps=self.eps, dtype=self.dtype)
        parts = self.up.split(self.up(h))
        y = self.down.operand(h.shape[0])
        ops.mixer_finish(y, 0, parts["gate"], act="silu", act_mul=parts["up"])
        return dict(self.feed.writer, gate=parts["rg"], y=self.down(y))


def sinusoid_frequencies(width: int) -> torch.Tensor:
    """``10000^(-2i / width)`` of every pair of columns as fp32 high and low parts ``[pairs, 2]``."""
    i = torch.arange(-(-width // 2), dtype=torch.float64)
    f = 10000.0 ** (-2.0 * i / width)
    high = f.float()
    return torch.stack([high, (f - high.double()).float()], dim=1).contiguous()


class StreamModel(HybridModel):
    layer_class = StreamLayer

    def __init__(self, args: HybridArgs, get, dtype: torch.dtype = torch.bfloat16, device="cuda") -> None:
        super().__init__(args, get, dtype, device)
        self.freq = sinusoid_frequencies(args.width).to(self.device)
        self.total = torch.ones(args.streams, dtype=torch.float32, device=self.device)

    def forward(self, input_ids: torch.Tensor, ctx, cache, meta=None, logits_rows=None) -> torch.Tensor:
        if meta is None:
            meta = segment_metadata(ctx, cache.block_size, self.device)
        ops, a = get_ops(), self.args
        streams = ops.embed_streams(input_ids, self.embed, a.streams, meta.positions, self.freq)
        result = None
        for i, layer in enumerate(self.layers):
            result = layer.run_mixer(streams, result, meta, cache, i)
            if layer.feed is not None:
                result = layer.run_feed_forward(streams, result)
            if self.residual_hook is not None:
                ops.stream_step(streams, result, eps=a.eps, dtype=self.dtype)
                self.residual_hook(i, streams.sum(1))
                result = None
        if logits_rows is not None and logits_rows.shape[0] == 0:
            return torch.empty((0, a.vocab), dtype=torch.float32, device=self.device)
        x, _ = ops.stream_step(streams, result, (self.total, self.final_norm), eps=a.eps, dtype=self.dtype, store=False,
                               rows=logits_rows)
        return self.head(x)

    __call__ = forward
