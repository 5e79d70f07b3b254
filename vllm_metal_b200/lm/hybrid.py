"""Decoder whose layers mix latent attention, Mamba-2 and mLSTM (architecture "Mapuvik"), over the C-ABI kernels.

A layer is parallel: one norm feeds the mixer and the feed-forward, and both add to the fp32 residual stream.  On the
device that is: norm -> ONE product for every projection of the norm's output -> the mixer's kernels, whose last one
also applies the feed-forward's activation -> ONE product that adds both halves into the stream.  Layers with
``weights_of`` share the weights object of their owner; what they keep between steps is theirs.

``forward`` has the signature of ``decoder.Model``, so the runner drives both alike."""

from __future__ import annotations

import torch

from ..attention.impls.segments import segment_metadata
from ..metal import get_ops
from .dense import DenseHead, SideBySideLinear, StackedLinear, pin_matmul_precision
from .hybrid_config import HybridArgs
from .mixers import MIXERS


class ParallelLayer:
    """The weights of one layer."""

    def __init__(self, args: HybridArgs, index: int, get, dtype, device) -> None:
        layer = args.owners()[index]
        own = f"l{index}."
        self.norm = get(own + "norm1", (args.width,)).to(device=device, dtype=torch.float32)
        self.mixer = MIXERS[type(layer.mixer)](layer.mixer, args.width, args.eps,
                                               lambda name, shape: get(f"{own}mix.{name}", tuple(shape)), dtype, device)
        ins, out = self.mixer.take_weights()
        outs = {"mix": out}
        if layer.ff:
            ins["mlp.up"] = get(own + "mlp.up", (layer.ff, args.width))
            outs["mlp.down"] = get(own + "mlp.down", (args.width, layer.ff))
        self.input = StackedLinear(ins, dtype, device)
        self.output = SideBySideLinear(outs, dtype, device)
        self.act_offset = self.output.offsets.get("mlp.down", 0)

    def add_to(self, x: torch.Tensor, args: HybridArgs, meta, cache, index: int) -> None:
        h = get_ops().stream_norm(x, self.norm, args.eps, 1.0, self.input.weight.dtype)
        parts = self.input.split(self.input(h))
        y = self.output.operand(x.shape[0])
        self.mixer.run(parts, parts.get("mlp.up"), meta, cache, index, y, self.act_offset)
        self.output.add_into(x, y)


class HybridModel:
    """``forward(input_ids [T], ctx | meta, cache) -> fp32 logits`` for the packed batch."""

    stateful = True   # the runner gives every segment a state slot
    vocab_parallel = False
    layer_class = ParallelLayer

    def __init__(self, args: HybridArgs, get, dtype: torch.dtype = torch.bfloat16, device="cuda") -> None:
        """``get(name, shape)`` returns a checkpoint tensor of that shape (or raises); a size of None is the tensor's own."""
        if dtype not in (torch.bfloat16, torch.float32):
            raise ValueError(f"hybrid decoders run in bfloat16 or float32, not {dtype}")
        pin_matmul_precision()
        self.args, self.dtype, self.device = args, dtype, torch.device(device)
        self.embed = get("embed", (args.vocab, args.width)).to(device=device, dtype=dtype).contiguous()
        owned = {i: self.layer_class(args, i, get, dtype, device) for i in args.owners()}
        self.layers = [owned[layer.weights] for layer in args.layers]
        self.final_norm = get("final.norm", (args.width,)).to(device=device, dtype=torch.float32)
        self.head = DenseHead(get("head", (args.vocab, args.width)), dtype, device)
        self.residual_hook = None  # called with (layer, stream) after every layer: debugging and tests

    @classmethod
    def from_folder(cls, args: HybridArgs, folder: str, dtype, device="cuda") -> HybridModel:
        from .safetensors_io import SafetensorsFolder

        files = SafetensorsFolder(folder)

        def get(name: str, shape: tuple[int, ...]) -> torch.Tensor:
            found = files.shape(name)
            if len(found) != len(shape) or any(n is not None and n != m for n, m in zip(shape, found)):
                raise ValueError(f"{folder}: tensor '{name}' is {found}, the configuration says {tuple(shape)}")
            return files.tensor(name)

        return cls(args, get, dtype, device)

    def forward(self, input_ids: torch.Tensor, ctx, cache, meta=None, logits_rows=None) -> torch.Tensor:
        if meta is None:
            meta = segment_metadata(ctx, cache.block_size, self.device)
        x = get_ops().embed_rows(input_ids, self.embed)
        for i, layer in enumerate(self.layers):
            layer.add_to(x, self.args, meta, cache, i)
            if self.residual_hook is not None:
                self.residual_hook(i, x)
        if logits_rows is not None and logits_rows.shape[0] == 0:
            return torch.empty((0, self.args.vocab), dtype=torch.float32, device=self.device)
        x = get_ops().stream_norm(x, self.final_norm, self.args.eps, 1.0, self.dtype, rows=logits_rows)
        return self.head(x)

    __call__ = forward
