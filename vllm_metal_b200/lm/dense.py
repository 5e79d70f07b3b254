"""Dense (unquantized) linears of the hybrid decoders.  Layers that feed several projections from one input run them as
ONE product (rows of all weights stacked), and the two halves of a parallel layer leave through one product as well:
their outputs are columns of one operand, their weights lie side by side along K, and the product accumulates straight
into the fp32 residual stream.  The products themselves are plain library GEMMs (fp32 accumulation)."""

from __future__ import annotations

import torch

_ALIGN = 8  # columns: 16 bytes of a 16-bit type, what vector loads and the tensor-core GEMMs want


def pin_matmul_precision() -> None:
    """fp32 stays fp32 and 16-bit products accumulate in fp32 whatever the process had set before."""
    torch.backends.cuda.matmul.allow_tf32 = False
    torch.backends.cuda.matmul.allow_bf16_reduced_precision_reduction = False


def _up(n: int) -> int:
    return -(-n // _ALIGN) * _ALIGN


def _wide_mm(x: torch.Tensor, weight: torch.Tensor) -> torch.Tensor:
    if x.dtype == torch.float32:
        return torch.mm(x, weight.t())
    return torch.mm(x, weight.t(), out_dtype=torch.float32)


class StackedLinear:
    """``y = x W^T`` for several weights ``[out_i, in]`` that share ``x``; ``split(y)`` gives the parts as views."""

    def __init__(self, parts: dict[str, torch.Tensor], dtype: torch.dtype, device, bias: torch.Tensor | None = None) -> None:
        """``bias``: of a single part."""
        self.slices: dict[str, tuple[int, int]] = {}
        at = 0
        for name, w in parts.items():
            self.slices[name] = (at, at + w.shape[0])
            at = _up(at + w.shape[0])
        width = next(iter(parts.values())).shape[1]
        self.weight = torch.zeros((at, width), dtype=dtype, device=device)
        for name, w in parts.items():
            if w.shape[1] != width:
                raise ValueError(f"'{name}' takes {w.shape[1]} inputs, the others {width}")
            lo, hi = self.slices[name]
            self.weight[lo:hi].copy_(w)
        self.bias = None
        if bias is not None:
            self.bias = torch.zeros(at, dtype=dtype, device=device)
            self.bias[:bias.shape[0]].copy_(bias)

    def __call__(self, x: torch.Tensor) -> torch.Tensor:
        if self.bias is not None:
            return torch.addmm(self.bias, x, self.weight.t())
        return torch.mm(x, self.weight.t())

    def wide(self, x: torch.Tensor) -> torch.Tensor:
        """The product kept in fp32."""
        return _wide_mm(x, self.weight)

    def split(self, y: torch.Tensor) -> dict[str, torch.Tensor]:
        return {name: y[:, lo:hi] for name, (lo, hi) in self.slices.items()}

    def span(self, y: torch.Tensor, first: str, last: str) -> torch.Tensor:
        """The columns from part ``first`` to part ``last``, alignment padding (zeros) between them included."""
        return y[:, self.slices[first][0]:self.slices[last][1]]


class BatchedLinear:
    """``y[i] = x[i] W_i^T`` for weights ``[out, in]`` of one size, an input each: one batched product."""

    def __init__(self, weights: list[torch.Tensor], dtype: torch.dtype, device) -> None:
        self.weight = torch.empty((len(weights), *weights[0].shape), dtype=dtype, device=device)
        for own, w in zip(self.weight, weights, strict=True):
            own.copy_(w)

    def __call__(self, x: torch.Tensor) -> torch.Tensor:
        return torch.bmm(x, self.weight.transpose(1, 2))


class SideBySideLinear:
    """``x += [a | b] [W_a | W_b]^T`` with an fp32 ``x`` (``add_into``), or the product alone (a call)."""

    def __init__(self, parts: dict[str, torch.Tensor], dtype: torch.dtype, device) -> None:
        self.offsets: dict[str, int] = {}
        at = 0
        for name, w in parts.items():
            self.offsets[name] = at
            at = _up(at + w.shape[1])
        self.columns = at
        rows = next(iter(parts.values())).shape[0]
        self.weight = torch.zeros((rows, at), dtype=dtype, device=device)
        for name, w in parts.items():
            self.weight[:, self.offsets[name]:self.offsets[name] + w.shape[1]].copy_(w)

    def operand(self, rows: int) -> torch.Tensor:
        return torch.empty((rows, self.columns), dtype=self.weight.dtype, device=self.weight.device)

    def __call__(self, y: torch.Tensor) -> torch.Tensor:
        return torch.mm(y, self.weight.t())

    def wide(self, y: torch.Tensor) -> torch.Tensor:
        """The product kept in fp32."""
        return _wide_mm(y, self.weight)

    def add_into(self, x: torch.Tensor, y: torch.Tensor) -> None:
        if y.dtype == torch.float32:
            torch.addmm(x, y, self.weight.t(), out=x)
        else:
            torch.addmm(x, y, self.weight.t(), out_dtype=torch.float32, out=x)


class DenseHead:
    """Logits in fp32."""

    def __init__(self, weight: torch.Tensor, dtype: torch.dtype, device) -> None:
        self.weight = weight.to(device=device, dtype=dtype).contiguous()

    def __call__(self, x: torch.Tensor) -> torch.Tensor:
        return _wide_mm(x, self.weight)
