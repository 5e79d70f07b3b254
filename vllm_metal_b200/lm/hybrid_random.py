"""Random weights for a hybrid configuration (benchmarks, tests, dummy loading): variances that keep the residual
stream, the gates and the decays in a range where every mechanism matters."""

from __future__ import annotations

import torch

from .hybrid_config import (BiasedAttentionArgs, HybridArgs, LatentAttentionArgs, LightningArgs, Mamba2Args, MLSTMArgs,
                            RotaryAttentionArgs, SideBySideArgs, TimeMixArgs)

DECAY_RANK = 64  # bottleneck of the decays where nothing says otherwise (a checkpoint has its own)


def tensor_shapes(args: HybridArgs) -> dict[str, tuple[int, ...]]:
    """Checkpoint tensor names and shapes of a configuration."""
    w = args.width
    shapes: dict[str, tuple[int, ...]] = {"embed": (args.vocab, w)}
    for i, layer in args.owners().items():
        m, p = layer.mixer, f"l{i}.mix."
        shapes[f"l{i}.norm1"] = (w,)
        if isinstance(m, Mamba2Args):
            shapes |= {p + "in": (2 * m.inner + 2 * m.groups * m.state + m.heads, w), p + "conv": (m.conv_channels, m.conv),
                       p + "conv.b": (m.conv_channels,), p + "dt_bias": (m.heads,), p + "A_log": (m.heads,),
                       p + "D": (m.heads,), p + "norm": (m.inner,), p + "o": (w, m.inner)}
        elif isinstance(m, MLSTMArgs):
            qk, v = m.heads * m.dim, m.heads * m.vdim
            shapes |= {p + "q": (qk, w), p + "k": (qk, w), p + "v": (v, w), p + "g": (v, w), p + "o": (w, v),
                       p + "norm": (v,), p + "i": (m.heads, w), p + "i.b": (m.heads,), p + "f": (m.heads, w),
                       p + "f.b": (m.heads,)}
        elif isinstance(m, LatentAttentionArgs):
            shapes |= {p + "q": (m.heads * (m.dim + m.rot_dim), w), p + "dkv": (m.kv_rank + m.rot_dim, w),
                       p + "dkv.norm": (m.kv_rank,), p + "uk": (m.heads * m.dim, m.kv_rank),
                       p + "uv": (m.heads * m.vdim, m.kv_rank), p + "g": (m.heads * m.vdim, w),
                       p + "o": (w, m.heads * m.vdim)}
        elif isinstance(m, LightningArgs):
            shapes |= _lightning_shapes(m, p, w)
        elif isinstance(m, SideBySideArgs):
            a = m.left
            shapes |= {p + "left.q": (a.heads * a.dim, w), p + "left.k": (a.kv_heads * a.dim, w),
                       p + "left.v": (a.kv_heads * a.vdim, w), p + "left.q.norm": (a.dim,), p + "left.k.norm": (a.dim,),
                       p + "left.o": (w, a.heads * a.vdim), **_lightning_shapes(m.right, p + "right.", w),
                       p + "left.out": (w,), p + "right.out": (w,)}
        elif isinstance(m, RotaryAttentionArgs):
            shapes |= {p + "q": (m.heads * m.dim, w), p + "k": (m.kv_heads * m.dim, w), p + "v": (m.kv_heads * m.vdim, w),
                       p + "temp": (m.heads,), p + "o": (w, m.heads * m.vdim)}
        elif isinstance(m, TimeMixArgs):
            rank = min(DECAY_RANK, w)
            shapes |= {p + "mu." + s: (w,) for s in "rkvgw"} | {p + s: (m.inner, w) for s in "rkvg"}
            shapes |= {p + "w1": (rank, w), p + "w2": (m.inner, rank), p + "w0": (m.inner,), p + "u": (m.heads, m.dim),
                       p + "norm": (m.inner,), p + "o": (w, m.inner)}
        elif isinstance(m, BiasedAttentionArgs):
            shapes |= {p + "q": (m.heads * m.dim, w), p + "k": (m.kv_heads * m.dim, w), p + "v": (m.kv_heads * m.vdim, w),
                       p + "q.norm": (m.dim,), p + "k.norm": (m.dim,), p + "g": (m.heads * m.vdim, w),
                       p + "o": (w, m.heads * m.vdim)}
        if layer.ff:
            shapes |= {f"l{i}.mlp.up": (layer.ff, w), f"l{i}.mlp.down": (w, layer.ff)}
        if layer.routed is not None:
            r, p = layer.routed, f"l{i}.mlp."
            units = [(f"e{e}.", r.ff) for e in range(r.experts)] + ([("shared.", r.shared_ff)] if r.shared_ff else [])
            for name, ff in units:
                shapes |= {p + name + "gate": (ff, w), p + name + "up": (ff, w), p + name + "down": (w, ff)}
            shapes |= {p + "router": (r.experts, w), p + ("router.b" if r.over_chosen else "correction"): (r.experts,)}
            if r.shared_ff:
                shapes |= {p + "shared.sg": (1, w)}
        if args.design.layout == "sandwich":
            shapes |= {f"l{i}.norm1b": (w,), f"l{i}.canon1": (w, args.input_taps)}
            if layer.routed is not None:
                shapes |= {f"l{i}.norm2": (w,), f"l{i}.norm2b": (w,)}
        if args.design.layout == "prenorm" and (layer.ff or layer.routed is not None):
            shapes |= {f"l{i}.norm2": (w,)}
            if layer.ff:
                shapes |= {f"l{i}.mlp.up.b": (layer.ff,), f"l{i}.mlp.down.b": (w,), f"l{i}.mlp.act": (2,)}
        if args.design.hyper_connected:
            s = args.streams
            shapes |= {f"l{i}.shift": (w,)}
            if layer.ff:
                shapes |= {f"l{i}.mlp.gate": (layer.ff, w), f"l{i}.norm2": (w,)}
            for q in (1, 2) if layer.ff else (1,):
                shapes |= {f"l{i}.hc{q}.in": (s,), f"l{i}.hc{q}.out": (s,), f"l{i}.hc{q}.mix": (s, s),
                           f"l{i}.rg{q}": (w, w), f"l{i}.rg{q}.b": (w,)}
    if args.passes:
        shapes |= {"loop.step": (args.loop_times, w)}
    return shapes | {"final.norm": (w,), "head": (args.vocab, w)}


def _lightning_shapes(m: LightningArgs, p: str, w: int) -> dict[str, tuple[int, ...]]:
    qk, v = m.heads * m.dim, m.heads * m.vdim
    return {p + "q": (qk, w), p + "k": (qk, w), p + "v": (v, w), p + "g": (v, w), p + "o": (w, v), p + "norm": (v,)}


def random_tensors(args: HybridArgs, device="cpu", seed: int = 0):
    """A ``get(name, shape)`` for ``HybridModel`` whose tensors are drawn when asked for."""
    shapes = tensor_shapes(args)
    number = {name: i for i, name in enumerate(shapes)}

    def get(name: str, shape: tuple[int, ...]) -> torch.Tensor:
        if len(shape) != len(shapes[name]) or any(n is not None and n != m for n, m in zip(shape, shapes[name])):
            raise ValueError(f"tensor '{name}': asked for {shape}, the configuration says {shapes[name]}")
        shape = shapes[name]
        gen = torch.Generator(device=device).manual_seed(seed * 1000003 + number[name])
        t = torch.empty(shape, dtype=torch.float32, device=device).normal_(0.0, 1.0, generator=gen)
        leaf = name.split(".", 1)[-1]
        plain_norm = args.design.layout != "parallel" and len(shape) == 1 and leaf.rsplit(".", 1)[-1] in (
            "norm", "norm1", "norm2", "norm1b", "norm2b", "temp")
        if leaf == "mlp.correction":          # of the size of the scores it is added to
            t = 0.5 * t / shape[0]
        elif leaf in ("mix.dkv.norm", "mix.norm", "mix.left.out", "mix.right.out") or plain_norm:
            t = 1.0 + 0.1 * t
        elif leaf in ("hc1.in", "hc2.in"):     # about the mean of the streams
            t = (1.0 + 0.3 * t) / shape[0]
        elif leaf in ("hc1.out", "hc2.out"):
            t = 1.0 + 0.3 * t
        elif leaf in ("hc1.mix", "hc2.mix"):   # near the identity: the stream neither dies nor grows
            t = torch.eye(shape[0], device=device) + 0.1 * t
        elif leaf == "shift":
            t = torch.sigmoid(t)
        elif leaf.startswith("mix.mu."):       # between the row and the one before it
            t = torch.sigmoid(t)
        elif leaf == "mix.w0":                 # decays from a few rows to some hundred
            t = 1.5 * t - 3.0
        elif leaf in ("norm1", "norm"):        # stored around zero
            t = 0.1 * t
        elif leaf == "mix.A_log":
            t = t.abs() * 0.7
        elif leaf == "mix.dt_bias":
            t = t - 2.0
        elif leaf == "mix.f.b":
            t = t + 2.0
        elif leaf == "mix.conv":
            t = t * shape[1] ** -0.5
        elif leaf in ("mix.D", "mix.i.b", "mix.conv.b", "mix.u", "embed", "step", "mlp.router.b", "mlp.up.b", "mlp.down.b"):
            t = 0.5 * t
        elif len(shape) == 2:
            t = t * shape[1] ** -0.5
        return t.to(torch.bfloat16)

    return get
