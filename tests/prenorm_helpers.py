"""Small configurations of pre-norm decoders with time mixing, and checkpoints whose routing leaves no close calls."""

from __future__ import annotations

import copy

import numpy as np
import torch

from .hybrid_helpers import make_config

ATTENTION = {"heads": 6, "kv_heads": 2, "dim": 24, "vdim": 40, "scale": 0.31, "mask": {"size": 29},
             "q_temp": {"coef": 0.7, "every": 19}}
DENSE = {"kind": "dense", "ff": 56}


def experts(ff: int = 40, n: int = 7, top: int = 3) -> dict:
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": n, "top": top}}


def wkv_layer(mlp: dict | None = DENSE, heads: int = 5, dim: int = 24) -> dict:
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim}, "mlp": copy.deepcopy(mlp)}


def attention_layer(mlp: dict | None = DENSE, **over) -> dict:
    return {"type": "attention", "mixer": {**copy.deepcopy(ATTENTION), **over}, "mlp": copy.deepcopy(mlp)}


def prenorm_config(layers: list[dict], loop: tuple[int, int, int] | None = None, groups: int = 4, scale: float = 3.0,
                   vocab: int = 203, width: int = 88, eps: float = 1e-6) -> dict:
    c = {**make_config(layers, vocab, width, eps), "architecture": "Retuvik", "embedding": {"scale": scale}}
    c["norm"]["groups"] = groups
    if loop is not None:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


def default_prenorm_config() -> dict:
    return prenorm_config([wkv_layer(), wkv_layer(experts(), heads=3, dim=40), attention_layer(),
                           attention_layer(None, mask=None, q_temp=None, heads=4, kv_heads=4, dim=16, vdim=8),
                           wkv_layer(experts(ff=24, n=12, top=5), heads=2, dim=32),
                           attention_layer(experts(ff=16, n=4, top=1), mask={"size": 16}, heads=3, kv_heads=1), wkv_layer(None, 1, 64)],
                          loop=(1, 3, 3))


def clear_routing(config: dict):
    """Edits a checkpoint so that no choice of experts is close: the router of a block of E experts reads the stream's first E
    columns, which only the embedding fills (evenly spaced levels in an order of the token's own), and the router's biases are
    well below the distance of two levels."""
    wide = max((layer["mlp"]["router"]["experts"] for layer in config["layers"] if (layer["mlp"] or {}).get("kind") == "moe"),
               default=0)

    def edit(t: dict[str, torch.Tensor]) -> None:
        rng = np.random.default_rng(11)
        levels = np.linspace(-1.5, 1.5, wide)
        t["embed"][:, :wide] = torch.tensor(np.stack([rng.permutation(levels) for _ in range(config["vocab"])])).bfloat16()
        for name, x in t.items():
            if name.endswith(("mix.o", ".down", "down.b")):
                x[:wide] = 0.0
        if "loop.step" in t:
            t["loop.step"][:, :wide] = 0.0
        for i, layer in enumerate(config["layers"]):
            if (layer["mlp"] or {}).get("kind") != "moe":
                continue
            n = layer["mlp"]["router"]["experts"]
            t[f"l{i}.norm2"][:wide] = 1.0
            t[f"l{i}.mlp.router"].zero_()
            t[f"l{i}.mlp.router"][range(n), range(n)] = 3.0
            t[f"l{i}.mlp.router.b"][:] = torch.tensor(np.where(rng.random(n) < 0.5, -0.08, 0.08)).bfloat16()

    return edit
