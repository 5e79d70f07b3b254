"""Small configurations of sandwich-norm decoders with routed experts, and checkpoints whose routing leaves no close calls."""

from __future__ import annotations

import copy

import numpy as np
import torch

from .hybrid_helpers import make_config

ATTENTION = {"heads": 6, "kv_heads": 2, "dim": 24, "vdim": 40, "scale": 0.31,
             "rot": {"base": 5000.0, "dims": 16, "scaling": {"factor": 4.0, "original": 96, "fast": 8.0, "slow": 0.5}},
             "mask": {"size": 29, "keep_first": 5}}
EXPERTS = {"kind": "moe", "expert": {"ff": 40}, "router": {"experts": 7, "scale": 1.7, "top": 3}, "shared": {"ff": 56}}


def experts(ff: int = 40, n: int = 7, top: int = 3, scale: float = 1.7, shared: int | None = 56) -> dict:
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": n, "scale": scale, "top": top}}
    return m if shared is None else {**m, "shared": {"ff": shared}}


def sandwich_layer(mlp: dict | None = EXPERTS, **over) -> dict:
    return {"type": "attention", "mixer": {**copy.deepcopy(ATTENTION), **over}, "mlp": copy.deepcopy(mlp)}


def sandwich_config(layers: list[dict], taps: int = 3, logit_scale: float = 0.7, vocab: int = 203, width: int = 88,
                    eps: float = 1e-6) -> dict:
    return {**make_config(layers, vocab, width, eps), "architecture": "Kerolorn", "canon": {"taps": taps},
            "logit_scale": logit_scale}


def default_sandwich_config() -> dict:
    plain = {"base": 300.0, "dims": 24}
    return sandwich_config([sandwich_layer(), sandwich_layer(experts(ff=72, n=4, top=1, scale=0.8, shared=None)),
                            sandwich_layer(None, mask={"size": 16, "keep_first": 0}, rot=plain),
                            sandwich_layer(experts(ff=24, n=12, top=5, shared=16), mask=None, heads=4, kv_heads=4, dim=16, vdim=8,
                                           rot={"base": 1e4, "dims": 4})], taps=4)


def clear_routing(config: dict):
    """Edits a checkpoint so that no choice of experts is close: the router of a block of E experts reads the stream's first E
    columns, which only the embedding fills (evenly spaced levels in an order of the token's own); expert 0 is always chosen
    and expert 1 never, by their corrections, where that leaves a choice."""
    wide = max((layer["mlp"]["router"]["experts"] for layer in config["layers"] if layer["mlp"]), default=0)

    def edit(t: dict[str, torch.Tensor]) -> None:
        rng = np.random.default_rng(11)
        levels = np.linspace(-1.5, 1.5, wide)
        t["embed"][:, :wide] = torch.tensor(np.stack([rng.permutation(levels) for _ in range(config["vocab"])])).bfloat16()
        for i, layer in enumerate(config["layers"]):
            t[f"l{i}.norm1b"][:wide] = 0.0
            if not layer["mlp"]:
                continue
            t[f"l{i}.norm2"][:wide] = 1.0
            t[f"l{i}.norm2b"][:wide] = 0.0
            n, top = (layer["mlp"]["router"][k] for k in ("experts", "top"))
            t[f"l{i}.mlp.router"].zero_()
            t[f"l{i}.mlp.router"][range(n), range(n)] = 2.0
            t[f"l{i}.mlp.correction"].zero_()
            if 1 < top < n:
                t[f"l{i}.mlp.correction"][0], t[f"l{i}.mlp.correction"][1] = 1.0, -1.0

    return edit
