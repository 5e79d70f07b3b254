"""Configuration of hybrid decoders: an ordered list of layers, each naming its mixer, the mixer's sizes and its
feed-forward.  Everything a ``config.json`` of such a model can vary is read here and validated once; the layer code
sees typed records only."""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any


class ConfigError(ValueError):
    """A config.json this build cannot run; the message names the entry."""


def _take(d: dict, key: str, where: str, kind=int):
    if key not in d:
        raise ConfigError(f"{where}: '{key}' is missing")
    v = d[key]
    if kind is int and (isinstance(v, bool) or int(v) != v):
        raise ConfigError(f"{where}: '{key}' must be an integer, got {v!r}")
    return kind(v)


def _positive(obj: Any, where: str, *names: str) -> None:
    for n in names:
        if getattr(obj, n) < 1:
            raise ConfigError(f"{where}: {n} must be at least 1, got {getattr(obj, n)}")


@dataclass(frozen=True)
class LatentAttentionArgs:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot_base: float
    rot_dims: int
    window: int  # 0: every earlier token is visible

    kind = "latent_attention"

    @classmethod
    def parse(cls, m: dict, where: str) -> LatentAttentionArgs:
        rot_dim = _take(m, "rot_dim", where)
        rot = m.get("rot") or {}
        mask = m.get("mask") or {}
        a = cls(heads=_take(m, "heads", where), dim=_take(m, "dim", where), rot_dim=rot_dim,
                vdim=_take(m, "vdim", where), kv_rank=_take(m, "kv_rank", where), scale=_take(m, "scale", where, float),
                rot_base=float(rot.get("base", 10000.0)), rot_dims=int(rot.get("dims", rot_dim)),
                window=int(mask.get("size") or 0))
        _positive(a, where, "heads", "dim", "vdim", "kv_rank")
        if a.rot_dims % 2 or not 0 <= a.rot_dims <= a.rot_dim or a.window < 0:
            raise ConfigError(f"{where}: rot.dims {a.rot_dims} of rot_dim {a.rot_dim}, mask.size {a.window}")
        return a


@dataclass(frozen=True)
class Mamba2Args:
    heads: int
    groups: int
    state: int
    vdim: int
    conv: int
    norm_groups: int

    kind = "mamba2"

    @property
    def inner(self) -> int:
        return self.heads * self.vdim

    @property
    def conv_channels(self) -> int:
        return self.inner + 2 * self.groups * self.state

    @classmethod
    def parse(cls, m: dict, where: str) -> Mamba2Args:
        a = cls(**{k: _take(m, k, where) for k in ("heads", "groups", "state", "vdim", "conv", "norm_groups")})
        _positive(a, where, "heads", "groups", "state", "vdim", "conv", "norm_groups")
        if a.heads % a.groups or a.inner % a.norm_groups:
            raise ConfigError(f"{where}: {a.heads} heads in {a.groups} groups, inner {a.inner} in {a.norm_groups} parts")
        return a


@dataclass(frozen=True)
class MLSTMArgs:
    heads: int
    dim: int
    vdim: int
    gate_cap: float

    kind = "mlstm"

    @classmethod
    def parse(cls, m: dict, where: str) -> MLSTMArgs:
        a = cls(heads=_take(m, "heads", where), dim=_take(m, "dim", where), vdim=_take(m, "vdim", where),
                gate_cap=_take(m, "gate_cap", where, float))
        _positive(a, where, "heads", "dim", "vdim")
        if a.gate_cap <= 0:
            raise ConfigError(f"{where}: gate_cap must be positive")
        return a


MIXER_ARGS = {c.kind: c for c in (LatentAttentionArgs, Mamba2Args, MLSTMArgs)}


@dataclass(frozen=True)
class LayerArgs:
    mixer: LatentAttentionArgs | Mamba2Args | MLSTMArgs
    ff: int       # 0: no feed-forward
    weights: int  # the layer whose tensors this one uses (itself unless shared)


@dataclass(frozen=True)
class HybridArgs:
    name: str
    vocab: int
    width: int
    eps: float
    layers: tuple[LayerArgs, ...]

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    def layers_of(self, kind: str) -> list[int]:
        return [i for i, layer in enumerate(self.layers) if layer.mixer.kind == kind]

    @classmethod
    def parse(cls, config: dict) -> HybridArgs:
        name = str(config.get("architecture", "hybrid"))
        layers: list[LayerArgs] = []
        for i, entry in enumerate(_take(config, "layers", name, list)):
            where = f"layers[{i}]"
            kind = _take(entry, "type", where, str)
            if kind not in MIXER_ARGS:
                raise ConfigError(f"{where}: unknown mixer '{kind}' (known: {', '.join(sorted(MIXER_ARGS))})")
            mixer = MIXER_ARGS[kind].parse(_take(entry, "mixer", where, dict), where)
            ff = 0
            if entry.get("mlp") is not None:
                mlp = entry["mlp"]
                if mlp.get("kind", "dense") != "dense":
                    raise ConfigError(f"{where}: feed-forward kind '{mlp.get('kind')}' is not supported (dense only)")
                ff = _take(mlp, "ff", where)
                if ff < 1:
                    raise ConfigError(f"{where}: ff must be at least 1")
            src = entry.get("weights_of")
            src = i if src is None else int(src)
            if src != i:
                # a shared layer may name another shared one: follow it to the owner
                if not 0 <= src < len(entry_list := config["layers"]):
                    raise ConfigError(f"{where}: weights_of {src} is not a layer")
                seen = {i}
                while entry_list[src].get("weights_of") is not None:
                    if src in seen:
                        raise ConfigError(f"{where}: weights_of runs in a circle")
                    seen.add(src)
                    src = int(entry_list[src]["weights_of"])
                if entry_list[src]["type"] != kind:
                    raise ConfigError(f"{where}: weights_of {src} names a layer of type {entry_list[src]['type']}")
            layers.append(LayerArgs(mixer, ff, src))
        if not layers:
            raise ConfigError(f"{name}: no layers")
        a = cls(name=name, vocab=_take(config, "vocab", name), width=_take(config, "width", name),
                eps=_take(_take(config, "norm", name, dict), "eps", name, float), layers=tuple(layers))
        _positive(a, name, "vocab", "width")
        return a
