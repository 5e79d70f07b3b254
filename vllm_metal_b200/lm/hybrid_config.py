"""Configuration of hybrid decoders: an ordered list of layers, each naming its mixer, the mixer's sizes and its
feed-forward.  Everything a ``config.json`` of such a model can vary is read here and validated once; the layer code
sees typed records only.  What a design fixes -- how a layer is arranged, its norm, its mixers -- is its ``Design``."""

from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Any

MAX_EXPERTS = 1024    # what the routing kernels take (B200_MAX_EXPERTS)
MAX_INPUT_TAPS = 16


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


@dataclass(frozen=True)
class SoftmaxAttentionArgs:
    """Softmax attention over every earlier token; query / key heads of ``dim``, value heads of ``vdim``."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float

    @classmethod
    def parse(cls, m: dict, where: str) -> SoftmaxAttentionArgs:
        a = cls(**{k: _take(m, k, where) for k in ("heads", "kv_heads", "dim", "vdim")}, scale=_take(m, "scale", where, float))
        _positive(a, where, "heads", "kv_heads", "dim", "vdim")
        if a.heads % a.kv_heads:
            raise ConfigError(f"{where}: {a.heads} query heads over {a.kv_heads} key/value heads")
        if not a.scale > 0:
            raise ConfigError(f"{where}: scale must be positive, got {a.scale}")
        return a


@dataclass(frozen=True)
class LightningArgs:
    """Linear attention whose state decays by a constant per head."""

    heads: int
    dim: int
    vdim: int
    decay: tuple[float, ...]

    kind = "lightning"

    @classmethod
    def parse(cls, m: dict, where: str) -> LightningArgs:
        a = cls(**{k: _take(m, k, where) for k in ("heads", "dim", "vdim")},
                decay=tuple(float(d) for d in _take(m, "decay", where, list)))
        _positive(a, where, "heads", "dim", "vdim")
        if len(a.decay) != a.heads or not all(0.0 <= d <= 1.0 for d in a.decay):
            raise ConfigError(f"{where}: decay must hold {a.heads} values from 0 to 1, got {list(a.decay)}")
        return a


@dataclass(frozen=True)
class SideBySideArgs:
    """Two mixers that read the same input; the result is the mean of their normed outputs."""

    left: SoftmaxAttentionArgs
    right: LightningArgs

    kind = "parallel"

    @classmethod
    def parse(cls, m: dict, where: str) -> SideBySideArgs:
        return cls(SoftmaxAttentionArgs.parse(_take(m, "left", where, dict), f"{where}.left"),
                   LightningArgs.parse(_take(m, "right", where, dict), f"{where}.right"))


@dataclass(frozen=True)
class RotaryArgs:
    """Rotation of the first ``dims`` dimensions of a head; with ``factor`` > 0 the frequencies are scaled (YaRN)."""

    dims: int
    base: float
    factor: float = 0.0
    original: float = 0.0
    fast: float = 0.0
    slow: float = 0.0

    @classmethod
    def parse(cls, rot: dict | None, where: str) -> RotaryArgs:
        if not rot:
            return cls(0, 1.0)
        where = f"{where}.rot"
        s = rot.get("scaling")
        a = cls(_take(rot, "dims", where), _take(rot, "base", where, float),
                **({} if not s else {k: _take(s, k, f"{where}.scaling", float) for k in ("factor", "original", "fast", "slow")}))
        if a.dims < 0 or a.dims % 2 or (a.dims and not a.base > 1):
            raise ConfigError(f"{where}: dims {a.dims} must be even, base {a.base} above 1")
        if s and not (a.factor > 0 and a.original > 0 and a.fast > 0 and a.slow > 0):
            raise ConfigError(f"{where}.scaling: factor, original, fast and slow must be positive")
        return a

    def frequencies(self) -> list[float]:
        """Angle per position of every pair."""
        plain = [self.base ** (-2.0 * i / self.dims) for i in range(self.dims // 2)]
        if not self.factor or not self.dims:
            return plain
        # the pair (a real number) that turns `t` times over the original length
        pair = lambda t: self.dims * math.log(self.original / (2 * math.pi * t)) / (2 * math.log(self.base))  # noqa: E731
        lo, hi = max(math.floor(pair(self.fast)), 0), min(math.ceil(pair(self.slow)), self.dims - 1)
        ramp = [min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0) for i in range(len(plain))]
        return [f / self.factor * r + f * (1.0 - r) for f, r in zip(plain, ramp)]

    @property
    def amplitude(self) -> float:
        """What cosine and sine are multiplied by."""
        return 0.1 * math.log(self.factor) + 1.0 if self.factor else 1.0


@dataclass(frozen=True)
class RotaryAttentionArgs:
    """Softmax attention with rotated, then normed heads; a window and the first tokens kept beside it."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: RotaryArgs
    window: int      # 0: every earlier token is visible
    keep_first: int  # of the first tokens, visible whatever the window

    kind = "attention"

    @classmethod
    def parse(cls, m: dict, where: str) -> RotaryAttentionArgs:
        a = SoftmaxAttentionArgs.parse(m, where)
        mask = m.get("mask") or {}
        b = cls(a.heads, a.kv_heads, a.dim, a.vdim, a.scale, RotaryArgs.parse(m.get("rot"), where),
                int(mask.get("size") or 0), int(mask.get("keep_first") or 0))
        if b.rot.dims > b.dim or b.window < 0 or b.keep_first < 0:
            raise ConfigError(f"{where}: rot.dims {b.rot.dims} of dim {b.dim}, mask.size {b.window}, mask.keep_first {b.keep_first}")
        return b


@dataclass(frozen=True)
class TimeMixArgs:
    """RWKV-style time mixing: a matrix state per head whose decay, per key channel, is a function of the input."""

    heads: int
    dim: int

    kind = "wkv"

    @property
    def inner(self) -> int:
        return self.heads * self.dim

    @classmethod
    def parse(cls, m: dict, where: str) -> TimeMixArgs:
        a = cls(heads=_take(m, "heads", where), dim=_take(m, "dim", where))
        _positive(a, where, "heads", "dim")
        return a


@dataclass(frozen=True)
class BiasedAttentionArgs:
    """Softmax attention whose scores fall with the distance; normed queries, keys and values, a factor on the queries that
    grows with the position, a window, and a sigmoid gate on the output."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int        # 0: every earlier token is visible
    temp_coef: float   # 0: no factor on the queries
    temp_every: float

    kind = "attention"

    @classmethod
    def parse(cls, m: dict, where: str) -> BiasedAttentionArgs:
        a, mask, temp = SoftmaxAttentionArgs.parse(m, where), m.get("mask") or {}, m.get("q_temp")
        coef, every = (_take(temp, k, f"{where}.q_temp", float) for k in ("coef", "every")) if temp else (0.0, 1.0)
        b = cls(a.heads, a.kv_heads, a.dim, a.vdim, a.scale, int(mask.get("size") or 0), coef, every)
        if b.window < 0 or not b.temp_every > 0:
            raise ConfigError(f"{where}: mask.size {b.window}, q_temp.every {b.temp_every}")
        return b

    def slopes(self) -> list[float]:
        """What every token of distance takes off a head's scores."""
        return [2.0 ** (-8.0 * (h + 1) / self.heads) for h in range(self.heads)]


MixerArgs = (LatentAttentionArgs | Mamba2Args | MLSTMArgs | LightningArgs | SideBySideArgs | RotaryAttentionArgs | TimeMixArgs |
             BiasedAttentionArgs)


@dataclass(frozen=True)
class RoutedArgs:
    """Feed-forward of routed experts, with a gated shared one beside them."""

    experts: int
    top: int
    ff: int
    scale: float
    shared_ff: int  # 0: none
    over_chosen: bool = False  # weights: softmax of the (biased) logits of the chosen alone; else of all, times scale

    @classmethod
    def parse(cls, mlp: dict, where: str, over_chosen: bool = False) -> RoutedArgs:
        where = f"{where}.mlp"
        router = _take(mlp, "router", where, dict)
        shared = None if over_chosen else mlp.get("shared")
        a = cls(_take(router, "experts", f"{where}.router"), _take(router, "top", f"{where}.router"),
                _take(_take(mlp, "expert", where, dict), "ff", f"{where}.expert"),
                1.0 if over_chosen else _take(router, "scale", f"{where}.router", float),
                _take(shared, "ff", f"{where}.shared") if shared else 0, over_chosen)
        _positive(a, where, "experts", "top", "ff")
        if a.top > a.experts or a.experts > MAX_EXPERTS:
            raise ConfigError(f"{where}: {a.top} of {a.experts} experts (at most {MAX_EXPERTS})")
        if shared and a.shared_ff < 1:
            raise ConfigError(f"{where}.shared: ff must be at least 1")
        return a


def paged_row(mixer: MixerArgs) -> int:
    """Elements a layer with this mixer caches per token."""
    if isinstance(mixer, LatentAttentionArgs):
        return mixer.kv_rank + mixer.rot_dim
    a = cached_heads(mixer)
    return a.kv_heads * (a.dim + a.vdim) if a is not None else 0


def cached_heads(mixer: MixerArgs) -> SoftmaxAttentionArgs | RotaryAttentionArgs | BiasedAttentionArgs | None:
    """The attention whose keys and values (of ``kv_heads``) a layer with this mixer caches, if any."""
    if isinstance(mixer, SideBySideArgs):
        return mixer.left
    return mixer if isinstance(mixer, (RotaryAttentionArgs, BiasedAttentionArgs)) else None


@dataclass(frozen=True)
class Design:
    """What the architecture fixes."""

    mixers: tuple[type, ...]
    # "parallel": mixer and feed-forward from one norm (lm/hybrid.py); "hyper": sublayers around several streams
    # (lm/streams.py); "sandwich": sublayers between two norms, a short convolution on the mixer's input (lm/sandwich.py);
    # "prenorm": a grouped norm ahead of every sublayer, looped layers take the embedding in again (lm/prenorm.py)
    layout: str = "parallel"
    feed_forward: tuple[str, ...] = ("dense",)
    route_over_chosen: bool = False

    @property
    def hyper_connected(self) -> bool:
        return self.layout == "hyper"


DESIGNS = {
    "Mapuvik": Design((LatentAttentionArgs, Mamba2Args, MLSTMArgs)),
    "Tatazen": Design((LightningArgs, SideBySideArgs), "hyper"),
    "Kerolorn": Design((RotaryAttentionArgs,), "sandwich", ("moe",)),
    "Retuvik": Design((TimeMixArgs, BiasedAttentionArgs), "prenorm", ("dense", "moe"), route_over_chosen=True),
}


@dataclass(frozen=True)
class LayerArgs:
    mixer: MixerArgs
    ff: int       # dense feed-forward; 0: none
    weights: int  # the layer whose tensors this one uses (itself unless shared)
    routed: RoutedArgs | None = None


@dataclass(frozen=True)
class HybridArgs:
    name: str
    vocab: int
    width: int
    eps: float
    layers: tuple[LayerArgs, ...]  # in the order they run: a looped layer is there once a pass
    streams: int = 1               # copies of the residual stream (hyper-connected designs)
    input_taps: int = 0            # of the convolution on a mixer's input (2: token shift); 0: none
    logit_scale: float = 1.0
    norm_groups: int = 1           # parts of a row that are normed on their own
    embedding_scale: float = 1.0
    passes: tuple[tuple[int, int], ...] = ()  # (layer run, number of the pass) where a pass of the loop begins
    loop_times: int = 0

    @property
    def design(self) -> Design:
        return DESIGNS.get(self.name, DESIGNS["Mapuvik"])

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    def layers_of(self, kind: str) -> list[int]:
        return [i for i, layer in enumerate(self.layers) if layer.mixer.kind == kind]

    def paged_layers(self) -> dict[int, int]:
        """Layers with a paged cache and the elements each keeps per token."""
        rows = {i: paged_row(layer.mixer) for i, layer in enumerate(self.layers)}
        return {i: n for i, n in rows.items() if n}

    def owners(self) -> dict[int, LayerArgs]:
        """The layers that have tensors, by the number in the tensors' names."""
        found: dict[int, LayerArgs] = {}
        for layer in self.layers:
            found.setdefault(layer.weights, layer)
        return dict(sorted(found.items()))

    @classmethod
    def parse(cls, config: dict) -> HybridArgs:
        name = str(config.get("architecture", "hybrid"))
        design = DESIGNS.get(name, DESIGNS["Mapuvik"])
        layers: list[LayerArgs] = []
        for i, entry in enumerate(_take(config, "layers", name, list)):
            where = f"layers[{i}]"
            kind = _take(entry, "type", where, str)
            known = {c.kind: c for c in design.mixers}
            if kind not in known:
                raise ConfigError(f"{where}: unknown mixer '{kind}' (known: {', '.join(sorted(known))})")
            mixer = known[kind].parse(_take(entry, "mixer", where, dict), where)
            ff, routed = 0, None
            if entry.get("mlp") is not None:
                mlp = entry["mlp"]
                if mlp.get("kind", "dense") not in design.feed_forward:
                    raise ConfigError(f"{where}: feed-forward kind '{mlp.get('kind')}' is not supported "
                                      f"({', '.join(design.feed_forward)} only)")
                if mlp.get("kind") == "moe":
                    routed = RoutedArgs.parse(mlp, where, design.route_over_chosen)
                else:
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
            layers.append(LayerArgs(mixer, ff, src, routed))
        if not layers:
            raise ConfigError(f"{name}: no layers")
        if config.get("loop") is not None:
            layers = cls._unroll(layers, config["loop"], name)
        extra: dict[str, Any] = {}
        if design.layout == "hyper":
            extra = dict(streams=_take(config, "streams", name), input_taps=2)
        elif design.layout == "sandwich":
            extra = dict(input_taps=_take(_take(config, "canon", name, dict), "taps", f"{name}: canon"),
                         logit_scale=_take(config, "logit_scale", name, float))
            if not 1 <= extra["input_taps"] <= MAX_INPUT_TAPS:
                raise ConfigError(f"{name}: canon.taps {extra['input_taps']} outside 1..{MAX_INPUT_TAPS}")
        elif design.layout == "prenorm":
            extra = dict(norm_groups=_take(_take(config, "norm", name, dict), "groups", f"{name}: norm"),
                         embedding_scale=_take(_take(config, "embedding", name, dict), "scale", f"{name}: embedding", float))
            if extra["norm_groups"] < 1 or _take(config, "width", name) % extra["norm_groups"]:
                raise ConfigError(f"{name}: width {config['width']} in {extra['norm_groups']} norm groups")
            if config.get("loop") is not None:
                start, stop, times = (config["loop"][k] for k in ("start", "stop", "times"))
                extra |= dict(loop_times=times,
                              passes=tuple((start + t * (stop - start), t) for t in range(times)) if stop > start else ())
        a = cls(name=name, vocab=_take(config, "vocab", name), width=_take(config, "width", name),
                eps=_take(_take(config, "norm", name, dict), "eps", name, float), layers=tuple(layers), **extra)
        _positive(a, name, "vocab", "width", "streams")
        return a

    @staticmethod
    def _unroll(layers: list[LayerArgs], loop: dict, name: str) -> list[LayerArgs]:
        """``start .. stop - 1`` several times in a row; each pass is a layer of its own with the same weights."""
        start, stop, times = (_take(loop, k, f"{name}: loop") for k in ("start", "stop", "times"))
        if not 0 <= start <= stop <= len(layers) or times < 1:
            raise ConfigError(f"{name}: loop over layers {start}..{stop} of {len(layers)}, {times} times")
        return layers[:start] + layers[start:stop] * times + layers[stop:]
