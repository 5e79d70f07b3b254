"""Sequence mixers of hybrid decoders over the C-ABI kernels.  A mixer owns its weights (which layers may share) and is
handed, per call, the stacked projections of its input and what its LAYER keeps between steps (a latent pool or state
slots); it leaves its heads' outputs, gated and normed, in the left columns of the layer's output operand.

Interface: ``spans`` names runs of parts the mixer also wants as one view, ``weights`` are to be stacked into the layer's input product, ``out_weight`` belongs to its output product
(the layer takes both away with ``take_weights``); ``run(parts, up, meta, cache, layer, y, act_offset)``.  A mixer with
``mix_weight [mixes, width]`` reads several mixes of a row with the row before, ``project(mixes [mixes, T, width])`` makes its
parts of them."""

from __future__ import annotations

from collections.abc import Callable

import torch

from ..attention.impls.segments import EXPAND_PAGE
from ..metal import get_ops
from .dense import BatchedLinear, SideBySideLinear, StackedLinear
from .hybrid_config import (BiasedAttentionArgs, LatentAttentionArgs, LightningArgs, Mamba2Args, MLSTMArgs, RotaryAttentionArgs,
                            SoftmaxAttentionArgs, TimeMixArgs)

Get = Callable[[str, tuple[int, ...]], torch.Tensor]


class Mixer:
    mix_weight: torch.Tensor | None = None
    spans: dict[str, tuple[str, str]] = {}
    weights: dict[str, torch.Tensor]
    out_weight: torch.Tensor

    def take_weights(self) -> tuple[dict[str, torch.Tensor], torch.Tensor]:
        w, o = self.weights, self.out_weight
        self.weights, self.out_weight = {}, None
        return w, o


class Mamba2Mixer(Mixer):
    """Selective state space with a scalar decay per head (Mamba-2): short convolution -> recurrence -> gated norm."""

    def __init__(self, m: Mamba2Args, width: int, eps: float, get: Get, dtype, device) -> None:
        self.m, self.eps = m, eps
        f32 = lambda name, *shape: get(name, shape).to(device=device, dtype=torch.float32)  # noqa: E731
        self.weights = {"in": get("in", (2 * m.inner + 2 * m.groups * m.state + m.heads, width))}
        self.out_weight = get("o", (width, m.inner))
        self.conv_w = f32("conv", m.conv_channels, m.conv).t().contiguous()
        self.conv_b = f32("conv.b", m.conv_channels)
        self.dt_bias = f32("dt_bias", m.heads)
        self.rate = torch.exp(f32("A_log", m.heads))
        self.skip = f32("D", m.heads)
        self.norm = f32("norm", m.inner)

    def run(self, parts, up, meta, cache, layer: int, y: torch.Tensor, act_offset: int) -> None:
        m, ops, st = self.m, get_ops(), cache.states[layer]
        z, xbc, dt = parts["in"].split([m.inner, m.conv_channels, m.heads], dim=1)
        xbc = ops.causal_conv(xbc, self.conv_w, self.conv_b, st.conv, meta)
        x, b, c = xbc.split([m.inner, m.groups * m.state, m.groups * m.state], dim=1)
        o = ops.recurrence("ssd", c, b, x, dt, None, meta, st.matrix, heads=m.heads, groups=m.groups, key_dim=m.state,
                           value_dim=m.vdim, bias_a=self.dt_bias, rate=self.rate, skip=self.skip)
        ops.mixer_finish(y, m.inner, up, act_offset, y=o, pre_gate=z, weight=self.norm,
                         group_size=m.inner // m.norm_groups, eps=self.eps)


class MLSTMMixer(Mixer):
    """Matrix memory with exponential gates (mLSTM): recurrence -> per-head norm -> output gate."""

    def __init__(self, m: MLSTMArgs, width: int, eps: float, get: Get, dtype, device) -> None:
        self.m, self.eps = m, eps
        f32 = lambda name, *shape: get(name, shape).to(device=device, dtype=torch.float32)  # noqa: E731
        qk, v = m.heads * m.dim, m.heads * m.vdim
        self.weights = {"q": get("q", (qk, width)), "k": get("k", (qk, width)), "v": get("v", (v, width)),
                        "g": get("g", (v, width)), "i": get("i", (m.heads, width)), "f": get("f", (m.heads, width))}
        self.out_weight = get("o", (width, v))
        self.i_bias, self.f_bias = f32("i.b", m.heads), f32("f.b", m.heads)
        self.norm = f32("norm", v)

    def run(self, parts, up, meta, cache, layer: int, y: torch.Tensor, act_offset: int) -> None:
        m, ops, st = self.m, get_ops(), cache.states[layer]
        o = ops.recurrence("mlstm", parts["q"], parts["k"], parts["v"], parts["i"], parts["f"], meta, st.matrix,
                           heads=m.heads, groups=m.heads, key_dim=m.dim, value_dim=m.vdim, bias_a=self.i_bias,
                           bias_b=self.f_bias, norm_state=st.normaliser, max_state=st.maximum,
                           q_scale=m.dim ** -0.5, gate_cap=m.gate_cap)
        ops.mixer_finish(y, m.heads * m.vdim, up, act_offset, y=o, post_gate=parts["g"], weight=self.norm,
                         group_size=m.vdim, eps=self.eps)


class LightningMixer(Mixer):
    """Linear attention with a constant decay per head: silu -> recurrence -> one norm over all heads -> output gate."""

    spans = {"qkv": ("q", "v")}

    def __init__(self, m: LightningArgs, width: int, eps: float, get: Get, dtype, device) -> None:
        self.m, self.eps = m, eps
        qk, v = m.heads * m.dim, m.heads * m.vdim
        self.weights = {"q": get("q", (qk, width)), "k": get("k", (qk, width)), "v": get("v", (v, width)),
                        "g": get("g", (v, width))}
        self.out_weight = get("o", (width, v))
        self.norm = get("norm", (v,)).to(device=device, dtype=torch.float32)
        decay = torch.tensor(m.decay, dtype=torch.float64)
        self.decay = decay.to(device=device, dtype=torch.float32)
        # a head that forgets at once still needs a finite logarithm: exp(-1e4) is zero in 32 bits
        self.rate = (-decay.log()).clamp(max=1e4).to(device=device, dtype=torch.float32)

    def run(self, parts, up, meta, cache, layer: int, y: torch.Tensor, act_offset: int) -> None:
        m, ops = self.m, get_ops()
        o = ops.recurrence("lightning", parts["q"], parts["k"], parts["v"], None, None, meta, cache.states[layer].matrix,
                           heads=m.heads, groups=m.heads, key_dim=m.dim, value_dim=m.vdim, rate=self.rate,
                           decay=self.decay, silu=parts["qkv"])
        inner = m.heads * m.vdim
        ops.mixer_finish(y, inner, up, act_offset, y=o, post_gate=parts["g"], weight=self.norm, group_size=inner,
                         eps=self.eps)


class SoftmaxAttentionMixer(Mixer):
    """Causal attention over paged keys and values, per-head norms of queries and keys, no rotation."""

    def __init__(self, m: SoftmaxAttentionArgs, width: int, eps: float, get: Get, dtype, device) -> None:
        self.m, self.eps = m, eps
        self.weights = {"q": get("q", (m.heads * m.dim, width)), "k": get("k", (m.kv_heads * m.dim, width)),
                        "v": get("v", (m.kv_heads * m.vdim, width))}
        self.out_weight = get("o", (width, m.heads * m.vdim))
        self.q_norm, self.k_norm = (get(n, (m.dim,)).to(device=device, dtype=dtype) for n in ("q.norm", "k.norm"))

    def run(self, parts, up, meta, cache, layer: int, y: torch.Tensor, act_offset: int) -> None:
        m, ops = self.m, get_ops()
        keys, values = cache.kv[layer]
        q, k, v = (parts[n].unflatten(1, (h, d)) for n, h, d in (("q", m.heads, m.dim), ("k", m.kv_heads, m.dim),
                                                                  ("v", m.kv_heads, m.vdim)))
        ops.norm_rope_cache(q, k, v, keys, values, meta.slot_mapping, q_norm_weight=self.q_norm,
                            k_norm_weight=self.k_norm, eps=self.eps)
        inner = m.heads * m.vdim
        ops.paged_attention_primitive(q, keys, values, m.kv_heads, m.scale, 0.0, meta.block_tables, meta.seq_lens,
                                      meta.cu_seqlens_q, meta.block_size, meta.max_seq_len, -1,
                                      y[:, :inner].unflatten(1, (m.heads, m.vdim)), wide_weights=True, plain_softmax=True,
                                      min_q_len=meta.min_q_len)
        if up is not None or y.shape[1] > inner:
            ops.mixer_finish(y, inner, up, act_offset)


class RotaryAttentionMixer(Mixer):
    """Causal attention over paged keys and values: heads rotated, then normed, scores scaled per head; a sliding window
    and the first tokens kept beside it."""

    def __init__(self, m: RotaryAttentionArgs, width: int, eps: float, get: Get, dtype, device) -> None:
        self.m, self.eps = m, eps
        self.weights = {"q": get("q", (m.heads * m.dim, width)), "k": get("k", (m.kv_heads * m.dim, width)),
                        "v": get("v", (m.kv_heads * m.vdim, width))}
        self.out_weight = get("o", (width, m.heads * m.vdim))
        self.temperature = get("temp", (m.heads,)).to(device=device, dtype=torch.float32)
        f = torch.tensor(m.rot.frequencies(), dtype=torch.float64)
        self.freq = torch.stack([f.float(), (f - f.float().double()).float()], dim=1).contiguous().to(device)

    def run(self, parts, up, meta, cache, layer: int, y: torch.Tensor, act_offset: int) -> None:
        m, ops = self.m, get_ops()
        keys, values = cache.kv[layer]
        q, k, v = (parts[n].unflatten(1, (h, d)) for n, h, d in (("q", m.heads, m.dim), ("k", m.kv_heads, m.dim),
                                                                  ("v", m.kv_heads, m.vdim)))
        ops.rope_norm_cache(q, k, v, keys, values, meta.slot_mapping, meta.positions, self.freq, m.rot.amplitude, self.eps,
                            self.temperature)
        inner = m.heads * m.vdim
        ops.paged_attention_primitive(q, keys, values, m.kv_heads, m.scale, 0.0, meta.block_tables, meta.seq_lens,
                                      meta.cu_seqlens_q, meta.block_size, meta.max_seq_len, m.window if m.window > 0 else -1,
                                      y[:, :inner].unflatten(1, (m.heads, m.vdim)), wide_weights=True, plain_softmax=True,
                                      min_q_len=meta.min_q_len, keep_first=m.keep_first)
        if up is not None or y.shape[1] > inner:
            ops.mixer_finish(y, inner, up, act_offset)


class TimeMixMixer(Mixer):
    """RWKV-style time mixing: five mixes of a row with the row before -> products, the decay's through a bottleneck ->
    recurrence -> per-head norm -> silu gate."""

    MIXES = "rkvgw"

    def __init__(self, m: TimeMixArgs, width: int, eps: float, get: Get, dtype, device) -> None:
        self.m, self.eps = m, eps
        f32 = lambda name, *shape: get(name, shape).to(device=device, dtype=torch.float32).contiguous()  # noqa: E731
        self.mix_weight = torch.stack([f32(f"mu.{s}", width) for s in self.MIXES]).contiguous()
        self.weights = {}
        self.out_weight = get("o", (width, m.inner))
        self.products = BatchedLinear([get(s, (m.inner, width)) for s in self.MIXES[:4]], dtype, device)
        down = get("w1", (None, width))
        self.decay_down = StackedLinear({"w": down}, dtype, device)
        self.decay_up = SideBySideLinear({"w": get("w2", (m.inner, down.shape[0]))}, dtype, device)
        self.decay_bias, self.bonus = f32("w0", m.inner), f32("u", m.heads, m.dim)
        self.norm = f32("norm", m.inner)

    def project(self, mixes: torch.Tensor) -> dict[str, torch.Tensor]:
        r, k, v, g = self.products(mixes[:4])
        z = self.decay_up.operand(mixes.shape[1])
        get_ops().mixer_finish(z, 0, self.decay_down(mixes[4]), act="tanh")
        return {"r": r, "k": k, "v": v, "g": g, "w": self.decay_up.wide(z)}

    def run(self, parts, up, meta, cache, layer: int, y: torch.Tensor, act_offset: int) -> None:
        m, ops = self.m, get_ops()
        o = ops.recurrence("wkv", parts["r"], parts["k"], parts["v"], parts["w"], None, meta, cache.states[layer].matrix,
                           heads=m.heads, groups=m.heads, key_dim=m.dim, value_dim=m.dim, bias_a=self.decay_bias, skip=self.bonus)
        ops.mixer_finish(y, m.inner, up, act_offset, y=o, post_gate=parts["g"], weight=self.norm, group_size=m.dim, eps=self.eps,
                         post="silu")


class BiasedAttentionMixer(Mixer):
    """Causal attention over paged keys and values, all three normed per head: scores fall with the distance, queries grow with
    the position; a sliding window and a sigmoid gate on the output."""

    def __init__(self, m: BiasedAttentionArgs, width: int, eps: float, get: Get, dtype, device) -> None:
        self.m, self.eps = m, eps
        self.weights = {"q": get("q", (m.heads * m.dim, width)), "k": get("k", (m.kv_heads * m.dim, width)),
                        "v": get("v", (m.kv_heads * m.vdim, width)), "g": get("g", (m.heads * m.vdim, width))}
        self.out_weight = get("o", (width, m.heads * m.vdim))
        self.q_norm, self.k_norm = (get(n, (m.dim,)).to(device=device, dtype=torch.float32).contiguous() for n in ("q.norm", "k.norm"))
        self.slopes = torch.tensor(m.slopes(), dtype=torch.float64).to(device=device, dtype=torch.float32)

    def run(self, parts, up, meta, cache, layer: int, y: torch.Tensor, act_offset: int) -> None:
        m, ops = self.m, get_ops()
        keys, values = cache.kv[layer]
        q, k, v = (parts[n].unflatten(1, (h, d)) for n, h, d in (("q", m.heads, m.dim), ("k", m.kv_heads, m.dim),
                                                                  ("v", m.kv_heads, m.vdim)))
        ops.rope_norm_cache(q, k, v, keys, values, meta.slot_mapping, meta.positions, None, 1.0, self.eps, q_norm=self.q_norm,
                            k_norm=self.k_norm, norm_values=True, temperature=(m.temp_coef, m.temp_every))
        inner = m.heads * m.vdim
        ops.paged_attention_primitive(q, keys, values, m.kv_heads, m.scale, 0.0, meta.block_tables, meta.seq_lens,
                                      meta.cu_seqlens_q, meta.block_size, meta.max_seq_len, m.window if m.window > 0 else -1,
                                      y[:, :inner].unflatten(1, (m.heads, m.vdim)), wide_weights=True, plain_softmax=True,
                                      min_q_len=meta.min_q_len, slopes=self.slopes)
        ops.mixer_finish(y, inner, up, act_offset, y=y[:, :inner], post_gate=parts["g"])


class LatentAttentionMixer(Mixer):
    """Latent attention: short segments attend in the latent space (queries are taken there by the keys' up-projection),
    long ones get their visible keys and values expanded first, whichever is the smaller work."""

    def __init__(self, m: LatentAttentionArgs, width: int, eps: float, get: Get, dtype, device) -> None:
        self.m, self.eps = m, eps
        h, d, r, v, rank = m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank
        self.weights = {"q": get("q", (h * (d + r), width)), "dkv": get("dkv", (rank + r, width)),
                        "g": get("g", (h * v, width))}
        self.out_weight = get("o", (width, h * v))
        self.latent_norm = get("dkv.norm", (rank,)).to(device=device, dtype=torch.float32)
        uk = get("uk", (h * d, rank)).to(device=device, dtype=dtype).view(h, d, rank)
        uv = get("uv", (h * v, rank)).to(device=device, dtype=dtype).view(h, v, rank)
        self.to_latent = uk.transpose(1, 2).contiguous()  # [H, rank, dim]: unrotated query -> latent query
        self.from_latent = uv.contiguous()                # [H, vdim, rank]: latent output -> value space
        i = torch.arange(m.rot_dims // 2, dtype=torch.float64)
        self.inv_freq = (m.rot_base ** (-2.0 * i / max(1, m.rot_dims))).to(device=device, dtype=torch.float32)
        # the tile kernel's head size that holds both keys and values (zero columns change neither product)
        self.head = next((n for n in (64, 128) if max(d + r, v) <= n), 0) if dtype == torch.bfloat16 else 0
        self.expand = None
        if self.head:
            # [latent | rotated part] -> [keys of all heads | values of all heads]: the rotated part passes through
            # identity rows, so one product yields finished keys
            w = torch.zeros((2, h, self.head, rank + r), dtype=dtype, device=device)
            w[0, :, :d, :rank] = uk
            w[0, :, d:d + r, rank:] = torch.eye(r, dtype=dtype, device=device)
            w[1, :, :v, :rank] = uv
            self.expand = w.view(2 * h * self.head, rank + r)

    @property
    def expand_from(self) -> int:
        """Rows from which expanding beats attending in the latent space: there the per-key cost of the expansion,
        rank (dk + dv), is paid back by the smaller head (dk + dv instead of 2 rank + rot per row); the tile kernel
        also runs about three times as fast as the latent one."""
        m = self.m
        if not self.head:
            return 1 << 30
        small = m.dim + m.rot_dim + m.vdim
        saved = 2 * m.kv_rank + m.rot_dim - small
        if saved <= 0:
            return 16
        return max(16, m.kv_rank * small // (3 * saved))

    def _short(self, parts, meta, pool, out, n: int, rows: int, longest: int) -> None:
        m, ops = self.m, get_ops()
        q = parts["q"][:rows]
        q_lat = torch.empty((rows, m.heads, m.kv_rank + m.rot_dim), dtype=q.dtype, device=q.device)
        self._prep(q, parts["dkv"][:rows], meta.positions[:rows], meta.slot_mapping[:rows], pool, q_lat, m.kv_rank, False)
        ops.head_linear(q.unflatten(1, (m.heads, -1))[:, :, :m.dim], self.to_latent, q_lat[:, :, :m.kv_rank])
        o = ops.latent_attention(q_lat, pool, meta, m.scale, m.window, m.kv_rank, longest, n)
        ops.head_linear(o, self.from_latent, out[:rows].unflatten(1, (m.heads, m.vdim)), gate=parts["g"][:rows])

    def _prep(self, q, down, positions, slots, pool, q_out, rot_offset: int, copy_nope: bool) -> None:
        m = self.m
        get_ops().latent_prep(q, down, self.latent_norm, positions, slots, self.inv_freq, pool, q_out, heads=m.heads,
                              dim=m.dim, rot_dim=m.rot_dim, kv_rank=m.kv_rank, eps=self.eps, rot_offset=rot_offset,
                              copy_nope=copy_nope)

    def _long(self, parts, meta, pool, plan) -> torch.Tensor:
        m, ops, r0 = self.m, get_ops(), plan.first_row
        q = parts["q"][r0:]
        q_full = torch.empty((q.shape[0], m.heads, self.head), dtype=q.dtype, device=q.device)
        self._prep(q, parts["dkv"][r0:], meta.positions[r0:], meta.slot_mapping[r0:], pool, q_full, m.dim, True)
        rows = torch.empty((plan.rows_total, pool.shape[1]), dtype=pool.dtype, device=pool.device)
        ops.latent_gather(pool, plan.source_tables, plan.first, plan.count, plan.out_row, rows, plan.max_count,
                          meta.block_size, EXPAND_PAGE)
        kv = torch.mm(rows, self.expand.t()).view(-1, EXPAND_PAGE, 2, m.heads, self.head)
        out = torch.empty_like(q_full)
        ops.paged_attention_primitive(
            q_full, kv[:, :, 0], kv[:, :, 1], m.heads, m.scale, 0.0, plan.block_tables, plan.count, plan.cu_seqlens_q,
            EXPAND_PAGE, plan.max_count, m.window if m.window > 0 else -1, out, wide_weights=True, _kernel=3)
        return out.view(q.shape[0], -1)

    def run(self, parts, up, meta, cache, layer: int, y: torch.Tensor, act_offset: int) -> None:
        m, ops, pool = self.m, get_ops(), cache.latent[layer]
        inner = m.heads * m.vdim
        n, rows, longest = meta.split(self.expand_from)
        plan = meta.expand_plan(self.expand_from, m.window)
        if rows:
            self._short(parts, meta, pool, y[:, :inner], n, rows, longest)
            if up is not None or y.shape[1] > inner:
                ops.mixer_finish(y[:rows], inner, None if up is None else up[:rows], act_offset)
        if plan is not None:
            o = self._long(parts, meta, pool, plan)
            ops.mixer_finish(y[rows:], inner, None if up is None else up[rows:], act_offset, y=o,
                             post_gate=parts["g"][rows:], y_head_dim=m.vdim, y_head_stride=self.head)


MIXERS = {c: k for c, k in ((LatentAttentionArgs, LatentAttentionMixer), (Mamba2Args, Mamba2Mixer),
                            (MLSTMArgs, MLSTMMixer), (LightningArgs, LightningMixer),
                            (SoftmaxAttentionArgs, SoftmaxAttentionMixer), (RotaryAttentionArgs, RotaryAttentionMixer),
                            (TimeMixArgs, TimeMixMixer), (BiasedAttentionArgs, BiasedAttentionMixer))}
