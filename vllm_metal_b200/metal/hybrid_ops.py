"""Operator surface of ``include/b200_hybrid_ops.h``: the mixers of hybrid decoders (latent attention, gated linear
recurrences), the norms / gates either side of them, the residual steps and the routed experts.  ``HybridOps`` is mixed into the object ``get_ops()`` returns;
like there, a CPU tensor or an unsupported size raises and nothing falls back."""

from __future__ import annotations

import ctypes

import torch

from .constants import DTYPE_BF16, DTYPE_F16, DTYPE_F32

_DTYPE = {torch.float32: DTYPE_F32, torch.float16: DTYPE_F16, torch.bfloat16: DTYPE_BF16}
_P, _I, _L, _F, _Z = ctypes.c_void_p, ctypes.c_int32, ctypes.c_int64, ctypes.c_float, ctypes.c_size_t

HYBRID_SYMBOLS = (
    "b200_embed_rows",
    "b200_stream_norm",
    "b200_mixer_finish",
    "b200_causal_conv",
    "b200_recurrence",
    "b200_recurrence_workspace_bytes",
    "b200_recurrence_chunk",
    "b200_recurrence_failed",
    "b200_recurrence_num_launches",
    "b200_latent_prep",
    "b200_head_linear",
    "b200_latent_attention",
    "b200_latent_attention_workspace_bytes",
    "b200_latent_attention_num_launches",
    "b200_latent_attention_failed",
    "b200_latent_gather",
)

STREAM_SYMBOLS = ("b200_embed_streams", "b200_stream_step")

SANDWICH_SYMBOLS = (
    "b200_residual_step",
    "b200_rope_norm_cache",
    "b200_expert_route",
    "b200_expert_plan",
    "b200_expert_product",
    "b200_expert_product_failed",
)

PRENORM_SYMBOLS = ("b200_token_mix",)

EXPERT_TILES = (32, 64, 128)  # pairs per tile of the expert products

RECURRENCE_CHUNKS = (64, 128)  # rows per chunk of the two chunked forms
RECURRENCE_TILE_V = 64


def _struct(name: str, doc: str, **fields):
    flat = []
    for ctype, names in fields.items():
        flat += [(n, {"P": _P, "I": _I, "L": _L, "F": _F, "Z": _Z}[ctype[0]]) for n in names.split()]
    return type(name, (ctypes.Structure,), {"_fields_": flat, "__doc__": doc})


MixerFinishArgs = _struct(
    "MixerFinishArgs", "b200_mixer_finish_args",
    P="y pre_gate post_gate weight act_in out",
    L="y_stride pre_stride post_stride act_stride out_stride",
    I="rows inner group_size act_dim act_offset out_cols y_head_dim y_head_stride",
    F="eps", I2="dtype", P2="act_mul", L2="mul_stride", I3="act_kind post_silu", F2="act_a act_b")
RecurrenceArgs = _struct(
    "RecurrenceArgs", "b200_recurrence_args",
    P="q k v gate_a gate_b bias_a bias_b rate skip state norm_state max_state cu_seqlens seq_lens slots chunk_seq "
      "chunk_row seq_chunk0 out workspace",
    Z="workspace_bytes",
    L="q_stride k_stride v_stride gate_stride out_stride",
    I="kind dtype num_tokens num_seqs num_heads num_groups key_dim value_dim num_chunks chunk seq_limit",
    F="q_scale gate_cap", P2="decay", I2="silu")
StreamStepArgs = _struct(
    "StreamStepArgs", "b200_stream_step_args",
    P="streams y y2 y_norm y2_norm gate gate_bias mix out_weight in_weight norm_weight h shift previous shifted slots "
      "seq_lens row_ids",
    L="y_stride y2_stride gate_stride h_stride shifted_stride",
    I="rows num_streams dim store",
    F="eps", I2="dtype")
LatentPrepArgs = _struct(
    "LatentPrepArgs", "b200_latent_prep_args",
    P="q down norm_weight positions slot_mapping inv_freq cache q_out",
    L="q_stride down_stride q_out_stride num_slots",
    I="num_tokens heads dim rot_dim rot_dims kv_rank q_cols rot_offset copy_nope",
    F="eps", I2="dtype")
ResidualStepArgs = _struct(
    "ResidualStepArgs", "b200_residual_step_args",
    P="x y part_weight extra extra_gate out_norm in_norm h conv_weight state slots seq_lens row_ids",
    L="y_stride extra_stride gate_stride h_stride", I="rows dim parts taps", F="eps", I2="dtype",
    P2="bias table ids add h32 mix_weight mix_state", L2="mix_stride", F2="table_scale", I3="vocab fresh groups mixes")
RopeNormCacheArgs = _struct(
    "RopeNormCacheArgs", "b200_rope_norm_cache_args",
    P="q k v q_weight freq positions slot_mapping key_cache value_cache",
    L="q_stride k_stride v_stride k_block_stride k_token_stride v_block_stride v_token_stride num_blocks",
    I="num_tokens heads kv_heads dim vdim rot_dims block_size", F="rot_factor eps", I2="dtype",
    P2="q_norm k_norm", F2="temp_coef temp_every", I3="norm_values")
ExpertProductArgs = _struct(
    "ExpertProductArgs", "b200_expert_product_args",
    P="x w out shared_x shared_w shared_out pairs first tiles",
    L="x_stride w_stride out_stride shared_x_stride shared_w_stride shared_out_stride",
    I="rows experts top n_out k shared_n_out shared_k tile_rows max_tiles gated dtype kernel")
HeadLinearArgs = _struct(
    "HeadLinearArgs", "b200_head_linear_args",
    P="x w gate y", L="x_stride x_head_stride y_stride y_head_stride gate_stride", I="rows heads n k dtype")
LatentAttnArgs = _struct(
    "LatentAttnArgs", "b200_latent_attn_args",
    P="q cache block_tables seq_lens cu_seqlens out workspace", Z="workspace_bytes",
    L="q_stride out_stride num_slots",
    I="num_tokens num_seqs heads kv_rank rot_dim block_size max_blocks_per_seq max_seq_len window max_q_len dtype "
      "kernel force_splits",
    F="scale")


def bind_hybrid(lib: ctypes.CDLL) -> None:
    vp, i32, i64, f32 = ctypes.c_void_p, ctypes.c_int, ctypes.c_int64, ctypes.c_float
    lib.b200_embed_rows.argtypes = [vp, vp, vp, i32, i32, i32, i64, i32, vp]
    lib.b200_stream_norm.argtypes = [vp, vp, vp, vp, i32, i32, i64, i64, f32, f32, i32, vp]
    lib.b200_causal_conv.argtypes = [vp] * 8 + [i32, i32, i32, i32, i64, i64, i32, i32, vp]
    lib.b200_latent_gather.argtypes = [vp] * 6 + [i32, i32, i32, i32, i32, i64, i32, i32, vp]
    lib.b200_embed_streams.argtypes = [vp] * 5 + [i32] * 5 + [vp]
    for name, struct in (("mixer_finish", MixerFinishArgs), ("stream_step", StreamStepArgs), ("recurrence", RecurrenceArgs),
                         ("latent_prep", LatentPrepArgs), ("head_linear", HeadLinearArgs),
                         ("residual_step", ResidualStepArgs), ("rope_norm_cache", RopeNormCacheArgs),
                         ("expert_product", ExpertProductArgs),
                         ("latent_attention", LatentAttnArgs)):
        getattr(lib, "b200_" + name).argtypes = [ctypes.POINTER(struct), vp]
    for name, struct in (("recurrence", RecurrenceArgs), ("latent_attention", LatentAttnArgs)):
        getattr(lib, f"b200_{name}_workspace_bytes").argtypes = [ctypes.POINTER(struct)]
        getattr(lib, f"b200_{name}_workspace_bytes").restype = ctypes.c_size_t
        getattr(lib, f"b200_{name}_num_launches").argtypes = [ctypes.POINTER(struct)]
    lib.b200_expert_route.argtypes = [vp, i64, vp, vp, vp, i32, i32, i32, f32, i32, vp]
    lib.b200_token_mix.argtypes = [vp] * 7 + [i32] * 4 + [i64] * 3 + [i32, vp]
    lib.b200_expert_plan.argtypes = [vp] * 4 + [i32] * 4 + [vp]
    lib.b200_recurrence_chunk.argtypes = [ctypes.POINTER(RecurrenceArgs)]


def _rows(name: str, t: torch.Tensor, dtype: torch.dtype | None = None) -> torch.Tensor:
    if not t.is_cuda:
        raise RuntimeError(f"{name} must live on a CUDA device; this path has no CPU implementation")
    if t.dim() != 2 or t.stride(1) != 1:
        raise ValueError(f"{name} must be [rows, columns] with unit column stride, got {tuple(t.shape)}")
    if dtype is not None and t.dtype != dtype:
        raise ValueError(f"{name} must be {dtype}, got {t.dtype}")
    return t


def _f32(name: str, t: torch.Tensor | None, n: int) -> int | None:
    if t is None:
        return None
    if not t.is_cuda or t.dtype != torch.float32 or not t.is_contiguous() or t.numel() != n:
        raise ValueError(f"{name} must be {n} contiguous float32 values on the device, got {tuple(t.shape)} {t.dtype}")
    return t.data_ptr()


def _stream() -> int:
    return torch.cuda.current_stream().cuda_stream


class HybridOps:
    """Methods over ``self._lib`` / ``self._check`` / ``self._workspace`` / ``self.launches`` of the operator object."""

    def embed_rows(self, ids: torch.Tensor, table: torch.Tensor) -> torch.Tensor:
        """Rows of ``table`` as an fp32 residual stream ``[T, dim]``."""
        _rows("table", table)
        if ids.dtype != torch.int32 or not table.is_contiguous():
            raise ValueError("embed_rows takes int32 ids and a contiguous table")
        out = torch.empty((ids.shape[0], table.shape[1]), dtype=torch.float32, device=table.device)
        self._check(self._lib.b200_embed_rows(ids.data_ptr(), table.data_ptr(), out.data_ptr(), ids.shape[0],
                                              table.shape[0], table.shape[1], out.stride(0), _DTYPE[table.dtype],
                                              _stream()))
        self.launches += 1
        return out

    def stream_norm(self, x, weight, eps: float, weight_offset: float, out_dtype, rows=None) -> torch.Tensor:
        """RMS norm of the fp32 stream (or of the rows listed in int64 ``rows``)."""
        _rows("x", x, torch.float32)
        if rows is not None and (rows.dtype != torch.int64 or not rows.is_cuda):
            raise ValueError("rows must be int64 on the device")
        n = x.shape[0] if rows is None else rows.shape[0]
        out = torch.empty((n, x.shape[1]), dtype=out_dtype, device=x.device)
        self._check(self._lib.b200_stream_norm(
            x.data_ptr(), None if rows is None else rows.data_ptr(), _f32("weight", weight, x.shape[1]), out.data_ptr(),
            n, x.shape[1], x.stride(0), out.stride(0), float(eps), float(weight_offset), _DTYPE[out_dtype], _stream()))
        self.launches += 1
        return out

    def mixer_finish(self, out, inner: int, act_in=None, act_offset: int = 0, y=None, pre_gate=None, post_gate=None,
                     weight=None, group_size: int = 0, eps: float = 0.0, y_head_dim: int = 0,
                     y_head_stride: int = 0, act: str = "gelu", act_mul=None, act_weights=(0.0, 0.0),
                     post: str = "sigmoid") -> None:
        """Gate -> group norm -> gate (``post``: "sigmoid" / "silu") into ``out[:, :inner]`` and ``act(act_in)`` ("gelu" /
        "silu" / "tanh" / "xielu" with its two ``act_weights``, times ``act_mul``) into ``out[:, act_offset:]``, one launch;
        ``y`` may be given per head with padding (``y_head_dim`` used of every ``y_head_stride`` columns)."""
        _rows("out", out)
        a = MixerFinishArgs()
        for name, t in (("y", y), ("pre_gate", pre_gate), ("post_gate", post_gate), ("act_in", act_in),
                        ("act_mul", act_mul)):
            if t is not None:
                _rows(name, t, out.dtype)
                if t.shape[0] != out.shape[0]:
                    raise ValueError(f"{name} has {t.shape[0]} rows, out {out.shape[0]}")
                setattr(a, name, t.data_ptr())
        a.y_stride = 0 if y is None else y.stride(0)
        a.pre_stride = 0 if pre_gate is None else pre_gate.stride(0)
        a.post_stride = 0 if post_gate is None else post_gate.stride(0)
        a.act_stride = 0 if act_in is None else act_in.stride(0)
        a.weight = _f32("weight", weight, inner)
        a.out, a.out_stride, a.out_cols, a.rows = out.data_ptr(), out.stride(0), out.shape[1], out.shape[0]
        a.inner, a.group_size, a.eps, a.dtype = inner, group_size, float(eps), _DTYPE[out.dtype]
        a.act_dim, a.act_offset = (0 if act_in is None else act_in.shape[1]), act_offset
        a.y_head_dim, a.y_head_stride = y_head_dim, y_head_stride
        a.post_silu, (a.act_a, a.act_b) = ("sigmoid", "silu").index(post), act_weights
        a.act_kind, a.mul_stride = ("gelu", "silu", "tanh", "xielu").index(act), 0 if act_mul is None else act_mul.stride(0)
        if act_mul is not None and act_mul.shape != act_in.shape:
            raise ValueError(f"act_mul is {tuple(act_mul.shape)}, act_in {tuple(act_in.shape)}")
        self._check(self._lib.b200_mixer_finish(ctypes.byref(a), _stream()))
        self.launches += 1

    def recurrence_failed(self) -> bool:
        """Whether a wait inside a tcgen05 kernel of the recurrences ever ran out (synchronises)."""
        return self._lib.b200_recurrence_failed() != 0

    def embed_streams(self, ids, table, num_streams: int, positions=None, freq=None) -> torch.Tensor:
        """Rows of ``table`` (plus the sinusoid of ``positions``: ``freq [pairs, 2]`` holds every frequency's high and
        low part) as ``num_streams`` equal fp32 streams ``[T, S, dim]``."""
        _rows("table", table)
        if ids.dtype != torch.int32 or not table.is_contiguous():
            raise ValueError("embed_streams takes int32 ids and a contiguous table")
        dim = table.shape[1]
        if positions is not None and (positions.dtype != torch.int32 or positions.shape != ids.shape):
            raise ValueError("positions must be int32, one per id")
        out = torch.empty((ids.shape[0], num_streams, dim), dtype=torch.float32, device=table.device)
        self._check(self._lib.b200_embed_streams(
            ids.data_ptr(), table.data_ptr(), None if positions is None else positions.data_ptr(),
            None if positions is None else _f32("freq", freq, 2 * (-(-dim // 2))), out.data_ptr(), ids.shape[0],
            table.shape[0], dim, num_streams, _DTYPE[table.dtype], _stream()))
        self.launches += 1
        return out

    def stream_step(self, streams, result=None, reader=None, *, eps: float, dtype, store: bool = True, rows=None,
                    shift=None, previous=None, seg=None):
        """What lies between two sublayers (one launch).  ``result``: what the last one left -- ``y``, optionally ``y2``
        with ``y_norm`` / ``y2_norm``, ``gate`` / ``gate_bias``, ``mix [S, S]``, ``out_weight [S]`` -- goes into
        ``streams [T, S, dim]``; ``reader`` = ``(in_weight [S], norm_weight [dim])`` of the next one gives its normed
        input, returned as ``(h, shifted)``.  ``shift`` with ``previous [slots, dim]`` and ``seg``: token shift for a batch
        of single rows.  ``rows`` (int64): only these rows are worked on, ``h`` is packed."""
        t, s, dim = streams.shape
        if not streams.is_cuda or streams.dtype != torch.float32 or not streams.is_contiguous():
            raise ValueError("streams must be contiguous float32 [T, S, dim] on the device")
        a = StreamStepArgs()
        a.streams, a.num_streams, a.dim, a.store = streams.data_ptr(), s, dim, int(store)
        a.rows, a.eps, a.dtype = t if rows is None else rows.shape[0], float(eps), _DTYPE[dtype]
        if rows is not None:
            if rows.dtype != torch.int64 or not rows.is_cuda:
                raise ValueError("rows must be int64 on the device")
            a.row_ids = rows.data_ptr()
        if result is not None:
            for name in ("y", "y2", "gate"):
                x = result.get(name)
                if x is not None:
                    _rows(name, x, dtype)
                    if x.shape != (t, dim):
                        raise ValueError(f"{name} is {tuple(x.shape)}, the streams have {t} rows of {dim}")
                    setattr(a, name, x.data_ptr())
                    setattr(a, name + "_stride", x.stride(0))
            for name, n in (("y_norm", dim), ("y2_norm", dim), ("gate_bias", dim), ("mix", s * s), ("out_weight", s)):
                setattr(a, name, _f32(name, result.get(name), n))
        h = shifted = None
        if reader is not None:
            h = torch.empty((a.rows, dim), dtype=dtype, device=streams.device)
            a.h, a.h_stride = h.data_ptr(), h.stride(0)
            a.in_weight, a.norm_weight = _f32("in_weight", reader[0], s), _f32("norm_weight", reader[1], dim)
        if shift is not None:
            if previous.dtype != dtype or previous.shape[1:].numel() != dim or not previous.is_contiguous():
                raise ValueError("previous must be contiguous [slots, (1,) dim] of the activation type")
            if seg.cu_seqlens_q.shape[0] - 1 != t:
                raise ValueError("the fused token shift takes one row per request")
            shifted = torch.empty_like(h)
            a.shift, a.previous = _f32("shift", shift, dim), previous.data_ptr()
            a.shifted, a.shifted_stride = shifted.data_ptr(), shifted.stride(0)
            a.slots, a.seq_lens = seg.state_slots.data_ptr(), seg.seq_lens.data_ptr()
        self._check(self._lib.b200_stream_step(ctypes.byref(a), _stream()))
        self.launches += 1
        return h, shifted

    def residual_step(self, x, result=None, in_norm=None, *, eps: float, dtype, rows=None, conv=None, seg=None, groups: int = 1,
                      embed=None, add=None, mix=None, wide: bool = False):
        """What lies between two sublayers (one launch).  ``result``: what the last one left -- ``y [T, dim]`` (or, with
        ``part_weight [T, parts]``, ``[T * parts, dim]``), optionally ``extra`` with ``extra_gate [T]``, a ``bias [dim]``, and
        its ``norm`` (None: as it is) -- is added to the fp32 stream ``x [T, dim]``; then ``embed`` = (ids, table, scale, fresh)
        -- scaled embedding rows, with which a fresh stream begins -- and the vector ``add``.  ``in_norm`` of the next one, in
        ``groups`` parts of a row, gives its input, returned (``wide``: in fp32).  For a batch of single rows ``conv`` =
        (weights [taps, dim], state) with ``seg``: the input plus its convolution; or ``mix`` = (weights [mixes, dim], fp32
        state [slots, dim]): the input mixed with the row before, ``[mixes, T, dim]``.  ``rows`` (int64): only these rows are
        worked on, the input is packed, ``x`` stays."""
        _rows("x", x, torch.float32)
        t, dim = x.shape
        if not x.is_contiguous():
            raise ValueError("x must be contiguous")
        a = ResidualStepArgs()
        a.x, a.dim, a.eps, a.dtype, a.groups = x.data_ptr(), dim, float(eps), _DTYPE[dtype], groups
        a.rows = t if rows is None else rows.shape[0]
        if rows is not None:
            if rows.dtype != torch.int64 or not rows.is_cuda:
                raise ValueError("rows must be int64 on the device")
            a.row_ids = rows.data_ptr()
        if result is not None:
            y, pw, extra = _rows("y", result["y"], dtype), result.get("part_weight"), result.get("extra")
            a.parts = 0 if pw is None else pw.shape[1]
            if y.shape != (t * max(1, a.parts), dim):
                raise ValueError(f"y is {tuple(y.shape)}, the stream has {t} rows of {dim}")
            a.y, a.y_stride, a.out_norm = y.data_ptr(), y.stride(0), _f32("norm", result.get("norm"), dim)
            a.bias = _f32("bias", result.get("bias"), dim)
            if pw is not None:
                a.part_weight = _f32("part_weight", pw, t * a.parts)
            if extra is not None:
                gate = result["extra_gate"]
                if _rows("extra", extra, dtype).shape != (t, dim) or gate.dtype != torch.float32 or gate.shape != (t,):
                    raise ValueError("extra must be [T, dim] and its gate float32 [T]")
                a.extra, a.extra_stride = extra.data_ptr(), extra.stride(0)
                a.extra_gate, a.gate_stride = gate.data_ptr(), gate.stride(0)
        if embed is not None:
            ids, table, scale, fresh = embed
            if ids.dtype != torch.int32 or ids.shape != (t,) or _rows("table", table, dtype).shape[1] != dim or \
                    not table.is_contiguous():
                raise ValueError(f"embed: int32 ids, one per row, and a contiguous table of {dim} columns")
            a.ids, a.table, a.table_scale = ids.data_ptr(), table.data_ptr(), float(scale)
            a.vocab, a.fresh = table.shape[0], int(fresh)
        a.add = _f32("add", add, dim)
        h = None
        if in_norm is not None:
            a.in_norm = _f32("in_norm", in_norm, dim)
            shape = (a.rows, dim) if mix is None else (mix[0].shape[0], a.rows, dim)
            h = torch.empty(shape, dtype=torch.float32 if wide else dtype, device=x.device)
            a.h_stride = h.stride(-2)
            if wide:
                a.h32 = h.data_ptr()
            else:
                a.h = h.data_ptr()
        if (conv is not None or mix is not None) and seg.cu_seqlens_q.shape[0] - 1 != t:
            raise ValueError("the fused convolution or mix takes one row per request")
        if conv is not None:
            weight, state = conv
            taps = weight.shape[0]
            if state.dtype != dtype or tuple(state.shape[1:]) != (taps - 1, dim) or not state.is_contiguous():
                raise ValueError(f"state must be contiguous [slots, {taps - 1}, {dim}] of the activation type")
            a.conv_weight, a.taps = _f32("conv weight", weight, taps * dim), taps
            a.state = state.data_ptr() if state.numel() else None
        if mix is not None:
            weight, state = mix
            a.mixes, a.mix_weight = weight.shape[0], _f32("mix weight", weight, weight.shape[0] * dim)
            a.mix_state, a.mix_stride = _f32("mix state", state, state.shape[0] * dim), h.stride(0)
        if conv is not None or mix is not None:
            a.slots, a.seq_lens = seg.state_slots.data_ptr(), seg.seq_lens.data_ptr()
        self._check(self._lib.b200_residual_step(ctypes.byref(a), _stream()))
        self.launches += 1
        return h

    def token_mix(self, h, weight, state, seg, dtype) -> torch.Tensor:
        """``h`` (fp32 ``[T, dim]``) mixed with the row before of its segment, once per row of ``weight [mixes, dim]``; the fp32
        ``state [slots, dim]`` carries a segment's last row: ``[mixes, T, dim]`` of ``dtype``."""
        _rows("h", h, torch.float32)
        t, dim = h.shape
        mixes = weight.shape[0]
        out = torch.empty((mixes, t, dim), dtype=dtype, device=h.device)
        self._check(self._lib.b200_token_mix(
            h.data_ptr(), _f32("mix weight", weight, mixes * dim), _f32("mix state", state, state.shape[0] * dim),
            seg.cu_seqlens_q.data_ptr(), seg.seq_lens.data_ptr(), seg.state_slots.data_ptr(), out.data_ptr(),
            seg.cu_seqlens_q.shape[0] - 1, seg.max_q_len, dim, mixes, h.stride(0), out.stride(1), out.stride(0), _DTYPE[dtype],
            _stream()))
        self.launches += 1
        return out

    def rope_norm_cache(self, q, k, v, key_cache, value_cache, slot_mapping, positions, freq, factor: float, eps: float,
                        q_weight=None, *, q_norm=None, k_norm=None, norm_values: bool = False,
                        temperature=(0.0, 1.0)) -> None:
        """Heads rotated (interleaved pairs, ``freq [pairs, 2]`` high and low parts, times ``factor``; None: not at all), then
        divided by their root mean square, queries times ``q_weight [H]``, with weights ``q_norm`` / ``k_norm`` ``[D]``:
        ``q [T, H, D]`` in place, ``k [T, G, D]`` and ``v [T, G, V]`` into the paged caches.  ``norm_values``: value heads are
        divided by theirs as well.  ``temperature`` = (coef, every): queries times 1 + coef ln(floor((p + 1) / every) + 1)."""
        t, heads, dim = q.shape
        groups, vdim = v.shape[1:]
        for name, x in (("q", q), ("k", k), ("v", v)):
            if not x.is_cuda or x.stride(2) != 1 or x.stride(1) != x.shape[2] or x.dtype != key_cache.dtype or x.shape[0] != t:
                raise ValueError(f"{name}: [T, heads, size] rows of the cache's type with contiguous heads, got {tuple(x.shape)}")
        if k.shape[1:] != (groups, dim) or key_cache.shape[2:] != (groups, dim) or value_cache.shape[2:] != (groups, vdim) or \
                key_cache.shape[:2] != value_cache.shape[:2] or key_cache.stride()[2:] != (dim, 1) or \
                value_cache.stride()[2:] != (vdim, 1) or value_cache.dtype != key_cache.dtype:
            raise ValueError("caches must be [num_blocks, block_size, G, D / V] with contiguous rows")
        if positions.dtype != torch.int32 or slot_mapping.dtype != torch.int64 or positions.shape != (t,) or \
                slot_mapping.shape != (t,):
            raise ValueError("positions must be int32 [T] and slot_mapping int64 [T]")
        a = RopeNormCacheArgs()
        a.q, a.k, a.v, a.key_cache, a.value_cache = (x.data_ptr() for x in (q, k, v, key_cache, value_cache))
        a.q_weight = _f32("q_weight", q_weight, heads)
        a.rot_dims = 0 if freq is None else freq.numel()
        a.freq = _f32("freq", freq, freq.numel()) if a.rot_dims else None
        a.q_norm, a.k_norm = _f32("q_norm", q_norm, dim), _f32("k_norm", k_norm, dim)
        a.norm_values, (a.temp_coef, a.temp_every) = int(norm_values), temperature
        a.positions, a.slot_mapping = positions.data_ptr(), slot_mapping.data_ptr()
        a.q_stride, a.k_stride, a.v_stride = q.stride(0), k.stride(0), v.stride(0)
        a.k_block_stride, a.k_token_stride = key_cache.stride()[:2]
        a.v_block_stride, a.v_token_stride = value_cache.stride()[:2]
        a.num_blocks, a.block_size = key_cache.shape[:2]
        a.num_tokens, a.heads, a.kv_heads, a.dim, a.vdim = t, heads, groups, dim, vdim
        a.rot_factor, a.eps, a.dtype = float(factor), float(eps), _DTYPE[q.dtype]
        self._check(self._lib.b200_rope_norm_cache(ctypes.byref(a), _stream()))
        self.launches += 1

    def expert_route(self, logits, correction, experts: int, top: int, scale: float, over_chosen: bool = False):
        """``(chosen int32 [T, top], weights fp32 [T, top])`` of fp32 router logits (their first ``experts`` columns).
        ``over_chosen``: the correction is part of the logits and the weights are the softmax over the chosen ones alone."""
        _rows("logits", logits, torch.float32)
        t = logits.shape[0]
        if logits.shape[1] < experts:
            raise ValueError(f"logits have {logits.shape[1]} columns for {experts} experts")
        chosen = torch.empty((t, top), dtype=torch.int32, device=logits.device)
        weights = torch.empty((t, top), dtype=torch.float32, device=logits.device)
        self._check(self._lib.b200_expert_route(
            logits.data_ptr(), logits.stride(0), _f32("correction", correction, experts), chosen.data_ptr(),
            weights.data_ptr(), t, experts, top, float(scale), int(over_chosen), _stream()))
        self.launches += 1
        return chosen, weights

    def expert_plan(self, chosen, experts: int, tile_rows: int):
        """The (row, place) pairs of ``chosen`` sorted by expert: ``(pairs, first, tiles, tile_rows)``."""
        if chosen.dtype != torch.int32 or not chosen.is_cuda or not chosen.is_contiguous():
            raise ValueError("chosen must be contiguous int32 on the device")
        t, top = chosen.shape
        buf = torch.empty((t * top + 2 * (experts + 1),), dtype=torch.int32, device=chosen.device)
        pairs, first, tiles = buf.split([t * top, experts + 1, experts + 1])
        self._check(self._lib.b200_expert_plan(chosen.data_ptr(), pairs.data_ptr(), first.data_ptr(), tiles.data_ptr(), t,
                                               experts, top, tile_rows, _stream()))
        self.launches += 1
        return pairs, first, tiles, tile_rows

    def expert_product(self, x, weight, plan, top: int, rows: int, *, gated: bool, shared_x=None, shared_weight=None,
                       k: int = 0, shared_k: int = 0, kernel: int = 0):
        """Products of all experts: ``weight [E, n, columns]`` of which ``k`` columns count (0: all).  ``gated``: ``x [rows,
        k]`` through the gate and up halves of ``n``, sorted by expert; else ``x`` sorted, results by pair.  A shared expert's
        ``shared_weight [n', columns]`` runs along (on ``shared_x``, or on ``x`` when gated).  ``(out, shared out or None)``;
        results have whole 8-column rows, of which the last may be padding."""
        pairs, first, tiles, tile_rows = plan
        experts, n, cols = weight.shape
        half = 2 if gated else 1
        _rows("x", x, weight.dtype)
        if not weight.is_contiguous() or x.shape[0] != (rows if gated else rows * top) or x.shape[1] < (k or cols):
            raise ValueError(f"expert_product: x {tuple(x.shape)} and weight {tuple(weight.shape)} disagree")
        up8 = lambda c: -(-c // 8) * 8  # noqa: E731
        empty = lambda r, c: torch.empty((r, up8(c)), dtype=x.dtype, device=x.device)[:, :c]  # noqa: E731
        a = ExpertProductArgs()
        a.x, a.x_stride, a.w, a.w_stride = x.data_ptr(), x.stride(0), weight.data_ptr(), cols
        a.rows, a.experts, a.top, a.n_out, a.k = rows, experts, top, n // half, k or cols
        out = empty(rows * top, n // half)
        a.out, a.out_stride = out.data_ptr(), out.stride(0)
        shared_out = None
        if shared_weight is not None:
            sn, scols = shared_weight.shape
            sx = x if gated else _rows("shared_x", shared_x, x.dtype)
            if sx.shape[0] != rows or not shared_weight.is_contiguous() or sx.shape[1] < (shared_k or scols):
                raise ValueError("expert_product: the shared expert's operands disagree")
            shared_out = empty(rows, sn // half)
            a.shared_x, a.shared_x_stride = sx.data_ptr(), sx.stride(0)
            a.shared_w, a.shared_w_stride = shared_weight.data_ptr(), scols
            a.shared_out, a.shared_out_stride = shared_out.data_ptr(), shared_out.stride(0)
            a.shared_n_out, a.shared_k = sn // half, shared_k or scols
        a.pairs, a.first, a.tiles = pairs.data_ptr(), first.data_ptr(), tiles.data_ptr()
        a.tile_rows, a.max_tiles = tile_rows, rows * top // tile_rows + min(experts, rows * top)
        a.gated, a.dtype, a.kernel = int(gated), _DTYPE[x.dtype], kernel
        self._check(self._lib.b200_expert_product(ctypes.byref(a), _stream()))
        self.launches += 1
        return out, shared_out

    def expert_product_failed(self) -> bool:
        """Whether a wait inside the tcgen05 kernel of the expert products ever ran out (synchronises)."""
        return self._lib.b200_expert_product_failed() != 0

    def causal_conv(self, x, weight, bias, state, seg, silu: bool = True) -> torch.Tensor:
        """Depthwise causal convolution of ``x [T, C]`` over the segments of ``seg`` (carried inputs in
        ``state [slots, taps-1, C]``); ``weight`` fp32 ``[taps, C]``, ``bias`` fp32 ``[C]``."""
        _rows("x", x)
        taps, ch = weight.shape
        if x.shape[1] != ch or state.dtype != x.dtype or tuple(state.shape[1:]) != (taps - 1, ch):
            raise ValueError("causal_conv: x, weight and state disagree")
        out = torch.empty((x.shape[0], ch), dtype=x.dtype, device=x.device)
        self._check(self._lib.b200_causal_conv(
            x.data_ptr(), _f32("weight", weight, taps * ch), _f32("bias", bias, ch),
            state.data_ptr() if state.numel() else None, seg.cu_seqlens_q.data_ptr(), seg.seq_lens.data_ptr(),
            seg.state_slots.data_ptr(), out.data_ptr(), seg.cu_seqlens_q.shape[0] - 1, seg.max_q_len, ch, taps,
            x.stride(0), out.stride(0), int(silu), _DTYPE[x.dtype], _stream()))
        self.launches += 1
        return out

    def recurrence(self, kind: str, q, k, v, gate_a, gate_b, seg, state, *, heads: int, groups: int, key_dim: int,
                   value_dim: int, bias_a=None, bias_b=None, rate=None, skip=None, norm_state=None, max_state=None,
                   q_scale: float = 1.0, gate_cap: float = 0.0, decay=None, silu=None,
                   force_sequential: bool = False, chunk: int = 0) -> torch.Tensor:
        """Linear recurrence (``kind`` "ssd" / "mlstm" gated, "wkv" with decays per head and key channel from the fp32 ``gate_a
        [T, heads * key_dim]`` and ``bias_a``, ``skip`` the current row's bonus, "lightning" with ``decay`` per head and ``rate``
        = -log(decay); there ``silu``, a view that covers q, k and v, says they still have to go through silu: as they are
        read where no chunk is involved, else in place beforehand) over the segments of ``seg``: outputs ``[T, heads *
        value_dim]``, the slots' fp32 states updated in place.  Segments longer than ``seg.chunk_limit`` rows run in
        chunks on tensor cores where type and sizes allow (``chunk``: a form by its rows per chunk, 0 = auto)."""
        a = RecurrenceArgs()
        for name, t in (("q", q), ("k", k), ("v", v), ("gate_a", gate_a), ("gate_b", gate_b)):
            if t is not None:
                _rows(name, t, torch.float32 if kind == "wkv" and name == "gate_a" else v.dtype)
                setattr(a, name, t.data_ptr())
        if kind == "wkv" and gate_a.shape != (v.shape[0], heads * key_dim):
            raise ValueError(f"recurrence: gates must be [T, {heads * key_dim}], got {tuple(gate_a.shape)}")
        if gate_b is not None and gate_b.stride(0) != gate_a.stride(0):
            raise ValueError("both gates must share one row stride")
        if q.shape[1] != groups * key_dim or v.shape[1] != heads * value_dim:
            raise ValueError("recurrence: q / k / v columns do not match the heads")
        slots = state.shape[0]
        if tuple(state.shape) != (slots, heads, key_dim, value_dim):
            raise ValueError(f"state must be [slots, {heads}, {key_dim}, {value_dim}], got {tuple(state.shape)}")
        tiles = -(-value_dim // RECURRENCE_TILE_V)
        wide = heads * (key_dim if kind == "wkv" else 1)
        a.bias_a, a.bias_b = _f32("bias_a", bias_a, wide), _f32("bias_b", bias_b, heads)
        a.rate, a.skip = _f32("rate", rate, heads), _f32("skip", skip, wide)
        a.state = _f32("state", state, state.numel())
        a.norm_state = _f32("norm_state", norm_state, slots * heads * tiles * key_dim)
        a.max_state = _f32("max_state", max_state, slots * heads * tiles)
        a.cu_seqlens, a.seq_lens = seg.cu_seqlens_q.data_ptr(), seg.seq_lens.data_ptr()
        a.slots = seg.state_slots.data_ptr()
        out = torch.empty((v.shape[0], heads * value_dim), dtype=v.dtype, device=v.device)
        a.out, a.out_stride = out.data_ptr(), out.stride(0)
        a.q_stride, a.k_stride, a.v_stride = q.stride(0), k.stride(0), v.stride(0)
        a.gate_stride = 0 if gate_a is None else gate_a.stride(0)
        a.kind, a.dtype = {"ssd": 0, "mlstm": 1, "lightning": 2, "wkv": 3}[kind], _DTYPE[v.dtype]
        a.decay = _f32("decay", decay, heads)
        a.num_tokens, a.num_seqs = v.shape[0], seg.cu_seqlens_q.shape[0] - 1
        a.num_heads, a.num_groups, a.key_dim, a.value_dim = heads, groups, key_dim, value_dim
        a.q_scale, a.gate_cap = float(q_scale), float(gate_cap)
        a.seq_limit = 0x7FFFFFFF
        a.chunk = 0
        if seg.chunks and not force_sequential:
            a.chunk = chunk or self._lib.b200_recurrence_chunk(ctypes.byref(a))
        if silu is not None and not a.chunk:
            a.silu = 1
        elif silu is not None:
            self.mixer_finish(silu, 0, silu, act="silu")
        if a.chunk:
            plan = seg.chunks[a.chunk]
            a.num_chunks = plan.num
            # the sequential launch only exists for the segments that need it
            a.seq_limit = seg.chunk_limit if seg.has_short else 0
            a.chunk_seq, a.chunk_row = plan.seq.data_ptr(), plan.row.data_ptr()
            a.seq_chunk0 = plan.seq0.data_ptr()
            need = self._lib.b200_recurrence_workspace_bytes(ctypes.byref(a))
            ws = self._workspace(v.device, need)
            a.workspace, a.workspace_bytes = ws.data_ptr(), ws.numel()
        self._check(self._lib.b200_recurrence(ctypes.byref(a), _stream()))
        self.launches += self._lib.b200_recurrence_num_launches(ctypes.byref(a))
        return out

    def latent_prep(self, q, down, norm_weight, positions, slot_mapping, inv_freq, cache, q_out, *, heads: int, dim: int,
                    rot_dim: int, kv_rank: int, eps: float, rot_offset: int, copy_nope: bool) -> None:
        """Latent norm + rotation + cache write (``cache [slots, kv_rank + rot_dim]``), and the queries' rotated (with
        ``copy_nope`` also the unrotated) parts into ``q_out [T, heads, columns]``."""
        t = q.shape[0]
        for name, x in (("q", q), ("down", down), ("cache", cache)):
            _rows(name, x, q_out.dtype)
        if not cache.is_contiguous() or cache.shape[1] != kv_rank + rot_dim or down.shape != (t, kv_rank + rot_dim):
            raise ValueError(f"cache and down must have {kv_rank + rot_dim} columns")
        if not q_out.is_contiguous() or q_out.shape[:2] != (t, heads) or q.shape[1] != heads * (dim + rot_dim):
            raise ValueError("q must be [T, heads * (dim + rot_dim)] and q_out contiguous [T, heads, columns]")
        if positions.dtype != torch.int32 or slot_mapping.dtype != torch.int64 or \
                positions.shape != (t,) or slot_mapping.shape != (t,):
            raise ValueError("positions must be int32 [T] and slot_mapping int64 [T]")
        a = LatentPrepArgs()
        a.q, a.down, a.cache, a.q_out = q.data_ptr(), down.data_ptr(), cache.data_ptr(), q_out.data_ptr()
        a.norm_weight = _f32("norm_weight", norm_weight, kv_rank)
        a.positions, a.slot_mapping = positions.data_ptr(), slot_mapping.data_ptr()
        a.inv_freq = _f32("inv_freq", inv_freq, inv_freq.numel()) if inv_freq.numel() else None
        a.rot_dims = 2 * inv_freq.numel()
        a.q_stride, a.down_stride, a.num_slots = q.stride(0), down.stride(0), cache.shape[0]
        a.q_out_stride, a.q_cols = q_out.stride(0), q_out.shape[2]
        a.num_tokens, a.heads, a.dim, a.rot_dim, a.kv_rank = t, heads, dim, rot_dim, kv_rank
        a.rot_offset, a.copy_nope = rot_offset, int(copy_nope)
        a.eps, a.dtype = float(eps), _DTYPE[q.dtype]
        self._check(self._lib.b200_latent_prep(ctypes.byref(a), _stream()))
        self.launches += 1

    def head_linear(self, x, w, y, gate=None) -> None:
        """``y[t, h] = w[h] x[t, h]`` (``w [H, n, k]``), times ``sigmoid(gate[t, h * n + i])``; ``x`` / ``y`` are
        ``[T, H, k]`` / ``[T, H, n]`` views with unit inner stride."""
        h, n, k = w.shape
        if x.shape[1:] != (h, k) or y.shape != (x.shape[0], h, n) or x.stride(2) != 1 or y.stride(2) != 1:
            raise ValueError("head_linear: x [T, H, k], w [H, n, k] and y [T, H, n] disagree")
        if not (x.dtype == w.dtype == y.dtype) or not w.is_contiguous() or not w.is_cuda:
            raise ValueError("head_linear: one dtype and a contiguous w on the device")
        a = HeadLinearArgs()
        a.x, a.w, a.y = x.data_ptr(), w.data_ptr(), y.data_ptr()
        if gate is not None:
            _rows("gate", gate, x.dtype)
            a.gate, a.gate_stride = gate.data_ptr(), gate.stride(0)
        a.x_stride, a.x_head_stride, a.y_stride, a.y_head_stride = x.stride(0), x.stride(1), y.stride(0), y.stride(1)
        a.rows, a.heads, a.n, a.k, a.dtype = x.shape[0], h, n, k, _DTYPE[x.dtype]
        self._check(self._lib.b200_head_linear(ctypes.byref(a), _stream()))
        self.launches += 1

    def latent_attention(self, q, cache, meta, scale: float, window: int, kv_rank: int, max_q_len: int,
                         num_seqs: int | None = None, *, kernel: int = 0, force_splits: int = 0) -> torch.Tensor:
        """Attention of ``q [T, H, kv_rank + rot]`` over the paged latent rows; returns ``[T, H, kv_rank]``.  The
        first ``num_seqs`` segments of ``meta`` cover q's rows; ``window <= 0``: causal only.  ``kernel``: 0 auto,
        1 any-size, 2 warp-level tensor cores, 3 tcgen05 (2 and 3 raise where they do not apply)."""
        t, heads, width = q.shape
        if not q.is_contiguous() or not q.is_cuda or cache.dtype != q.dtype or cache.shape[1] != width:
            raise ValueError("latent_attention: q must be contiguous and match the cache rows")
        out = torch.empty((t, heads, kv_rank), dtype=q.dtype, device=q.device)
        a = LatentAttnArgs()
        a.q, a.cache, a.out = q.data_ptr(), cache.data_ptr(), out.data_ptr()
        a.block_tables, a.seq_lens = meta.block_tables.data_ptr(), meta.seq_lens.data_ptr()
        a.cu_seqlens = meta.cu_seqlens_q.data_ptr()
        a.q_stride, a.out_stride, a.num_slots = q.stride(0), out.stride(0), cache.shape[0]
        a.num_tokens, a.num_seqs = t, meta.seq_lens.shape[0] if num_seqs is None else num_seqs
        a.heads, a.kv_rank, a.rot_dim = heads, kv_rank, width - kv_rank
        a.block_size, a.max_blocks_per_seq = meta.block_size, max(1, meta.block_tables.stride(0))
        a.max_seq_len, a.window, a.max_q_len = meta.max_seq_len, window, max_q_len
        a.dtype, a.kernel, a.force_splits, a.scale = _DTYPE[q.dtype], kernel, force_splits, float(scale)
        need = self._lib.b200_latent_attention_workspace_bytes(ctypes.byref(a))
        ws = self._workspace(q.device, need)
        a.workspace, a.workspace_bytes = (None, 0) if ws is None else (ws.data_ptr(), ws.numel())
        self._check(self._lib.b200_latent_attention(ctypes.byref(a), _stream()))
        self.launches += self._lib.b200_latent_attention_num_launches(ctypes.byref(a))
        return out

    def latent_attention_failed(self) -> bool:
        """Whether a wait inside the tcgen05 kernel ever ran out (synchronises)."""
        return self._lib.b200_latent_attention_failed() != 0

    def latent_gather(self, cache, block_tables, first, count, out_row, out, max_count: int, block_size: int,
                      pad: int) -> None:
        """Cached rows ``first .. first + count`` of every request into consecutive rows of ``out``; the rows up
        to the next multiple of ``pad`` are zeroed."""
        _rows("cache", cache)
        self._check(self._lib.b200_latent_gather(
            cache.data_ptr(), block_tables.data_ptr(), first.data_ptr(), count.data_ptr(), out_row.data_ptr(),
            out.data_ptr(), first.shape[0], max_count, cache.shape[1], block_size, max(1, block_tables.stride(0)),
            cache.shape[0], pad, _DTYPE[cache.dtype], _stream()))
        self.launches += 1
