#!/usr/bin/env python
"""Hybrid decoders (latent attention / Mamba-2 / mLSTM layers) beside the closest transformer of the framework:
whole-model prefill and decode throughput, and every kernel against its roofline.

    python bench.py --hybrid [--hybrid-sizes s,m] [--hybrid-kernels]      (or this file directly)

Whole-model decode: one CUDA-graph step for the batch, replayed with device-side token feedback; prefill: one chunk
through ``PagedModelRunner.execute``.  Kernel times: calls over as many operand sets as exceed the 126 MB L2, captured in
one CUDA graph, CUDA events around the replays.
"""

from __future__ import annotations

import json
import os
import sys

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
if ROOT not in sys.path:
    sys.path.insert(0, ROOT)

L2_BYTES = 126 << 20

SIZES = {
    # width, mamba2 heads, mlstm heads, latent heads, ff, window
    "s": dict(width=2048, mamba=64, mlstm=4, latent=16, ff=8192, window=1024),
    "m": dict(width=4096, mamba=128, mlstm=8, latent=32, ff=16384, window=4096),
}
VOCAB = 32000
PATTERN = ("mamba2", "mlstm", "latent_attention", "latent_attention") * 2


def config(size: str, pattern=PATTERN) -> dict:
    s = SIZES[size]
    mixers = {
        "mamba2": {"heads": s["mamba"], "groups": 8, "state": 128, "vdim": 64, "conv": 4, "norm_groups": 8},
        "mlstm": {"heads": s["mlstm"], "dim": 256, "vdim": 512, "gate_cap": 15.0},
        "latent_attention": {"heads": s["latent"], "dim": 64, "rot_dim": 64, "vdim": 128, "kv_rank": 512,
                             "scale": 128 ** -0.5, "rot": {"base": 10000.0, "dims": 64}, "mask": {"size": s["window"]}},
    }
    layers = [{"type": k, "mixer": mixers[k], "mlp": {"kind": "dense", "ff": s["ff"]}} for k in pattern]
    return {"architecture": "Mapuvik", "vocab": VOCAB, "width": s["width"], "norm": {"eps": 1e-5}, "layers": layers}


def peaks() -> tuple[float, float, str]:
    try:
        with open(os.path.join(ROOT, "MEASURED_PEAKS.json"), encoding="utf-8") as f:
            p = json.load(f)
        return float(p["hbm_gbs"]), float(p["bf16_tflops"]), "measured"
    except (OSError, KeyError, ValueError):
        return 6650.0, 1590.0, "fallback"


def graph_us(calls, reps: int = 20, warmup: int = 3) -> float:
    """Microseconds per call of a list of closures captured in one CUDA graph."""
    import torch

    s = torch.cuda.Stream()
    s.wait_stream(torch.cuda.current_stream())
    with torch.cuda.stream(s):
        for c in calls:
            c()
    torch.cuda.current_stream().wait_stream(s)
    torch.cuda.synchronize()
    g = torch.cuda.CUDAGraph()
    with torch.cuda.graph(g):
        for c in calls:
            c()
    for _ in range(warmup):
        g.replay()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    torch.cuda.synchronize()
    a.record()
    for _ in range(reps):
        g.replay()
    b.record()
    torch.cuda.synchronize()
    return a.elapsed_time(b) * 1e3 / (reps * len(calls))


def _segments(q_lens, ctx, block=16):
    import torch

    from vllm_metal_b200.attention.context import PagedAttentionContext
    from vllm_metal_b200.attention.impls.segments import segment_metadata

    cu, tables, at, mapping = [0], [], 1, []
    for q, c in zip(q_lens, ctx):
        k = -(-c // block)
        t = list(range(at, at + k))
        at += k
        tables.append(t)
        cu.append(cu[-1] + q)
        mapping += [t[p // block] * block + p % block for p in range(c - q, c)]
    c = PagedAttentionContext(slot_mapping=mapping, block_tables=tables, context_lens=list(ctx), cu_seqlens=cu,
                              offsets=[c - q for q, c in zip(q_lens, ctx)], state_slots=list(range(1, len(ctx) + 1)))
    return segment_metadata(c, block, torch.device("cuda")), at


def kernel_table(size: str, batch: int = 64, ctx: int = 4096, chunk: int = 2048) -> list[dict]:
    """Every kernel of one layer of each kind at this size, alone: decode (``batch`` rows at ``ctx``) and prefill (one
    chunk of ``chunk`` rows that continues at ``ctx``)."""
    import torch

    from vllm_metal_b200.lm.hybrid import HybridModel
    from vllm_metal_b200.lm.registry import family_of
    from vllm_metal_b200.metal import get_ops

    ops, hbm, tf, _ = get_ops(), *peaks()
    rows = []

    def add(phase, name, us, nbytes=0.0, flops=0.0):
        bound = max(nbytes / (hbm * 1e3), flops / (tf * 1e6))  # us at the measured peaks
        rows.append({"phase": phase, "kernel": name, "us": round(us, 2), "roofline_us": round(bound, 2),
                     "bound": "hbm" if nbytes / (hbm * 1e3) >= flops / (tf * 1e6) else "tensor",
                     "frac": round(bound / us, 3)})

    cfg = config(size, ("mamba2", "mlstm", "latent_attention"))
    family = family_of(cfg)
    args = family.parse(cfg)
    from vllm_metal_b200.lm.hybrid_random import random_tensors

    model = HybridModel(args, random_tensors(args, "cuda", 1), torch.bfloat16, "cuda")
    W, bf = args.width, torch.bfloat16
    for phase, q_lens, ctxs in (("decode", [1] * batch, [ctx] * batch), ("prefill", [chunk], [ctx + chunk])):
        meta, blocks = _segments(q_lens, ctxs)
        T = sum(q_lens)
        cache = family.make_cache(args, blocks, 16, len(q_lens), bf, "cuda")
        for p in cache.latent.values():
            p.normal_()
        x = torch.randn((T, W), device="cuda")
        n_x = max(1, -(-L2_BYTES // (x.numel() * 6)))
        xs = [torch.randn((T, W), device="cuda") for _ in range(min(n_x, 64))]
        add(phase, "stream_norm", graph_us([lambda x=x: ops.stream_norm(x, model.final_norm, 1e-5, 1.0, bf) for x in xs]),
            T * W * 6)
        for li, layer in enumerate(model.layers):
            m, lay = args.layers[li].mixer, model.layers[li]
            h = torch.randn((T, W), device="cuda").to(bf)
            kin, kout = lay.input.weight.shape[0], lay.output.columns
            copies = max(2, -(-L2_BYTES // (lay.input.weight.numel() * 2)))
            ws = [lay.input.weight] + [lay.input.weight.clone() for _ in range(copies - 1)]
            add(phase, f"{m.kind}: input product {kin}x{W} (library)", graph_us([lambda w=w: torch.mm(h, w.t()) for w in ws]),
                2 * (kin * W + T * (W + kin)), 2.0 * T * kin * W)
            ws = [lay.output.weight] + [lay.output.weight.clone() for _ in range(copies)]
            y0 = torch.randn((T, kout), device="cuda").to(bf)
            add(phase, f"{m.kind}: output product {W}x{kout} + residual (library)",
                graph_us([lambda w=w: torch.addmm(x, y0, w.t(), out_dtype=torch.float32, out=x) for w in ws]),
                2 * (kout * W + T * kout) + 8 * T * W, 2.0 * T * kout * W)
            del ws
            proj_bytes = T * kin * 2
            sets = max(2, min(16, -(-L2_BYTES // proj_bytes)))
            ps = [lay.input.split(torch.randn((T, kin), device="cuda").to(bf)) for _ in range(sets)]
            y = lay.output.operand(T)
            act = T * args.layers[li].ff * 4
            if m.kind == "mamba2":
                st, mx = cache.states[li], lay.mixer
                n, v, inner, ch = m.state, m.vdim, m.inner, m.conv_channels
                sp = [p["in"].split([inner, ch, m.heads], dim=1) for p in ps]
                add(phase, "mamba2: causal_conv", graph_us([lambda p=p: ops.causal_conv(p[1], mx.conv_w, mx.conv_b, st.conv, meta)
                                                             for p in sp]), T * ch * 4 + len(q_lens) * 3 * ch * 4)
                cv = [torch.randn((T, ch), device="cuda").to(bf).split([inner, m.groups * n, m.groups * n], dim=1) for _ in ps]
                state = 2 * len(q_lens) * m.heads * n * v * 4
                fl = 2.0 * T * m.heads * (64 * n / 2 + 64 * v / 2 + 2 * n * v) if phase == "prefill" else 0
                add(phase, "mamba2: recurrence", graph_us([lambda p=p, c=c: ops.recurrence(
                    "ssd", c[2], c[1], c[0], p[2], None, meta, st.matrix, heads=m.heads, groups=m.groups, key_dim=n,
                    value_dim=v, bias_a=mx.dt_bias, rate=mx.rate, skip=mx.skip) for p, c in zip(sp, cv)]),
                    state + T * (2 * inner + 2 * m.groups * n) * 2, fl)
                o = [torch.randn((T, inner), device="cuda").to(bf) for _ in ps]
                add(phase, "mamba2: gate, norm, gelu", graph_us([lambda p=p, s=s, q=q: ops.mixer_finish(
                    y, inner, p["mlp.up"], lay.act_offset, y=q, pre_gate=s[0], weight=mx.norm, group_size=inner // m.norm_groups,
                    eps=1e-5) for p, s, q in zip(ps, sp, o)]), T * inner * 6 + act)
            elif m.kind == "mlstm":
                st, mx = cache.states[li], lay.mixer
                qk, vv = m.heads * m.dim, m.heads * m.vdim
                state = 2 * len(q_lens) * m.heads * m.dim * m.vdim * 4
                fl = 2.0 * T * m.heads * (64 * m.dim / 2 + 64 * m.vdim / 2 + 2 * m.dim * m.vdim) if phase == "prefill" else 0
                add(phase, "mlstm: recurrence", graph_us([lambda p=p: ops.recurrence(
                    "mlstm", p["q"], p["k"], p["v"], p["i"], p["f"], meta, st.matrix, heads=m.heads, groups=m.heads,
                    key_dim=m.dim, value_dim=m.vdim, bias_a=mx.i_bias, bias_b=mx.f_bias, norm_state=st.normaliser,
                    max_state=st.maximum, q_scale=m.dim ** -0.5, gate_cap=m.gate_cap) for p in ps]),
                    state + T * (2 * qk + 2 * vv) * 2, fl)
                o = [torch.randn((T, vv), device="cuda").to(bf) for _ in ps]
                add(phase, "mlstm: norm, gate, gelu", graph_us([lambda p=p, q=q: ops.mixer_finish(
                    y, vv, p["mlp.up"], lay.act_offset, y=q, post_gate=p["g"], weight=mx.norm, group_size=m.vdim, eps=1e-5)
                    for p, q in zip(ps, o)]), T * vv * 6 + act)
            else:
                _latent_rows(ops, add, phase, m, lay, ps, meta, cache.latent[li], y, T, q_lens, ctxs, act)
        del cache
    return rows


def like_table(size: str, batch: int = 64, ctx: int = 4096, chunk: int = 2048) -> list[dict]:
    """The closest transformer's kernels of the same kinds at the same sizes: what the table above is held against."""
    import torch

    from vllm_metal_b200.metal import get_ops

    ops, hbm, tf, _ = get_ops(), *peaks()
    a, bf, rows = transformer_args(size, 1), torch.bfloat16, []
    H, Hk, D = a.n_heads, a.n_kv_heads, a.head_dim

    def add(phase, name, us, nbytes=0.0, flops=0.0):
        bound = max(nbytes / (hbm * 1e3), flops / (tf * 1e6))
        rows.append({"phase": phase, "kernel": "like: " + name, "us": round(us, 2), "roofline_us": round(bound, 2),
                     "bound": "hbm" if nbytes / (hbm * 1e3) >= flops / (tf * 1e6) else "tensor", "frac": round(bound / us, 3)})

    for phase, q_lens, ctxs in (("decode", [1] * batch, [ctx] * batch), ("prefill", [chunk], [ctx + chunk])):
        meta, blocks = _segments(q_lens, ctxs)
        T = sum(q_lens)
        sets = max(2, min(32, L2_BYTES // (T * a.hidden * 4)))
        r = lambda *s: torch.randn(s, device="cuda").to(bf)  # noqa: E731
        w = torch.ones(a.hidden, dtype=bf, device="cuda")
        xs, res = [r(T, a.hidden) for _ in range(sets)], [r(T, a.hidden) for _ in range(sets)]
        add(phase, "rms_norm + residual", graph_us([lambda x=x, y=y: ops.rms_norm(x, w, 1e-5, residual=y)
                                                     for x, y in zip(xs, res)]), T * a.hidden * 8)
        gu = [r(T, 2 * a.intermediate) for _ in range(max(2, min(16, L2_BYTES // (T * a.intermediate * 4))))]
        add(phase, "silu_mul", graph_us([lambda g=g: ops.silu_mul(g) for g in gu]), T * a.intermediate * 6)
        kc, vc = r(blocks, 16, Hk, D), r(blocks, 16, Hk, D)
        qkv = [r(T, (H + 2 * Hk) * D) for _ in range(max(2, min(16, L2_BYTES // (T * (H + 2 * Hk) * D * 2))))]
        parts = [[z.reshape(T, -1, D) for z in t.split([H * D, Hk * D, Hk * D], 1)] for t in qkv]
        add(phase, "norm_rope_cache", graph_us([lambda p=p: ops.norm_rope_cache(
            *p, kc, vc, meta.slot_mapping, positions=meta.positions, rot_dim=D, base=1e4) for p in parts]),
            T * ((2 * H + Hk) * D * 2 + 4 * Hk * D * 2))
        q, out = r(T, H, D), torch.empty((T, H, D), dtype=bf, device="cuda")
        caches = [(kc, vc), (kc.clone(), vc.clone())]
        pairs = sum(c - n + i + 1 for n, c in zip(q_lens, ctxs) for i in range(n))
        add(phase, "paged attention", graph_us([lambda c=c: ops.paged_attention_primitive(
            q, c[0], c[1], Hk, D ** -0.5, 0.0, meta.block_tables, meta.seq_lens, meta.cu_seqlens_q, 16, max(ctxs), -1, out)
            for c in caches]), sum(ctxs) * Hk * D * 4 + T * H * D * 4, 4.0 * pairs * H * D)
    return rows


def _latent_rows(ops, add, phase, m, lay, ps, meta, pool, y, T, q_lens, ctxs, act) -> None:
    import torch

    from vllm_metal_b200.attention.impls.segments import EXPAND_PAGE

    bf, mx = torch.bfloat16, lay.mixer
    H, width, inner = m.heads, m.kv_rank + m.rot_dim, m.heads * m.vdim
    window = m.window or max(ctxs)
    prep_bytes = T * (H * (m.dim + m.rot_dim) * 2 + width * 4)
    if phase == "decode":
        q_lat = torch.randn((T, H, width), device="cuda").to(bf)
        add(phase, "latent: norm, rotation, cache write", graph_us([lambda p=p: mx._prep(
            p["q"], p["dkv"], meta.positions, meta.slot_mapping, pool, q_lat, m.kv_rank, False) for p in ps]),
            prep_bytes + T * H * m.rot_dim * 2)
        add(phase, "latent: queries to latent space", graph_us([lambda p=p: ops.head_linear(
            p["q"].unflatten(1, (H, -1))[:, :, :m.dim], mx.to_latent, q_lat[:, :, :m.kv_rank]) for p in ps]),
            2 * (mx.to_latent.numel() + T * H * (m.dim + m.kv_rank)), 2.0 * T * mx.to_latent.numel())
        keys = sum(min(window, c) for c in ctxs)
        pools = [pool] + [pool.clone() for _ in range(1)]
        add(phase, "latent: attention", graph_us([lambda c=c: ops.latent_attention(
            q_lat, c, meta, m.scale, m.window, m.kv_rank, 1) for c in pools]),
            keys * width * 2 + T * H * (width + m.kv_rank) * 2, 2.0 * keys * H * (width + m.kv_rank))
        o = torch.randn((T, H, m.kv_rank), device="cuda").to(bf)
        add(phase, "latent: outputs to value space, gate", graph_us([lambda p=p: ops.head_linear(
            o, mx.from_latent, y[:, :inner].unflatten(1, (H, m.vdim)), gate=p["g"]) for p in ps]),
            2 * (mx.from_latent.numel() + T * H * (m.kv_rank + 2 * m.vdim)), 2.0 * T * mx.from_latent.numel())
        add(phase, "latent: gelu", graph_us([lambda p=p: ops.mixer_finish(y, inner, p["mlp.up"], lay.act_offset) for p in ps]), act)
        return
    plan = meta.expand_plan(mx.expand_from, m.window)
    q_full = torch.randn((T, H, mx.head), device="cuda").to(bf)
    add(phase, "latent: norm, rotation, cache write, queries", graph_us([lambda p=p: mx._prep(
        p["q"], p["dkv"], meta.positions, meta.slot_mapping, pool, q_full, m.dim, True) for p in ps]),
        prep_bytes + T * H * mx.head * 2)
    rows = torch.empty((plan.rows_total, width), dtype=bf, device="cuda")
    add(phase, "latent: page gather", graph_us([lambda: ops.latent_gather(
        pool, plan.source_tables, plan.first, plan.count, plan.out_row, rows, plan.max_count, meta.block_size, EXPAND_PAGE)] * 4),
        plan.rows_total * width * 4)
    add(phase, "latent: key / value expansion (library)", graph_us([lambda: torch.mm(rows, mx.expand.t())] * 4),
        2 * (rows.numel() + mx.expand.numel() + plan.rows_total * mx.expand.shape[0]),
        2.0 * plan.rows_total * mx.expand.numel())
    kvs = [torch.mm(rows, mx.expand.t()).view(-1, EXPAND_PAGE, 2, H, mx.head) for _ in range(3)]
    out = torch.empty_like(q_full)
    pairs = sum(min(window, c - q + i + 1) for q, c in zip(q_lens, ctxs) for i in range(q))
    add(phase, "latent: attention over expanded keys", graph_us([lambda kv=kv: ops.paged_attention_primitive(
        q_full, kv[:, :, 0], kv[:, :, 1], H, m.scale, 0.0, plan.block_tables, plan.count, plan.cu_seqlens_q, EXPAND_PAGE,
        plan.max_count, m.window if m.window > 0 else -1, out, wide_weights=True, _kernel=3) for kv in kvs]),
        2 * (2 * kvs[0].numel() // 2 + 2 * q_full.numel()), 2.0 * pairs * H * (m.dim + m.rot_dim + m.vdim))
    add(phase, "latent: the same, weights rounded to 16 bits", graph_us([lambda kv=kv: ops.paged_attention_primitive(
        q_full, kv[:, :, 0], kv[:, :, 1], H, m.scale, 0.0, plan.block_tables, plan.count, plan.cu_seqlens_q, EXPAND_PAGE,
        plan.max_count, m.window if m.window > 0 else -1, out, _kernel=3) for kv in kvs]),
        2 * (2 * kvs[0].numel() // 2 + 2 * q_full.numel()), 2.0 * pairs * H * (m.dim + m.rot_dim + m.vdim))
    o = out.view(T, -1)
    add(phase, "latent: gate, gelu", graph_us([lambda p=p: ops.mixer_finish(
        y, inner, p["mlp.up"], lay.act_offset, y=o, post_gate=p["g"], y_head_dim=m.vdim, y_head_stride=mx.head) for p in ps]),
        T * inner * 6 + act)


def transformer_args(size: str, layers: int):
    """The framework's closest model at equal width, depth, heads and feed-forward parameters (SwiGLU's three matrices
    against two)."""
    from vllm_metal_b200.lm.decoder import ModelArgs

    s = SIZES[size]
    return ModelArgs(f"transformer-{size}", layers, s["width"], s["latent"], max(1, s["latent"] // 4), 128,
                     -(-s["ff"] * 2 // 3 // 256) * 256, VOCAB)


def _events(run, steps: int) -> float:
    import torch

    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    torch.cuda.synchronize()
    a.record()
    for _ in range(steps):
        run()
    b.record()
    torch.cuda.synchronize()
    return a.elapsed_time(b) / steps


def whole_model(size: str, kind: str, batch: int, ctx: int, chunk: int, steps: int, warmup: int) -> dict:
    import dataclasses

    import torch

    from vllm_metal_b200.v1.model_runner import PagedModelRunner

    bf = torch.bfloat16
    per = -(-(ctx + 2 * (steps + warmup) + chunk) // 16) + 1
    blocks = 1 + per * batch
    if kind == "hybrid":
        from vllm_metal_b200.lm.registry import family_of

        cfg = config(size)
        fam = family_of(cfg)
        args = fam.parse(cfg)
        model = fam.load(args, None, bf, "cuda")
        cache = fam.make_cache(args, blocks, 16, batch, bf, "cuda")
        for p in cache.latent.values():
            p.normal_()
        weights = sum(x.input.weight.numel() + x.output.weight.numel() for x in model.layers) + model.head.weight.numel()
        bits = 16
    else:
        from vllm_metal_b200.attention.caches.kv_cache import B200PagedKVCache
        from vllm_metal_b200.lm.decoder import Model

        args = dataclasses.replace(transformer_args(size, len(PATTERN)))
        model = Model(args, bf, "cuda", prefill_layout=True)
        cache = B200PagedKVCache(args.num_layers, args.n_kv_heads, args.head_dim, blocks, 16, bf, "cuda")
        for t in (*cache.key_caches, *cache.value_caches):
            t.normal_()
        d = args.head_dim
        weights = args.num_layers * (args.hidden * (args.n_heads + 2 * args.n_kv_heads) * d + args.hidden * args.n_heads * d +
                                     3 * args.hidden * args.intermediate) + args.vocab * args.hidden
        bits = args.bits
    runner = PagedModelRunner(model, cache, max_batch=batch, max_model_len=per * 16)
    tables = [list(range(1 + i * per, 1 + (i + 1) * per)) for i in range(batch)]
    slots = {"state_slots": list(range(1, batch + 1))} if runner.stateful else {}
    runner.fill_decode([1] * batch, tables, [ctx] * batch, *slots.values())
    runner.buf.upload()
    limit = ctx + 2 * (steps + warmup) + 1
    for _ in range(warmup):
        runner.run_decode(batch, limit, advance=True)
    ms = _events(lambda: runner.run_decode(batch, limit, advance=True), steps)
    out = {"model": kind, "weights": weights, "weight_bits": bits, "decode_ms": round(ms, 3),
           "decode_tok_s": round(batch * 1e3 / ms, 1), "decode_launches": next(iter(runner.launches_per_graph.values()))}
    ids = [3] * chunk
    one = {"state_slots": [1]} if runner.stateful else {}
    for offset in (0, ctx):
        def run(offset=offset):
            runner.execute(ids, [], [(tables[0], chunk, offset)], **one)

        for _ in range(3):
            run()
        ms = _events(run, max(3, steps // 8))
        out[f"prefill_ms_at_{offset}"] = round(ms, 3)
        out[f"prefill_tok_s_at_{offset}"] = round(chunk * 1e3 / ms, 1)
    return out


def main(sizes=("s", "m"), kernels: bool = True, steps: int = 32, warmup: int = 5, batch: int = 64, ctx: int = 4096,
         chunk: int = 2048) -> dict:
    import torch

    hbm, tf, source = peaks()
    result = {"metric": "hybrid decoder prefill / decode tok/s", "unit": "tok/s", "data": "synthetic", "dtype": "bf16",
              "n_gpus": 1, "steps": steps, "warmup": warmup, "peaks": {"hbm_gbs": hbm, "bf16_tflops": tf, "source": source},
              "config": {"batch": batch, "ctx": ctx, "chunk": chunk, "layers": len(PATTERN), "vocab": VOCAB,
                         "l2_policy": "operand sets larger than L2 (kernels); weights and caches larger than L2 (models)"},
              "sizes": {}}
    for size in sizes:
        entry = {"shape": SIZES[size], "models": []}
        for kind in ("hybrid", "transformer"):
            entry["models"].append(whole_model(size, kind, batch, ctx, chunk, steps, warmup))
            torch.cuda.empty_cache()
        if kernels:
            entry["kernels"] = kernel_table(size, batch, ctx, chunk) + like_table(size, batch, ctx, chunk)
            torch.cuda.empty_cache()
        result["sizes"][size] = entry
    return result


if __name__ == "__main__":
    r = main(tuple(sys.argv[1].split(",")) if len(sys.argv) > 1 else ("s", "m"))
    for size, e in r["sizes"].items():
        for m in e["models"]:
            print(size, json.dumps(m))
        for k in e.get("kernels", []):
            print(f"{size} {k['phase']:8s} {k['kernel']:62s} {k['us']:9.2f} us  roofline {k['roofline_us']:8.2f} us "
                  f"({k['bound']})  {k['frac']:.3f}")
