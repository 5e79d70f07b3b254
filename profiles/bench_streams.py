#!/usr/bin/env python
"""Hyper-connected decoders (lightning attention, softmax attention beside it) next to the closest transformer of the
framework: whole-model prefill and decode throughput, and every kernel against its roofline.

    python bench.py --streams [--stream-sizes s,m,w]      (or this file directly)

Method as in bench_hybrid.py: CUDA graphs, operand sets larger than L2, CUDA events on the launching stream.
"""

from __future__ import annotations

import json
import os
import sys

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
if ROOT not in sys.path:
    sys.path.insert(0, ROOT)

from profiles.bench_hybrid import L2_BYTES, VOCAB, _events, _segments, graph_us, peaks  # noqa: E402

SIZES = {
    "s": dict(width=2048, heads=16, kv_heads=4, dim=64, vdim=128, lin=(16, 64, 128), ff=5632),
    "m": dict(width=4096, heads=32, kv_heads=8, dim=128, vdim=128, lin=(32, 128, 128), ff=11008),
    "w": dict(width=2560, heads=20, kv_heads=4, dim=80, vdim=160, lin=(20, 64, 96), ff=7168),
}
STREAMS = 4
PATTERN = ("parallel", "lightning") * 4


def config(size: str, pattern=PATTERN) -> dict:
    s = SIZES[size]
    h, k, v = s["lin"]
    lightning = {"heads": h, "dim": k, "vdim": v, "decay": [1.0 - 2.0 ** -(2 + 8 * i / h) for i in range(h)]}
    mixers = {"lightning": lightning,
              "parallel": {"left": {**{n: s[n] for n in ("heads", "kv_heads", "dim", "vdim")}, "scale": s["dim"] ** -0.5},
                           "right": lightning}}
    layers = [{"type": t, "mixer": mixers[t], "mlp": {"kind": "dense", "ff": s["ff"]}} for t in pattern]
    return {"architecture": "Tatazen", "vocab": VOCAB, "width": s["width"], "streams": STREAMS, "norm": {"eps": 1e-5},
            "layers": layers}


def transformer_args(size: str, layers: int):
    """The framework's closest model at equal width, depth, query heads and feed-forward."""
    from vllm_metal_b200.lm.decoder import ModelArgs

    s = SIZES[size]
    head = 128 if s["width"] // s["heads"] >= 128 else 64
    return ModelArgs(f"transformer-{size}", layers, s["width"], s["heads"], s["kv_heads"], head, s["ff"], VOCAB)


def kernel_table(size: str, batch: int = 64, ctx: int = 4096, chunk: int = 2048) -> list[dict]:
    """Every kernel of one layer of each kind, alone: decode (``batch`` rows at ``ctx``) and prefill (one portion of
    ``chunk`` rows that continues at ``ctx``)."""
    import torch

    from vllm_metal_b200.lm.registry import family_of
    from vllm_metal_b200.metal import get_ops

    ops, hbm, tf, _ = get_ops(), *peaks()
    rows = []

    def add(phase, name, us, nbytes=0.0, flops=0.0):
        bound = max(nbytes / (hbm * 1e3), flops / (tf * 1e6))  # us at the measured peaks
        rows.append({"phase": phase, "kernel": name, "us": round(us, 2), "roofline_us": round(bound, 2),
                     "bound": "hbm" if nbytes / (hbm * 1e3) >= flops / (tf * 1e6) else "tensor", "frac": round(bound / us, 3)})

    cfg = config(size, ("parallel",))
    family = family_of(cfg)
    args = family.parse(cfg)
    model = family.load(args, None, torch.bfloat16, "cuda")
    W, S, bf = args.width, args.streams, torch.bfloat16
    lay, m = model.layers[0], args.layers[0].mixer
    a, r = m.left, m.right
    left, right = (b.mixer for b in lay.branches)
    rnd = lambda *s: torch.randn(s, device="cuda").to(bf)  # noqa: E731
    n_sets = lambda nbytes: max(2, min(24, -(-L2_BYTES // nbytes)))  # noqa: E731
    for phase, q_lens, ctxs in (("decode", [1] * batch, [ctx] * batch), ("prefill", [chunk], [ctx + chunk])):
        meta, blocks = _segments(q_lens, ctxs)
        T, n = sum(q_lens), len(q_lens)
        cache = family.make_cache(args, blocks, 16, n, bf, "cuda")
        for t in cache.kv[0]:
            t.normal_()
        decode = phase == "decode"

        # between the sublayers
        step = dict(eps=1e-5, dtype=bf)
        row = W * (2 * S * 4 + 2 * 2)
        xs = [torch.randn((T, S, W), device="cuda") for _ in range(n_sets(T * S * W * 4))]
        y, y2, g = rnd(T, W), rnd(T, W), rnd(T, W)
        pair = dict(lay.mix.writer, y=y, y2=y2, gate=g, y_norm=lay.branches[0].norm, y2_norm=lay.branches[1].norm)
        add(phase, "stream step after a pair of mixers", graph_us([lambda x=x: ops.stream_step(x, pair, lay.feed.reader, **step)
                                                                   for x in xs]), T * (row + 2 * W * 2))
        one = dict(lay.feed.writer, y=y, gate=g)
        shift = dict(shift=lay.shift, previous=cache.previous[0], seg=meta) if decode else {}
        add(phase, "stream step after a feed-forward" + (", token shift" if decode else ""),
            graph_us([lambda x=x: ops.stream_step(x, one, lay.mix.reader, **shift, **step) for x in xs]),
            T * (row + W * 2 + (W * 6 if decode else 0)))
        if not decode:
            hs = [rnd(T, W) for _ in range(n_sets(T * W * 2))]
            add(phase, "token shift", graph_us([lambda h=h: ops.causal_conv(h, lay.shift_taps, None, cache.previous[0],
                                                                            meta, silu=False) for h in hs]), T * W * 4)
        ids = torch.randint(0, VOCAB, (T,), device="cuda", dtype=torch.int32)
        add(phase, "embedding + positions", graph_us([lambda: ops.embed_streams(ids, model.embed, S, meta.positions, model.freq)] * 4),
            T * W * (2 + 4 * S))
        del xs

        def product(name, lin, x):
            out, k = lin.weight.shape
            ws = [lin.weight] + [lin.weight.clone() for _ in range(n_sets(out * k * 2))]
            add(phase, f"{name} {out}x{k} (library)", graph_us([lambda w=w: torch.mm(x, w.t()) for w in ws]),
                2 * (out * k + T * (out + k)), 2.0 * T * out * k)

        h = rnd(T, W)
        for name, lin in (("input product", lay.input), ("residual gate product", lay.gate), ("feed-forward input product", lay.up)):
            product(name, lin, h)
        for name, lin in (("attention output product", lay.branches[0].output), ("lightning output product", lay.branches[1].output),
                          ("feed-forward output product", lay.down)):
            product(name, lin, rnd(T, lin.columns))

        # softmax attention
        kin = lay.input.weight.shape[0]
        stacks = [rnd(T, kin) for _ in range(n_sets(T * kin * 2))]
        ps = [lay.input.split(t) for t in stacks]
        qkv = [[p["left." + c].unflatten(1, (hh, d)) for c, hh, d in (("q", a.heads, a.dim), ("k", a.kv_heads, a.dim),
                                                                      ("v", a.kv_heads, a.vdim))] for p in ps]
        kc, vc = cache.kv[0]
        cols = a.kv_heads * (a.dim + a.vdim)
        add(phase, "attention: head norms, cache write", graph_us([lambda t=t: ops.norm_rope_cache(
            *t, kc, vc, meta.slot_mapping, q_norm_weight=left.q_norm, k_norm_weight=left.k_norm, eps=1e-5) for t in qkv]),
            T * 2 * (2 * a.heads * a.dim + a.kv_heads * a.dim + 2 * cols))
        out = torch.empty((T, a.heads, a.vdim), dtype=bf, device="cuda")
        pairs = sum(c - q + i + 1 for q, c in zip(q_lens, ctxs) for i in range(q))
        caches = [(kc, vc), (kc.clone(), vc.clone())]
        q = qkv[0][0]
        for name, kw in (("attention", dict(wide_weights=True)), ("attention, weights rounded to 16 bits", {})):
            if not kw and (a.dim != a.vdim or a.dim not in (64, 128)):
                continue
            add(phase, name, graph_us([lambda c=c: ops.paged_attention_primitive(
                q, c[0], c[1], a.kv_heads, a.scale, 0.0, meta.block_tables, meta.seq_lens, meta.cu_seqlens_q, 16, max(ctxs), -1, out,
                plain_softmax=True, min_q_len=meta.min_q_len, **kw) for c in caches]), sum(ctxs) * cols * 2 + T * a.heads * (a.dim + a.vdim) * 2,
                2.0 * pairs * a.heads * (a.dim + a.vdim))
        del caches

        # lightning attention
        rs = [{c: p["right." + c] for c in "qkvg"} for p in ps]
        qk, vv = r.heads * r.dim, r.heads * r.vdim
        spans = [lay.input.span(t, "right.q", "right.v") for t in stacks]
        st = cache.states[0].matrix
        state = 2 * n * r.heads * r.dim * r.vdim * 4
        if not decode:
            add(phase, "lightning: silu", graph_us([lambda t=t: ops.mixer_finish(t, 0, t, act="silu") for t in spans]),
                T * (2 * qk + vv) * 4)
        fl = 2.0 * T * r.heads * (64 * r.dim / 2 + 64 * r.vdim / 2 + 2 * r.dim * r.vdim) if not decode else 0
        add(phase, "lightning: recurrence", graph_us([lambda p=p, t=t: ops.recurrence(
            "lightning", p["q"], p["k"], p["v"], None, None, meta, st, heads=r.heads, groups=r.heads, key_dim=r.dim,
            value_dim=r.vdim, rate=right.rate, decay=right.decay, silu=t if decode else None) for p, t in zip(rs, spans)]),
            state + T * (2 * qk + 2 * vv) * 2, fl)
        os_ = [rnd(T, vv) for _ in ps]
        y = lay.branches[1].output.operand(T)
        add(phase, "lightning: norm, gate", graph_us([lambda p=p, o=o: ops.mixer_finish(
            y, vv, y=o, post_gate=p["g"], weight=right.norm, group_size=vv, eps=1e-5) for p, o in zip(rs, os_)]), T * vv * 6)
        ff = args.layers[0].ff
        ups = [lay.up.split(rnd(T, lay.up.weight.shape[0])) for _ in range(n_sets(T * ff * 4))]
        y = lay.down.operand(T)
        add(phase, "feed-forward: silu, product", graph_us([lambda p=p: ops.mixer_finish(y, 0, p["gate"], act="silu", act_mul=p["up"])
                                                            for p in ups]), T * ff * 6)
        del cache, stacks, ps, ups
    assert not ops.recurrence_failed()
    return rows


def like_table(size: str, batch: int, ctx: int, chunk: int) -> list[dict]:
    from profiles import bench_hybrid

    real = bench_hybrid.transformer_args
    bench_hybrid.transformer_args = transformer_args
    try:
        return bench_hybrid.like_table(size, batch, ctx, chunk)
    finally:
        bench_hybrid.transformer_args = real


def whole_model(size: str, kind: str, batch: int, ctx: int, chunk: int, steps: int, warmup: int) -> dict:
    import torch

    from vllm_metal_b200.v1.model_runner import PagedModelRunner

    bf = torch.bfloat16
    per = -(-(ctx + 2 * (steps + warmup) + chunk) // 16) + 1
    blocks = 1 + per * batch
    if kind == "streams":
        from vllm_metal_b200.lm.registry import family_of

        cfg = config(size)
        fam = family_of(cfg)
        args = fam.parse(cfg)
        model = fam.load(args, None, bf, "cuda")
        cache = fam.make_cache(args, blocks, 16, batch, bf, "cuda")
        for kv in cache.kv.values():
            for t in kv:
                t.normal_()
        weights = model.head.weight.numel() + sum(
            lin.weight.numel() for x in model.layers for lin in (x.input, x.gate, x.up, x.down, *(b.output for b in x.branches)))
        bits = 16
    else:
        from vllm_metal_b200.attention.caches.kv_cache import B200PagedKVCache
        from vllm_metal_b200.lm.decoder import Model

        args = transformer_args(size, len(PATTERN))
        model = Model(args, bf, "cuda", prefill_layout=True)
        cache = B200PagedKVCache(args.num_layers, args.n_kv_heads, args.head_dim, blocks, 16, bf, "cuda")
        for t in (*cache.key_caches, *cache.value_caches):
            t.normal_()
        d = args.head_dim
        weights = args.num_layers * (args.hidden * (2 * args.n_heads + 2 * args.n_kv_heads) * d +
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
    one = {"state_slots": [1]} if runner.stateful else {}
    for offset in (0, ctx):
        def run(offset=offset):
            runner.execute([3] * chunk, [], [(tables[0], chunk, offset)], **one)

        for _ in range(3):
            run()
        ms = _events(run, max(3, steps // 4))
        out[f"prefill_ms_at_{offset}"] = round(ms, 3)
        out[f"prefill_tok_s_at_{offset}"] = round(chunk * 1e3 / ms, 1)
    return out


def main(sizes=tuple(SIZES), kernels: bool = True, steps: int = 32, warmup: int = 5, batch: int = 64, ctx: int = 4096,
         chunk: int = 2048) -> dict:
    import torch

    hbm, tf, source = peaks()
    result = {"metric": "hyper-connected decoder prefill / decode tok/s", "unit": "tok/s", "data": "synthetic", "dtype": "bf16",
              "n_gpus": 1, "steps": steps, "warmup": warmup, "peaks": {"hbm_gbs": hbm, "bf16_tflops": tf, "source": source},
              "config": {"batch": batch, "ctx": ctx, "chunk": chunk, "layers": len(PATTERN), "streams": STREAMS, "vocab": VOCAB,
                         "l2_policy": "operand sets larger than L2 (kernels); weights and caches larger than L2 (models)"},
              "sizes": {}}
    for size in sizes:
        entry = {"shape": SIZES[size], "models": []}
        for kind in ("streams", "transformer"):
            entry["models"].append(whole_model(size, kind, batch, ctx, chunk, steps, warmup))
            torch.cuda.empty_cache()
        if kernels:
            entry["kernels"] = kernel_table(size, batch, ctx, chunk) + like_table(size, batch, ctx, chunk)
            torch.cuda.empty_cache()
        result["sizes"][size] = entry
    return result


def show(result: dict) -> str:
    lines = []
    for size, e in result["sizes"].items():
        lines += [f"{size} {json.dumps(m)}" for m in e["models"]]
        lines += [f"{size} {k['phase']:8s} {k['kernel']:58s} {k['us']:9.2f} us  roofline {k['roofline_us']:8.2f} us ({k['bound']})  "
                  f"{k['frac']:.3f}" for k in e.get("kernels", [])]
    return "\n".join(lines)


if __name__ == "__main__":
    print(show(main(tuple(sys.argv[1].split(",")) if len(sys.argv) > 1 else tuple(SIZES))))
