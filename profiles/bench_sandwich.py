#!/usr/bin/env python
"""Sandwich-norm decoders (windowed attention with kept first tokens, routed experts beside a shared one) next to the closest
model of the framework, the transformer with routed int4 experts: whole-model prefill and decode throughput, and every kernel
against its roofline.

    python bench.py --sandwich [--sandwich-sizes s,m,w]      (or this file directly)

Method as in bench_hybrid.py: CUDA graphs, operand sets larger than L2, CUDA events on the launching stream.  The
transformer's expert block reads its row counts back to the host, so it runs eagerly.
"""

from __future__ import annotations

import json
import os
import sys

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
if ROOT not in sys.path:
    sys.path.insert(0, ROOT)

from profiles.bench_hybrid import L2_BYTES, VOCAB, _events, _segments, graph_us, peaks  # noqa: E402
from profiles.bench_streams import show  # noqa: E402

SIZES = {
    "s": dict(width=2048, heads=32, kv_heads=4, dim=64, vdim=64, window=1024, keep=16, experts=64, top=6, ff=768, shared=1536),
    "m": dict(width=4096, heads=32, kv_heads=8, dim=128, vdim=128, window=4096, keep=64, experts=64, top=8, ff=1536, shared=3072),
    "w": dict(width=2880, heads=64, kv_heads=8, dim=64, vdim=64, window=128, keep=4, experts=32, top=4, ff=2880, shared=2880),
}
LAYERS = 4
TAPS = 4


def config(size: str, layers: int = LAYERS) -> dict:
    s = SIZES[size]
    mixer = {**{n: s[n] for n in ("heads", "kv_heads", "dim", "vdim")}, "scale": s["dim"] ** -0.5,
             "rot": {"base": 5e5, "dims": s["dim"], "scaling": {"factor": 4.0, "original": 8192, "fast": 32.0, "slow": 1.0}},
             "mask": {"size": s["window"], "keep_first": s["keep"]}}
    mlp = {"kind": "moe", "expert": {"ff": s["ff"]}, "router": {"experts": s["experts"], "top": s["top"], "scale": 2.0},
           "shared": {"ff": s["shared"]}}
    return {"architecture": "Kerolorn", "vocab": VOCAB, "width": s["width"], "canon": {"taps": TAPS}, "logit_scale": 0.5,
            "norm": {"eps": 1e-5}, "layers": [{"type": "attention", "mixer": mixer, "mlp": mlp}] * layers}


def transformer_args(size: str, layers: int = LAYERS):
    """The framework's closest model at equal width, depth, heads, window and experts (it has no shared expert)."""
    from vllm_metal_b200.lm.decoder import ModelArgs

    s = SIZES[size]
    return ModelArgs(f"transformer-{size}", layers, s["width"], s["heads"], s["kv_heads"], s["dim"], s["ff"], VOCAB,
                     sliding_window=s["window"], layer_types=["sliding_attention"] * layers, num_experts=s["experts"],
                     experts_per_tok=s["top"], moe_routing="softmax_topk")


def kernel_table(size: str, batch: int = 64, ctx: int = 4096, chunk: int = 2048) -> list[dict]:
    """Every kernel of a layer, alone: decode (``batch`` rows at ``ctx``) and prefill (one portion of ``chunk`` rows that
    continues at ``ctx``); and the like kernels of the transformer."""
    import torch

    from vllm_metal_b200.lm.decoder import Model
    from vllm_metal_b200.lm.registry import family_of
    from vllm_metal_b200.metal import get_ops

    ops, hbm, tf, _ = get_ops(), *peaks()
    rows = []

    def add(phase, name, us, nbytes=0.0, flops=0.0):
        bound = max(nbytes / (hbm * 1e3), flops / (tf * 1e6))  # us at the measured peaks
        rows.append({"phase": phase, "kernel": name, "us": round(us, 2), "roofline_us": round(bound, 2),
                     "bound": "hbm" if nbytes / (hbm * 1e3) >= flops / (tf * 1e6) else "tensor", "frac": round(bound / us, 3)})

    cfg = config(size, 1)
    family = family_of(cfg)
    args = family.parse(cfg)
    model = family.load(args, None, torch.bfloat16, "cuda")
    like = Model(transformer_args(size, 1), torch.bfloat16, "cuda")
    W, bf = args.width, torch.bfloat16
    lay, m, r = model.layers[0], args.layers[0].mixer, args.layers[0].routed
    ex = lay.experts
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
        xs = [torch.randn((T, W), device="cuda") for _ in range(n_sets(T * W * 4))]
        y, extra = rnd(T, W), rnd(T, W)
        mixed = {"y": y, "norm": lay.norm1b}
        add(phase, "residual step after attention", graph_us([lambda x=x: ops.residual_step(x, mixed, lay.norm2, **step) for x in xs]),
            T * W * (8 + 2 + 2))
        parts = {"y": rnd(T * r.top, W), "part_weight": torch.rand((T, r.top), device="cuda"), "extra": extra,
                 "extra_gate": torch.randn(T, device="cuda"), "norm": lay.norm2b}
        conv = dict(conv=(lay.conv, cache.previous[0]), seg=meta) if decode else {}
        add(phase, "residual step after experts" + (", convolution" if decode else ""),
            graph_us([lambda x=x: ops.residual_step(x, parts, lay.norm1, **conv, **step) for x in xs]),
            T * W * (8 + 2 * r.top + 2 + 2 + (4 * (TAPS - 1) if decode else 0)))
        if not decode:
            hs = [rnd(T, W) for _ in range(n_sets(T * W * 2))]
            add(phase, "convolution", graph_us([lambda h=h: ops.causal_conv(h, lay.conv_and_input, None, cache.previous[0], meta,
                                                                            silu=False) for h in hs]), T * W * 4)
        ids = torch.randint(0, VOCAB, (T,), device="cuda", dtype=torch.int32)
        add(phase, "embedding", graph_us([lambda: ops.embed_rows(ids, model.embed)] * 4), T * W * 6)
        del xs, parts

        # attention
        kin = lay.input.weight.shape[0]
        stacks = [rnd(T, kin) for _ in range(n_sets(T * kin * 2))]
        ps = [lay.input.split(t) for t in stacks]
        qkv = [[p[c].unflatten(1, (hh, dd)) for c, hh, dd in (("q", m.heads, m.dim), ("k", m.kv_heads, m.dim),
                                                              ("v", m.kv_heads, m.vdim))] for p in ps]
        kc, vc = cache.kv[0]
        cols = m.kv_heads * (m.dim + m.vdim)
        add(phase, "attention: rotation, head norms, cache write", graph_us([lambda t=t: ops.rope_norm_cache(
            *t, kc, vc, meta.slot_mapping, meta.positions, lay.mixer.freq, m.rot.amplitude, 1e-5, lay.mixer.temperature)
            for t in qkv]), T * 2 * (2 * m.heads * m.dim + 2 * cols))
        add(phase, "like: norm_rope_cache", graph_us([lambda t=t: ops.norm_rope_cache(
            *t, kc, vc, meta.slot_mapping, positions=meta.positions, rot_dim=m.dim, base=1e4) for t in qkv]),
            T * 2 * (2 * m.heads * m.dim + m.kv_heads * m.dim + 2 * cols))
        out = torch.empty((T, m.heads, m.vdim), dtype=bf, device="cuda")
        caches = [(kc, vc), (kc.clone(), vc.clone())]
        q = qkv[0][0]
        for name, keep, kw in (("attention", m.keep_first, dict(wide_weights=True, plain_softmax=True)),
                               ("attention without kept tokens", 0, dict(wide_weights=True, plain_softmax=True)),
                               ("like: paged attention (16-bit weights)", 0, {})):
            seen = sum(min(m.window + keep, c - a + i + 1) for a, c in zip(q_lens, ctxs) for i in range(a))
            held = sum(min(m.window + a - 1 + keep, c) for a, c in zip(q_lens, ctxs))
            add(phase, name, graph_us([lambda c=c, keep=keep, kw=kw: ops.paged_attention_primitive(
                q, c[0], c[1], m.kv_heads, m.scale, 0.0, meta.block_tables, meta.seq_lens, meta.cu_seqlens_q, 16, max(ctxs),
                m.window, out, min_q_len=meta.min_q_len, keep_first=keep, **kw) for c in caches]),
                held * cols * 2 + T * m.heads * (m.dim + m.vdim) * 2, 2.0 * seen * m.heads * (m.dim + m.vdim))
        del caches, stacks, ps, qkv

        # products
        def product(name, weight, x, wide=False):
            o, k = weight.shape
            ws = [weight] + [weight.clone() for _ in range(n_sets(o * k * 2))]
            kw = {"out_dtype": torch.float32} if wide else {}
            add(phase, f"{name} {o}x{k} (library)", graph_us([lambda w=w: torch.mm(x, w.t(), **kw) for w in ws]),
                2 * (o * k + T * k) + T * o * (4 if wide else 2), 2.0 * T * o * k)

        h = rnd(T, W)
        product("input product", lay.input.weight, h)
        product("output product", lay.output.weight, rnd(T, lay.output.columns))
        product("router product", ex.router.weight, h, wide=True)

        # experts
        heads = ex.router.split(ex.router.wide(h))
        zs = [heads["router"].contiguous() for _ in range(4)]
        add(phase, "experts: routing", graph_us([lambda z=z: ops.expert_route(z, ex.correction, r.experts, r.top, r.scale) for z in zs]),
            T * (r.experts * 4 + r.top * 8))
        chosen, _ = ops.expert_route(zs[0], ex.correction, r.experts, r.top, r.scale)
        tile = ex.tile_rows(T)
        add(phase, "experts: sort", graph_us([lambda: ops.expert_plan(chosen, r.experts, tile)] * 4), T * r.top * 12)
        plan = ops.expert_plan(chosen, r.experts, tile)
        hit = int((plan[1].diff() > 0).sum())
        P = T * r.top
        pairs_flops, shared_flops = 2.0 * P * r.ff * W, 2.0 * T * r.shared_ff * W
        w_bytes, s_bytes = hit * r.ff * W * 2, r.shared_ff * W * 2
        act, s_act = ops.expert_product(h, ex.way_in, plan, r.top, T, gated=True, shared_weight=ex.shared_in)
        add(phase, f"experts: way in ({hit} hit, tiles of {tile})", graph_us([lambda: ops.expert_product(
            h, ex.way_in, plan, r.top, T, gated=True, shared_weight=ex.shared_in)] * 4),
            2 * w_bytes + 2 * s_bytes + T * W * 2 + (P * r.ff + T * r.shared_ff) * 2, 2 * (pairs_flops + shared_flops))
        add(phase, "experts: way out", graph_us([lambda: ops.expert_product(
            act, ex.way_out, plan, r.top, T, gated=False, k=r.ff, shared_x=s_act, shared_weight=ex.shared_out, shared_k=r.shared_ff)] * 4),
            w_bytes + s_bytes + (P * r.ff + T * r.shared_ff + P * W + T * W) * 2, pairs_flops + shared_flops)
        add(phase, "experts: whole block", graph_us([lambda: ex(h)] * 4),
            3 * (w_bytes + s_bytes) + 2 * T * W * 2, 3 * (pairs_flops + shared_flops))
        blk = like.layers[0].mlp.block
        for _ in range(3):
            blk(h)
        add(phase, "like: int4 expert block (eager)", _events(lambda: blk(h), 5) * 1e3,
            3 * hit * (r.ff * W // 2 + r.ff * W // 16) + 2 * T * W * 2, 3 * pairs_flops)
        x2, w2 = rnd(T, W), torch.ones(W, dtype=bf, device="cuda")
        ress = [rnd(T, W) for _ in range(n_sets(T * W * 2))]
        add(phase, "like: rms_norm + residual", graph_us([lambda y=y: ops.rms_norm(x2, w2, 1e-5, residual=y) for y in ress]), T * W * 8)
        del cache, act, s_act, ress
    assert not ops.expert_product_failed()
    return rows


def whole_model(size: str, kind: str, batch: int, ctx: int, chunk: int, steps: int, warmup: int) -> dict:
    import torch

    from vllm_metal_b200.metal import get_ops
    from vllm_metal_b200.v1.model_runner import PagedModelRunner

    bf = torch.bfloat16
    per = -(-(ctx + 2 * (steps + warmup) + chunk) // 16) + 1
    blocks = 1 + per * batch
    s = SIZES[size]
    if kind == "sandwich":
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
            t.numel() for x in model.layers for t in (x.input.weight, x.output.weight, x.experts.way_in, x.experts.way_out,
                                                      x.experts.shared_in, x.experts.shared_out, x.experts.router.weight))
        bits = 16
    else:
        from vllm_metal_b200.attention.caches.kv_cache import B200PagedKVCache
        from vllm_metal_b200.lm.decoder import Model

        args = transformer_args(size)
        model = Model(args, bf, "cuda")
        cache = B200PagedKVCache(args.num_layers, args.n_kv_heads, args.head_dim, blocks, 16, bf, "cuda",
                                 sliding_window_per_layer=args.sliding_window_per_layer())
        for t in (*cache.key_caches, *cache.value_caches):
            t.normal_()
        weights = args.num_layers * (args.hidden * (2 * args.n_heads + 2 * args.n_kv_heads) * args.head_dim +
                                     3 * s["experts"] * args.hidden * args.intermediate) + args.vocab * args.hidden
        bits = args.bits
    runner = PagedModelRunner(model, cache, max_batch=batch, max_model_len=per * 16)
    tables = [list(range(1 + i * per, 1 + (i + 1) * per)) for i in range(batch)]
    slots = {"state_slots": list(range(1, batch + 1))} if runner.stateful else {}
    runner.fill_decode([1 + 7 * i for i in range(batch)], tables, [ctx] * batch, *slots.values())
    runner.buf.upload()
    limit = ctx + 2 * (steps + warmup) + 1
    ops = get_ops()
    for _ in range(warmup):
        runner.run_decode(batch, limit, advance=True)
    n0 = ops.launches
    ms = _events(lambda: runner.run_decode(batch, limit, advance=True), steps)
    launches = next(iter(runner.launches_per_graph.values()), (ops.launches - n0) // steps)
    out = {"model": kind, "weights": weights, "weight_bits": bits, "decode_ms": round(ms, 3),
           "decode_tok_s": round(batch * 1e3 / ms, 1), "decode_launches": launches, "cuda_graph": runner.use_cuda_graph}
    one = {"state_slots": [1]} if runner.stateful else {}
    tokens = [(17 * i + 3) % VOCAB for i in range(chunk)]
    for offset in (0, ctx):
        def run(offset=offset):
            runner.execute(tokens, [], [(tables[0], chunk, offset)], **one)

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
    result = {"metric": "sandwich-norm decoder prefill / decode tok/s", "unit": "tok/s", "data": "synthetic", "dtype": "bf16",
              "n_gpus": 1, "steps": steps, "warmup": warmup, "peaks": {"hbm_gbs": hbm, "bf16_tflops": tf, "source": source},
              "config": {"batch": batch, "ctx": ctx, "chunk": chunk, "layers": LAYERS, "taps": TAPS, "vocab": VOCAB,
                         "l2_policy": "operand sets larger than L2 (kernels); weights and caches larger than L2 (models)"},
              "sizes": {}}
    for size in sizes:
        entry = {"shape": SIZES[size], "models": []}
        for kind in ("sandwich", "transformer"):
            entry["models"].append(whole_model(size, kind, batch, ctx, chunk, steps, warmup))
            torch.cuda.empty_cache()
        if kernels:
            entry["kernels"] = kernel_table(size, batch, ctx, chunk)
            torch.cuda.empty_cache()
        result["sizes"][size] = entry
    return result


if __name__ == "__main__":
    print(show(main(tuple(sys.argv[1].split(",")) if len(sys.argv) > 1 else tuple(SIZES))))
