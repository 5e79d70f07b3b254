#!/usr/bin/env python
"""Pre-norm decoders with time mixing next to the closest model of the framework, the hyper-connected decoder with one stream
(lightning attention, softmax attention beside it): whole-model prefill and decode throughput, and every kernel against its
roofline beside the like kernel at the same size.

    python bench.py --prenorm [--prenorm-sizes s,m,w]      (or this file directly)

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
from profiles.bench_streams import show  # noqa: E402

SIZES = {
    "s": dict(width=2048, groups=4, wkv=(32, 64), heads=32, kv_heads=8, dim=64, vdim=64, window=1024, ff=8192, experts=32, top=4, eff=2048),
    "m": dict(width=4096, groups=8, wkv=(64, 64), heads=32, kv_heads=8, dim=128, vdim=128, window=4096, ff=16384, experts=64, top=8,
              eff=1536),
    "w": dict(width=2560, groups=1, wkv=(20, 128), heads=20, kv_heads=4, dim=96, vdim=128, window=512, ff=8960, experts=16, top=2, eff=2560),
}
PATTERN = (("wkv", "dense"), ("wkv", "moe"), ("attention", "dense"), ("wkv", "moe"))
KINDS = ("prenorm", "prenorm, dense", "streams")


def config(size: str, pattern=PATTERN) -> dict:
    s = SIZES[size]
    mixers = {"wkv": {"heads": s["wkv"][0], "dim": s["wkv"][1]},
              "attention": {**{n: s[n] for n in ("heads", "kv_heads", "dim", "vdim")}, "scale": s["dim"] ** -0.5,
                            "mask": {"size": s["window"]}, "q_temp": {"coef": 0.1, "every": 8192}}}
    mlps = {"dense": {"kind": "dense", "ff": s["ff"]},
            "moe": {"kind": "moe", "expert": {"ff": s["eff"]}, "router": {"experts": s["experts"], "top": s["top"]}}}
    return {"architecture": "Retuvik", "vocab": VOCAB, "width": s["width"], "embedding": {"scale": 4.0},
            "norm": {"eps": 1e-5, "groups": s["groups"]},
            "layers": [{"type": t, "mixer": mixers[t], "mlp": mlps[f]} for t, f in pattern]}


def like_config(size: str, pattern=PATTERN) -> dict:
    """One stream; recurrence heads of the same sizes; a gated feed-forward with the weights of the dense one."""
    s = SIZES[size]
    (h, d), ff = s["wkv"], 2 * s["ff"] // 3 // 64 * 64
    lightning = {"heads": h, "dim": d, "vdim": d, "decay": [1.0 - 2.0 ** -(2 + 8 * i / h) for i in range(h)]}
    mixers = {"wkv": ("lightning", lightning),
              "attention": ("parallel", {"left": {**{n: s[n] for n in ("heads", "kv_heads", "dim", "vdim")}, "scale": s["dim"] ** -0.5},
                                         "right": lightning})}
    layers = [{"type": mixers[t][0], "mixer": mixers[t][1], "mlp": {"kind": "dense", "ff": ff}} for t, _ in pattern]
    return {"architecture": "Tatazen", "vocab": VOCAB, "width": s["width"], "streams": 1, "norm": {"eps": 1e-5}, "layers": layers}


def kernel_table(size: str, batch: int = 64, ctx: int = 4096, chunk: int = 2048) -> list[dict]:
    """Every kernel of a layer of each kind, alone: decode (``batch`` rows at ``ctx``) and prefill (one portion of ``chunk``
    rows that continues at ``ctx``); and the like kernels of the framework's other models."""
    import torch

    from vllm_metal_b200.lm.registry import family_of
    from vllm_metal_b200.metal import get_ops

    ops, hbm, tf, _ = get_ops(), *peaks()
    rows = []

    def add(phase, name, us, nbytes=0.0, flops=0.0):
        bound = max(nbytes / (hbm * 1e3), flops / (tf * 1e6))  # us at the measured peaks
        rows.append({"phase": phase, "kernel": name, "us": round(us, 2), "roofline_us": round(bound, 2),
                     "bound": "hbm" if nbytes / (hbm * 1e3) >= flops / (tf * 1e6) else "tensor", "frac": round(bound / us, 3)})

    cfg = config(size, (("wkv", "dense"), ("attention", "moe")))
    family = family_of(cfg)
    args = family.parse(cfg)
    model = family.load(args, None, torch.bfloat16, "cuda")
    W, bf = args.width, torch.bfloat16
    mixing, attending = model.layers
    m, a, r = args.layers[0].mixer, args.layers[1].mixer, args.layers[1].routed
    mix, att, ex, dense = mixing.mixer, attending.mixer, attending.feed, mixing.feed
    mu, inner, ff = mix.mix_weight, m.inner, args.layers[0].ff
    rnd = lambda *s: torch.randn(s, device="cuda").to(bf)  # noqa: E731
    n_sets = lambda nbytes: max(2, min(24, -(-L2_BYTES // nbytes)))  # noqa: E731
    ones = torch.ones(W, device="cuda")
    for phase, q_lens, ctxs in (("decode", [1] * batch, [ctx] * batch), ("prefill", [chunk], [ctx + chunk])):
        meta, blocks = _segments(q_lens, ctxs)
        T, n = sum(q_lens), len(q_lens)
        cache = family.make_cache(args, blocks, 16, n, bf, "cuda")
        for t in cache.kv[1]:
            t.normal_()
        decode = phase == "decode"
        state, last = cache.states[0].matrix, cache.states[0].last

        # between the sublayers
        step = dict(eps=1e-5, dtype=bf, groups=args.norm_groups)
        xs = [torch.randn((T, W), device="cuda") for _ in range(n_sets(T * W * 4))]
        y = rnd(T, W)
        plain, biased = {"y": y}, {"y": y, "bias": dense.down_bias}
        routed = {"y": rnd(T * r.top, W), "part_weight": torch.rand((T, r.top), device="cuda")}
        ids = torch.randint(0, VOCAB, (T,), device="cuda", dtype=torch.int32)
        again = dict(embed=(ids, model.embed, 4.0, False), add=ones)
        into = dict(mix=(mu, last), seg=meta) if decode else dict(wide=True)
        what, out_bytes = (", mixes", 10 + 8) if decode else (", 32-bit input", 4)
        add(phase, "step after a mixer", graph_us([lambda x=x: ops.residual_step(x, plain, mixing.norm2, **step) for x in xs]), T * W * 12)
        for name, result, more, nbytes in (("dense feed-forward", biased, {}, 2), ("experts", routed, {}, 2 * r.top),
                                           ("experts, start of a pass", routed, again, 2 * r.top + 2)):
            add(phase, f"step after {name}{what}", graph_us([lambda x=x, res=result, kw=more: ops.residual_step(
                x, res, mixing.norm1, **into, **kw, **step) for x in xs]), T * W * (8 + nbytes + out_bytes))
        between = {"eps": 1e-5, "dtype": bf}
        normed = [dict(p, norm=ones) for p in (plain, routed)]
        for name, result, nbytes in (("like: step between norms", normed[0], 2), ("like: step between norms after experts", normed[1], 2 * r.top)):
            add(phase, name, graph_us([lambda x=x, res=result: ops.residual_step(x, res, ones, **between) for x in xs]),
                T * W * (10 + nbytes))
        if not decode:
            add(phase, "token mixes", graph_us([lambda x=x: ops.token_mix(x, mu, last, meta, bf) for x in xs]), T * W * 14)
            taps, kept = torch.rand((2, W), device="cuda"), torch.zeros((n + 1, 1, W), dtype=bf, device="cuda")
            hs = [rnd(T, W) for _ in range(n_sets(T * W * 2))]
            add(phase, "like: token shift", graph_us([lambda h=h: ops.causal_conv(h, taps, None, kept, meta, silu=False) for h in hs]),
                T * W * 4)
            del hs
        del xs, routed, normed

        # products
        def product(name, weight, x, wide=False, count=1, bias=None):
            o, k = weight.shape[-2:]
            ws = [weight] + [weight.clone() for _ in range(n_sets(count * o * k * 2))]
            kw = {"out_dtype": torch.float32} if wide else {}
            if count > 1:
                calls = [lambda w=w: torch.bmm(x, w.transpose(1, 2)) for w in ws]
            elif bias is not None:
                calls = [lambda w=w: torch.addmm(bias, x, w.t()) for w in ws]
            else:
                calls = [lambda w=w: torch.mm(x, w.t(), **kw) for w in ws]
            add(phase, f"{name} {f'{count} x ' if count > 1 else ''}{o}x{k} (library)", graph_us(calls),
                count * (2 * (o * k + T * k) + T * o * (4 if wide else 2)), 2.0 * count * T * o * k)

        h = rnd(T, W)
        product("time mixing: products", mix.products.weight, rnd(4, T, W), count=4)
        product("time mixing: decay, down", mix.decay_down.weight, h)
        product("time mixing: decay, up", mix.decay_up.weight, rnd(T, mix.decay_up.columns), wide=True)
        product("time mixing: output product", mixing.output.weight, rnd(T, mixing.output.columns))
        product("attention: input product", attending.input.weight, h)
        product("attention: output product", attending.output.weight, rnd(T, attending.output.columns))
        product("feed-forward: way in", dense.up.weight, h, bias=dense.up.bias)
        product("feed-forward: way out", dense.down.weight, rnd(T, dense.down.columns))
        product("router product", ex.router.weight, h, wide=True)

        # time mixing
        parts = [{**dict(zip("rkvg", rnd(4, T, inner))), "w": torch.randn((T, inner), device="cuda") - 3.0}
                 for _ in range(n_sets(T * inner * 12))]
        both = 2 * n * m.heads * m.dim * m.dim * 4
        add(phase, "time mixing: recurrence", graph_us([lambda p=p: ops.recurrence(
            "wkv", p["r"], p["k"], p["v"], p["w"], None, meta, state, heads=m.heads, groups=m.heads, key_dim=m.dim, value_dim=m.dim,
            bias_a=mix.decay_bias, skip=mix.bonus) for p in parts]), both + T * inner * 12)
        rate = torch.linspace(1e-3, 0.3, m.heads, device="cuda")
        decay = torch.exp(-rate)
        add(phase, "like: lightning recurrence", graph_us([lambda p=p: ops.recurrence(
            "lightning", p["r"], p["k"], p["v"], None, None, meta, state, heads=m.heads, groups=m.heads, key_dim=m.dim, value_dim=m.dim,
            rate=rate, decay=decay) for p in parts]), both + T * inner * 8)
        gates = torch.randn((T, m.heads), device="cuda").to(bf)
        zero, one = torch.zeros(m.heads, device="cuda"), torch.ones(m.heads, device="cuda")
        add(phase, "like: Mamba-2 recurrence", graph_us([lambda p=p: ops.recurrence(
            "ssd", p["r"], p["k"], p["v"], gates, None, meta, state, heads=m.heads, groups=m.heads, key_dim=m.dim, value_dim=m.dim,
            bias_a=zero, rate=one, skip=one) for p in parts]), both + T * inner * 8)
        y = mixing.output.operand(T)
        add(phase, "time mixing: head norm, gate", graph_us([lambda p=p: ops.mixer_finish(
            y, inner, y=p["r"], post_gate=p["g"], weight=mix.norm, group_size=m.dim, eps=1e-5, post="silu") for p in parts]), T * inner * 6)
        add(phase, "like: norm of all heads, gate", graph_us([lambda p=p: ops.mixer_finish(
            y, inner, y=p["r"], post_gate=p["g"], weight=mix.norm, group_size=inner, eps=1e-5) for p in parts]), T * inner * 6)
        z, low = mix.decay_up.operand(T), rnd(T, mix.decay_down.weight.shape[0])
        add(phase, "time mixing: decay, tanh", graph_us([lambda: ops.mixer_finish(z, 0, low, act="tanh")] * 4), low.numel() * 4)
        del parts

        # feed-forward
        ups = [rnd(T, ff) for _ in range(n_sets(T * ff * 2))]
        y = dense.down.operand(T)
        add(phase, "feed-forward: xIELU", graph_us([lambda u=u: ops.mixer_finish(y, 0, u, act="xielu", act_weights=dense.act) for u in ups]),
            T * ff * 4)
        add(phase, "like: gelu", graph_us([lambda u=u: ops.mixer_finish(y, 0, u) for u in ups]), T * ff * 4)
        del ups

        # attention
        kin = attending.input.weight.shape[0]
        stacks = [rnd(T, kin) for _ in range(n_sets(T * kin * 2))]
        ps = [attending.input.split(t) for t in stacks]
        qkv = [[p[c].unflatten(1, (hh, dd)) for c, hh, dd in (("q", a.heads, a.dim), ("k", a.kv_heads, a.dim),
                                                              ("v", a.kv_heads, a.vdim))] for p in ps]
        kc, vc = cache.kv[1]
        cols = a.kv_heads * (a.dim + a.vdim)
        norms = dict(q_norm=att.q_norm, k_norm=att.k_norm, norm_values=True, temperature=(a.temp_coef, a.temp_every))
        freq = torch.rand((a.dim // 2, 2), device="cuda")
        for name, f, kw in (("attention: head norms, temperature, cache write", None, norms), ("like: rotation, head norms, cache write", freq, {})):
            add(phase, name, graph_us([lambda t=t, f=f, kw=kw: ops.rope_norm_cache(
                *t, kc, vc, meta.slot_mapping, meta.positions, f, 1.0, 1e-5, **kw) for t in qkv]), T * 2 * (2 * a.heads * a.dim + 2 * cols))
        out = torch.empty((T, a.heads, a.vdim), dtype=bf, device="cuda")
        caches = [(kc, vc), (kc.clone(), vc.clone())]
        q = qkv[0][0]
        seen = sum(min(a.window, c - b + i + 1) for b, c in zip(q_lens, ctxs) for i in range(b))
        held = sum(min(a.window + b - 1, c) for b, c in zip(q_lens, ctxs))
        for name, slopes in (("attention", att.slopes), ("like: attention without a distance bias", None)):
            add(phase, name, graph_us([lambda c=c, sl=slopes: ops.paged_attention_primitive(
                q, c[0], c[1], a.kv_heads, a.scale, 0.0, meta.block_tables, meta.seq_lens, meta.cu_seqlens_q, 16, max(ctxs), a.window, out,
                wide_weights=True, plain_softmax=True, min_q_len=meta.min_q_len, slopes=sl) for c in caches]),
                held * cols * 2 + T * a.heads * (a.dim + a.vdim) * 2, 2.0 * seen * a.heads * (a.dim + a.vdim))
        ys = [rnd(T, attending.output.columns) for _ in ps]
        ai = a.heads * a.vdim
        add(phase, "attention: gate", graph_us([lambda p=p, y=y: ops.mixer_finish(y, ai, y=y[:, :ai], post_gate=p["g"])
                                                for p, y in zip(ps, ys)]), T * ai * 6)
        del caches, stacks, ps, qkv, ys

        # experts
        logits = ex.router.split(ex.router.wide(h))["router"]
        for name, over in (("experts: routing over the chosen", True), ("like: routing over all", False)):
            add(phase, name, graph_us([lambda o=over: ops.expert_route(logits, ex.correction, r.experts, r.top, 1.0, o)] * 4),
                T * (r.experts * 4 + r.top * 8))
        chosen, _ = ops.expert_route(logits, ex.correction, r.experts, r.top, 1.0, True)
        tile = ex.tile_rows(T)
        add(phase, "experts: sort", graph_us([lambda: ops.expert_plan(chosen, r.experts, tile)] * 4), T * r.top * 12)
        plan = ops.expert_plan(chosen, r.experts, tile)
        hit = int((plan[1].diff() > 0).sum())
        P = T * r.top
        flops, w_bytes = 2.0 * P * r.ff * W, hit * r.ff * W * 2
        act, _ = ops.expert_product(h, ex.way_in, plan, r.top, T, gated=True)
        add(phase, f"experts: way in ({hit} hit, tiles of {tile})", graph_us([lambda: ops.expert_product(
            h, ex.way_in, plan, r.top, T, gated=True)] * 4), 2 * w_bytes + T * W * 2 + P * r.ff * 2, 2 * flops)
        add(phase, "experts: way out", graph_us([lambda: ops.expert_product(act, ex.way_out, plan, r.top, T, gated=False, k=r.ff)] * 4),
            w_bytes + (P * r.ff + P * W) * 2, flops)
        del cache, act
    assert not ops.expert_product_failed() and not ops.recurrence_failed()
    return rows


def weight_count(layer) -> int:
    lin = [getattr(layer, n, None) for n in ("input", "gate", "up", "down", "output")]
    lin += [b.output for b in getattr(layer, "branches", ())]
    mixer, feed = getattr(layer, "mixer", None), getattr(layer, "feed", None)
    lin += [getattr(mixer, n, None) for n in ("products", "decay_down", "decay_up")]
    lin += [getattr(feed, n, None) for n in ("up", "down", "router")]
    total = sum(x.weight.numel() for x in lin if x is not None)
    return total + sum(getattr(feed, n).numel() for n in ("way_in", "way_out") if hasattr(feed, n))


def whole_model(size: str, kind: str, batch: int, ctx: int, chunk: int, steps: int, warmup: int) -> dict:
    import torch

    from vllm_metal_b200.lm.registry import family_of
    from vllm_metal_b200.v1.model_runner import PagedModelRunner

    bf = torch.bfloat16
    per = -(-(ctx + 2 * (steps + warmup) + chunk) // 16) + 1
    blocks = 1 + per * batch
    cfg = {"prenorm": config, "streams": like_config}[kind.split(",")[0]](
        size, PATTERN if kind == "prenorm" else tuple((t, "dense") for t, _ in PATTERN))
    fam = family_of(cfg)
    args = fam.parse(cfg)
    model = fam.load(args, None, bf, "cuda")
    cache = fam.make_cache(args, blocks, 16, batch, bf, "cuda")
    for kv in cache.kv.values():
        for t in kv:
            t.normal_()
    runner = PagedModelRunner(model, cache, max_batch=batch, max_model_len=per * 16)
    tables = [list(range(1 + i * per, 1 + (i + 1) * per)) for i in range(batch)]
    runner.fill_decode([1 + 7 * i for i in range(batch)], tables, [ctx] * batch, list(range(1, batch + 1)))
    runner.buf.upload()
    limit = ctx + 2 * (steps + warmup) + 1
    for _ in range(warmup):
        runner.run_decode(batch, limit, advance=True)
    ms = _events(lambda: runner.run_decode(batch, limit, advance=True), steps)
    out = {"model": kind, "weights": model.head.weight.numel() + sum(weight_count(x) for x in model.layers), "weight_bits": 16,
           "decode_ms": round(ms, 3), "decode_tok_s": round(batch * 1e3 / ms, 1),
           "decode_launches": next(iter(runner.launches_per_graph.values()))}
    tokens = [(17 * i + 3) % VOCAB for i in range(chunk)]
    for offset in (0, ctx):
        def run(offset=offset):
            runner.execute(tokens, [], [(tables[0], chunk, offset)], state_slots=[1])

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
    result = {"metric": "pre-norm time-mixing decoder prefill / decode tok/s", "unit": "tok/s", "data": "synthetic", "dtype": "bf16",
              "n_gpus": 1, "steps": steps, "warmup": warmup, "peaks": {"hbm_gbs": hbm, "bf16_tflops": tf, "source": source},
              "config": {"batch": batch, "ctx": ctx, "chunk": chunk, "layers": len(PATTERN), "vocab": VOCAB,
                         "l2_policy": "operand sets larger than L2 (kernels); weights and caches larger than L2 (models)"},
              "sizes": {}}
    for size in sizes:
        entry = {"shape": SIZES[size], "models": []}
        for kind in KINDS:
            entry["models"].append(whole_model(size, kind, batch, ctx, chunk, steps, warmup))
            torch.cuda.empty_cache()
        if kernels:
            entry["kernels"] = kernel_table(size, batch, ctx, chunk)
            torch.cuda.empty_cache()
        result["sizes"][size] = entry
    return result


if __name__ == "__main__":
    print(show(main(tuple(sys.argv[1].split(",")) if len(sys.argv) > 1 else tuple(SIZES))))
