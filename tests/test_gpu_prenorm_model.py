"""Pre-norm decoders with time mixing on the device, whole: the model through the engine's step against the
whole-sequence oracle -- portions, batches, reused pages and slots, windows, loops, long decoding, generation."""

from __future__ import annotations

import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

from oracle import retuvik as oracle

from .hybrid_helpers import Harness, make_engine, random_checkpoint, rounded_products, to_oracle, write_folder
from .prenorm_helpers import attention_layer, clear_routing, default_prenorm_config, experts, prenorm_config, wkv_layer

pytestmark = pytest.mark.gpu

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
BOTH = pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])


def harness(config, dtype, scale=None, **kw):
    def edit(tensors):
        clear_routing(config)(tensors)
        if scale is not None:
            scale(tensors)

    return Harness(config, dtype, oracle=oracle, scale=edit, **kw)


def checkpoint(config, seed=0):
    tensors = random_checkpoint(config, seed)
    clear_routing(config)(tensors)
    return tensors


def configs():
    odd = [wkv_layer({"kind": "dense", "ff": 19}, heads=3, dim=11), attention_layer(experts(ff=33, n=3, top=3), heads=3, kv_heads=3, dim=11,
                                                                               vdim=5, mask={"size": 7}, q_temp={"coef": -0.1, "every": 1}),
           wkv_layer(experts(ff=9, n=5, top=2), heads=1, dim=7)]
    wide = [attention_layer(experts(ff=176, n=9, top=4), heads=4, kv_heads=1, dim=136, vdim=200, scale=0.1, mask={"size": 130},
                            q_temp={"coef": 0.3, "every": 64}),
            wkv_layer({"kind": "dense", "ff": 200}, heads=4, dim=64), wkv_layer(experts(ff=72, n=16, top=8), heads=2, dim=136),
            attention_layer(None, heads=18, kv_heads=1, dim=16, vdim=16, mask={"size": 128}),
            attention_layer({"kind": "dense", "ff": 96}, heads=8, kv_heads=4, dim=64, vdim=128, mask={"size": 64})]
    ones = [wkv_layer({"kind": "dense", "ff": 1}, heads=1, dim=1), attention_layer(experts(ff=1, n=1, top=1), heads=1, kv_heads=1, dim=8, vdim=8,
                                                                               scale=1.0, mask={"size": 1}),
            wkv_layer(experts(ff=8, n=2, top=1), heads=1, dim=8), attention_layer({"kind": "dense", "ff": 8}, heads=1, kv_heads=1, dim=8, vdim=8,
                                                                                  mask={"size": 2}, q_temp=None)]
    return {"default": default_prenorm_config(),
            "odd": prenorm_config(odd, (0, 2, 2), groups=1, vocab=61, width=37, eps=1e-3, scale=1.0),
            "wide": prenorm_config(wide, (1, 4, 2), groups=5, vocab=130, width=160, scale=12.0),
            "ones": prenorm_config(ones, (3, 4, 1), groups=2, vocab=33, width=24),
            "time_mixing_only": prenorm_config([wkv_layer(), wkv_layer(None)], (1, 2, 4), groups=2, width=96, eps=1e-5),
            "attention_only": prenorm_config([attention_layer(None), attention_layer()], groups=3, width=96, eps=1e-5)}


@BOTH
@pytest.mark.parametrize("name", list(configs()))
def test_prompts_portions_and_decoding_agree_with_the_oracle(name, dtype):
    h = harness(configs()[name], dtype)
    for i, portions in enumerate(([400], [150, 1, 1, 2], [64], [16, 3], [2], [1, 7, 90])):
        h.request(str(i), 230 if i < 2 else 70, seed=i)
        h.drain(str(i), portions)
    h.request("one", 1)
    h.drain("one", [1])
    from vllm_metal_b200.metal import get_ops

    assert not get_ops().expert_product_failed() and not get_ops().recurrence_failed()


def test_random_routing_in_32_bits():
    h = Harness(default_prenorm_config(), torch.float32, seed=5, oracle=oracle)
    h.request("a", 150)
    h.drain("a", [70, 1, 1, 30])


@BOTH
def test_token_by_token_from_the_first_token(dtype):
    h = harness(default_prenorm_config(), dtype)
    h.request("a", 90)
    h.drain("a", [1])


@BOTH
def test_batches_of_unequal_requests_with_reused_pages_and_slots(dtype):
    """Four slots and pages for little more than four requests; eleven requests come and go, each in its own rhythm."""
    h = harness(default_prenorm_config(), dtype, max_tokens=640, max_num_seqs=4)
    rng = np.random.default_rng(5)
    lengths = [150, 33, 97, 5, 160, 16, 2, 120, 64, 1, 75]
    for i, n in enumerate(lengths):
        h.request(str(i), n, seed=i)
    waiting, live = [str(i) for i in range(len(lengths))], []
    while waiting or live:
        while waiting and len(live) < 4:
            live.append(waiting.pop(0))
        chosen = [r for r in live if rng.random() < 0.8] or live[:1]
        h.step({r: int(rng.choice([1, 1, 2, 5, 17, 40, 64])) for r in chosen})
        live = [r for r in live if h.at[r] < len(h.tokens[r])]
    assert h.engine.pool.num_free == h.engine.pool.num_blocks and h.engine.slots.num_free == 4


@BOTH
def test_a_request_alone_and_in_a_batch(dtype):
    cfg = default_prenorm_config()
    tensors = checkpoint(cfg)
    from vllm_metal_b200.v1.engine import StepEntry

    rng = np.random.default_rng(0)
    toks = [rng.integers(0, cfg["vocab"], n).tolist() for n in (90, 41, 7)]
    alone = make_engine(cfg, tensors, dtype)
    first = [alone.advance([StepEntry(str(i), t, [len(t) - 1])]).clone() for i, t in enumerate(toks)]
    second = [alone.advance([StepEntry(str(i), [3], [0])]).clone() for i in range(3)]
    together = make_engine(cfg, tensors, dtype)
    a = together.advance([StepEntry(str(i), t, [len(t) - 1]) for i, t in enumerate(toks)])
    tol = 2e-5 if dtype == torch.float32 else 4e-2
    torch.testing.assert_close(a, torch.cat(first), atol=tol * float(a.abs().max()), rtol=0)
    b = together.advance([StepEntry(str(i), [3], [0]) for i in (2, 0, 1)])
    torch.testing.assert_close(b, torch.cat([second[i] for i in (2, 0, 1)]), atol=tol * float(b.abs().max()), rtol=0)


@BOTH
def test_long_decoding_past_windows_pages_and_graph_buckets(dtype):
    cfg = prenorm_config([wkv_layer(None), attention_layer(experts(ff=24, n=5, top=2), mask={"size": 150}, q_temp={"coef": 0.4, "every": 64})],
                         (0, 1, 2))
    h = harness(cfg, dtype)
    h.request("long", 620, seed=2)
    h.drain("long", [300] + [1] * 400)


@BOTH
@pytest.mark.parametrize("at", [0, 3, 15, 16, 100, 128])
def test_one_outstanding_key_counts_as_long_as_it_is_visible(dtype, at):
    """The weights are made so that every query asks for token 7's key: the logits of exactly those positions depend on it
    that see it, those inside the window."""
    size = 37
    cfg = prenorm_config([attention_layer(None, heads=4, kv_heads=2, dim=32, vdim=24, scale=0.6, mask={"size": size})], groups=1)

    def shape(t):
        t["embed"][:, 0], t["embed"][:, 1] = 0.0, 6.0
        t["embed"][7, 0] = 9.0
        t["l0.norm1"][:] = 1.0
        t["l0.mix.q.norm"][:] = t["l0.mix.k.norm"][:] = 1.0
        q, k = t["l0.mix.q"].view(4, 32, -1), t["l0.mix.k"].view(2, 32, -1)
        q.zero_()
        k.zero_()
        q[:, 20, 1] = 1.0                    # every query points along one dimension
        k[:, 20, 0], k[:, 21, 1] = 1.0, 1.0  # keys too where the token is 7, along another elsewhere

    h = harness(cfg, dtype, scale=shape)
    n = 240
    h.request("a", n)
    toks = [t if t != 7 else 8 for t in h.tokens["a"]]
    plain = oracle.forward(cfg, h.oracle_tensors, toks)
    toks[at] = 7
    h.tokens["a"], h.want["a"] = toks, oracle.forward(cfg, h.oracle_tensors, toks)
    h.limit["a"][:] = 4e-5 if dtype == torch.float32 else 4e-2
    moved = np.sqrt(((plain - h.want["a"]) ** 2).mean(1)) / h.want["a"].std()
    last = at + size
    assert (moved[at:last] > 0.1).all() and (moved[:at] == 0).all() and (moved[last:] == 0).all(), (moved[at:last].min())
    for req_id, portions in (("a", [n]), ("b", [at + 20] + [1] * n), ("c", [2, 31]), ("d", [at + size - 1, 2, 1, 16])):
        h.tokens[req_id], h.want[req_id], h.limit[req_id], h.at[req_id] = toks, h.want["a"], h.limit["a"], 0
        h.drain(req_id, portions)


@BOTH
def test_a_far_token_lives_on_in_the_state(dtype):
    """Weights that never let the state decay and write to it for token 7 alone: it shows hundreds of tokens later, however the
    sequence was cut, and not in a request that takes the slot afterwards."""
    cfg = prenorm_config([wkv_layer(None, heads=2, dim=24)], groups=1)

    def shape(t):
        t["embed"][:, 0], t["embed"][:, 1] = 0.0, 6.0
        t["embed"][7, 0] = 9.0
        t["l0.norm1"][:] = 1.0
        for s in "rkvgw":
            t[f"l0.mix.mu.{s}"][:] = 0.0
        t["l0.mix.k"].zero_()
        t["l0.mix.k"][:, 0] = 1.0
        t["l0.mix.r"].zero_()
        t["l0.mix.r"][:, 1] = 1.0  # every row reads all of it: no head's output nearly vanishes before its norm
        t["l0.mix.w0"][:] = -20.0
        t["l0.mix.w2"].zero_()

    h = harness(cfg, dtype, scale=shape, max_num_seqs=1)
    n, at = 420, 3
    h.request("a", n)
    toks = [t if t != 7 else 8 for t in h.tokens["a"]]
    plain = oracle.forward(cfg, h.oracle_tensors, toks)
    toks[at] = 7
    want = oracle.forward(cfg, h.oracle_tensors, toks)
    moved = np.sqrt(((plain - want) ** 2).mean(1)) / want.std()
    assert (moved[at:] > 0.1).all() and (moved[:at] == 0).all()
    limit = np.full(n, 4e-5 if dtype == torch.float32 else 4e-2)
    for req_id, portions in (("a", [n]), ("b", [40] + [1] * 200 + [n]), ("c", [2, 31]), ("d", [4, 64, 1])):
        h.tokens[req_id], h.want[req_id], h.limit[req_id], h.at[req_id] = toks, want, limit, 0
        h.drain(req_id, portions)
    h.tokens["e"], h.want["e"], h.limit["e"], h.at["e"] = [8] + toks[4:], oracle.forward(cfg, h.oracle_tensors, [8] + toks[4:]), limit, 0
    h.drain("e", [1, 5, 100])


@BOTH
def test_residual_stream_after_every_layer(dtype):
    from vllm_metal_b200.v1.engine import StepEntry

    cfg = default_prenorm_config()
    tensors = checkpoint(cfg)
    e = make_engine(cfg, tensors, dtype)
    got, want, toks = [], [], list(range(40))
    e.model.residual_hook = lambda i, x: got.append(x.double().cpu().numpy())
    e.advance([StepEntry("a", toks)])
    oracle.forward(cfg, to_oracle(tensors), toks, want)
    rounded = []
    with rounded_products(oracle):
        oracle.forward(cfg, to_oracle(tensors), toks, rounded)
    assert len(got) == len(want) == 11
    error = lambda a, b: np.sqrt(((a - b) ** 2).mean(1)) / b.std()  # noqa: E731
    for i, (a, b, r) in enumerate(zip(got, want, rounded)):
        limit = 2e-5 if dtype == torch.float32 else 1.5e-2 + 3 * error(r, b)
        over = error(a, b) / limit
        assert over.max() <= (1 if dtype == torch.float32 else 4) and (over > 1).mean() <= 0.2, (i, over.max())


def test_a_step_that_wants_nothing_still_moves_the_state():
    from vllm_metal_b200.v1.engine import StepEntry

    cfg = default_prenorm_config()
    tensors = checkpoint(cfg)
    toks = np.random.default_rng(3).integers(0, cfg["vocab"], 50).tolist()
    e = make_engine(cfg, tensors, torch.float32)
    for lo, hi in ((0, 20), (20, 21), (21, 49)):
        assert e.advance([StepEntry("a", toks[lo:hi])]).shape == (0, cfg["vocab"])
    got = e.advance([StepEntry("a", toks[49:], [0])]).double().cpu().numpy()
    np.testing.assert_allclose(got[0], oracle.forward(cfg, to_oracle(tensors), toks)[-1], atol=1e-3)


# -- the framework's entry points --------------------------------------------------------------------------------

def greedy(cfg, tensors, prompt, n):
    toks, t = list(prompt), to_oracle(tensors)
    for _ in range(n):
        toks.append(int(oracle.forward(cfg, t, toks)[-1].argmax()))
    return toks[len(prompt):]


def test_greedy_generation_through_scheduler_and_command_line(tmp_path):
    from vllm_metal_b200.v1.engine import Engine

    cfg = default_prenorm_config()
    tensors = random_checkpoint(cfg, seed=3)
    folder = write_folder(tmp_path / "model", cfg, tensors)
    rng = np.random.default_rng(1)
    prompts = [rng.integers(0, cfg["vocab"], n).tolist() for n in (70, 1, 18, 33, 9, 50)]
    want = [greedy(cfg, tensors, p, 12) for p in prompts]
    # three slots, a budget smaller than the prompts and a pool for about three requests: portions, waiting, reuse
    e = Engine.from_folder(folder, dtype="float32", max_tokens=256, max_num_seqs=3, max_batched_tokens=32)
    assert e.generate(prompts, 12) == want
    assert e.pool.num_free == e.pool.num_blocks and not e.live
    (tmp_path / "p.jsonl").write_text("\n".join(json.dumps(p) for p in prompts))
    r = subprocess.run([sys.executable, "-m", "vllm_metal_b200", "generate", "--model", folder, "--prompts",
                        str(tmp_path / "p.jsonl"), "--max-new-tokens", "12", "--dtype", "float32", "--max-tokens", "512"],
                       cwd=ROOT, capture_output=True, text=True, timeout=240)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [json.loads(x) for x in r.stdout.splitlines() if x.startswith("[")] == want


def test_trace_replay_program(tmp_path):
    cfg = default_prenorm_config()
    tensors = random_checkpoint(cfg, seed=4)
    folder = write_folder(tmp_path / "model", cfg, tensors)
    toks = {k: np.random.default_rng(i).integers(0, cfg["vocab"], 50).tolist() for i, k in enumerate("ab")}
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks["a"][:20], "want": [19, 3]},
                                      {"id": "b", "tokens": toks["b"][:1], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": toks["b"][1:49], "want": [0]},
                                      {"id": "a", "tokens": toks["a"][20:21], "want": [0]}], "end": ["a"]},
             {"step": 2, "entries": [{"id": "b", "tokens": toks["b"][49:], "want": []}], "end": ["b"]}]
    out = tmp_path / "out"
    out.mkdir()
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", "float32", "--out", str(out),
                        "--max-tokens", "128"], input="\n".join(map(json.dumps, steps)) + "\n", capture_output=True,
                       text=True, timeout=240)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    w = {k: oracle.forward(cfg, to_oracle(tensors), t) for k, t in toks.items()}
    for n, rows in ((0, [w["a"][19], w["a"][3]]), (1, [w["b"][1], w["a"][20]])):
        got = np.fromfile(out / f"{n}.f32", "<f4").reshape(len(rows), -1)
        np.testing.assert_allclose(got, np.stack(rows), atol=1e-3)
    assert not (out / "2.f32").exists()


def test_worker_serves_the_model_from_scheduler_outputs(tmp_path):
    """The vLLM worker: loading by architecture, cache from the KV config, chunked prefill beside decoding."""
    pytest.importorskip("vllm")
    import types

    from vllm.v1.core.sched.output import CachedRequestData, NewRequestData, SchedulerOutput

    from vllm_metal_b200.v1.worker import B200Worker

    cfg = default_prenorm_config()
    tensors = random_checkpoint(cfg, seed=6)
    w = object.__new__(B200Worker)
    w._requests, w._pending, w._drafts, w._drafter, w._pipeline = {}, None, {}, None, None
    w.device, w.model = torch.device("cuda", 0), None
    w.parallel_config = types.SimpleNamespace(tensor_parallel_size=1)
    w.model_config = types.SimpleNamespace(hf_config=types.SimpleNamespace(**cfg),
                                           model=write_folder(tmp_path / "model", cfg, tensors), seed=0, max_model_len=256,
                                           enforce_eager=False, dtype=torch.float32)
    w.scheduler_config = types.SimpleNamespace(max_num_seqs=2)
    w.cache_config = types.SimpleNamespace(block_size=16, gpu_memory_utilization=0.5)
    w.vllm_config = types.SimpleNamespace(load_config=types.SimpleNamespace(load_format="auto"))
    w.load_model()
    assert sorted(w.get_kv_cache_spec()) == sorted(f"layers.{i}.self_attn" for i in (2, 4, 6, 7, 9))
    assert w.get_cache_block_size_bytes() == 16 * 4 * (3 * 2 * (24 + 40) + 4 * (16 + 8) + 24 + 40) and w.determine_available_memory() > 0
    w.initialize_from_config(types.SimpleNamespace(num_blocks=40, kv_cache_groups=[object()]))
    w.compile_or_warm_up_model()
    rng = np.random.default_rng(2)
    prompts = {r: rng.integers(0, cfg["vocab"], n).tolist() for r, n in (("A", 37), ("B", 9), ("C", 21))}
    blocks = {"A": [5, 9, 2, 17], "B": [3, 20], "C": [5, 7, 1]}
    computed, out = dict.fromkeys(prompts, 0), {r: [] for r in prompts}

    def run(num, new=(), finished=()):
        new_reqs = [NewRequestData(req_id=r, prompt_token_ids=prompts[r], mm_features=[], sampling_params=None,
                                   pooling_params=None, block_ids=(blocks[r],), num_computed_tokens=0, lora_request=None)
                    for r in new]
        old = [r for r in num if r not in new]
        cached = CachedRequestData(req_ids=old, resumed_req_ids=set(), new_token_ids=[[] for _ in old], all_token_ids={},
                                   new_block_ids=[None] * len(old), num_computed_tokens=[computed[r] for r in old],
                                   num_output_tokens=[1] * len(old))
        w.execute_model(SchedulerOutput(
            scheduled_new_reqs=new_reqs, scheduled_cached_reqs=cached, num_scheduled_tokens=num,
            total_num_scheduled_tokens=sum(num.values()), scheduled_spec_decode_tokens={}, scheduled_encoder_inputs={},
            num_common_prefix_blocks=[0], finished_req_ids=set(finished), free_encoder_mm_hashes=[]))
        got = w.sample_tokens(None)
        for r, t in zip(got.req_ids, got.sampled_token_ids, strict=True):
            computed[r] += num[r]
            out[r] += t

    run({"A": 20, "B": 9}, new=["A", "B"])
    run({"A": 17, "B": 1})
    for _ in range(3):
        run({"A": 1, "B": 1})
    run({"B": 1, "C": 21}, new=["C"], finished=["A"])  # C takes A's slot and one of its pages
    for _ in range(3):
        run({"B": 1, "C": 1})
    for r in prompts:
        assert out[r] == greedy(cfg, tensors, prompts[r], len(out[r])), r
