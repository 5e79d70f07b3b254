"""Host side of the pre-norm decoders with time mixing (no GPU): configuration, tensors, cache, component -- and the oracle's
mechanisms against closed forms."""

from __future__ import annotations

import copy
import math
import os
import re

import numpy as np
import pytest
import torch

from oracle import retuvik as oracle

from .hybrid_helpers import random_checkpoint, to_oracle, write_folder
from .prenorm_helpers import attention_layer, clear_routing, default_prenorm_config, experts, prenorm_config, wkv_layer


def test_configuration_reads_every_size_and_constant():
    from vllm_metal_b200.lm.hybrid_config import BiasedAttentionArgs, HybridArgs, RoutedArgs, TimeMixArgs
    from vllm_metal_b200.lm.hybrid_random import tensor_shapes

    c = prenorm_config([wkv_layer(experts(ff=9, n=5, top=5), heads=2, dim=12), attention_layer(), attention_layer(None, mask=None, q_temp=None)],
                       loop=(0, 2, 4), groups=5, scale=-0.5, vocab=99, width=40, eps=1e-3)
    a = HybridArgs.parse(c)
    assert (a.vocab, a.width, a.eps, a.norm_groups, a.embedding_scale, a.num_layers) == (99, 40, 1e-3, 5, -0.5, 9)
    assert a.design.layout == "prenorm" and a.streams == 1 and a.input_taps == 0
    assert a.passes == ((0, 0), (2, 1), (4, 2), (6, 3)) and a.loop_times == 4
    assert [layer.weights for layer in a.layers] == [0, 1] * 4 + [2]
    assert a.layers[0].mixer == TimeMixArgs(2, 12) and a.layers[0].routed == RoutedArgs(5, 5, 9, 1.0, 0, True)
    m = a.layers[1].mixer
    assert m == BiasedAttentionArgs(6, 2, 24, 40, 0.31, 29, 0.7, 19.0) and a.layers[1].ff == 56
    assert m.slopes() == [2.0 ** (-8 * (h + 1) / 6) for h in range(6)]
    n = a.layers[8].mixer
    assert (n.window, n.temp_coef) == (0, 0.0) and a.layers[8].routed is None and a.layers[8].ff == 0
    assert a.paged_layers() == {i: 2 * (24 + 40) for i in (1, 3, 5, 7, 8)}
    s = tensor_shapes(a)
    assert s["l0.mix.w2"] == (24, 40) and s["l0.mix.u"] == (2, 12) and s["l0.mix.mu.w"] == (40,) and s["l0.mlp.router.b"] == (5,)
    assert s["l1.mix.g"] == (240, 40) and s["l1.mlp.act"] == (2,) and s["l1.mlp.up.b"] == (56,) and s["loop.step"] == (4, 40)
    assert "l2.norm2" not in s and "l0.mlp.act" not in s and "l0.mlp.shared.up" not in s and "l1.mix.q.norm" in s
    assert HybridArgs.parse(prenorm_config([wkv_layer()])).passes == ()
    assert HybridArgs.parse(prenorm_config([wkv_layer()], loop=(1, 1, 3))).passes == ()


@pytest.mark.parametrize("edit,message", [
    (lambda c: c["layers"][0].update(type="mamba2"), "unknown mixer"),
    (lambda c: c["layers"][0]["mixer"].pop("dim"), "'dim' is missing"),
    (lambda c: c["layers"][0]["mixer"].update(heads=0), "heads must be"),
    (lambda c: c["layers"][1]["mixer"].pop("scale"), "'scale' is missing"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=4), "key/value heads"),
    (lambda c: c["layers"][1]["mixer"]["q_temp"].pop("every"), "'every' is missing"),
    (lambda c: c["layers"][1]["mixer"]["q_temp"].update(every=0), "q_temp.every"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(size=-2), "mask.size"),
    (lambda c: c["layers"][0]["mlp"].update(kind="swiglu"), "feed-forward kind"),
    (lambda c: c["layers"][2]["mlp"]["router"].update(top=8), "8 of 7 experts"),
    (lambda c: c["norm"].update(groups=3), "norm groups"),
    (lambda c: c["norm"].pop("groups"), "'groups' is missing"),
    (lambda c: c.pop("embedding"), "'embedding' is missing"),
    (lambda c: c["loop"].update(stop=4), "loop over layers"),
    (lambda c: c["loop"].update(times=0), "loop over layers"),
])
def test_configuration_errors_name_the_entry(edit, message):
    from vllm_metal_b200.lm.hybrid_config import ConfigError, HybridArgs

    c = prenorm_config([wkv_layer(), attention_layer(), wkv_layer(experts())], loop=(0, 2, 2))
    edit(c)
    with pytest.raises(ConfigError, match=message):
        HybridArgs.parse(c)


def test_registry_model_class_and_cache():
    from vllm_metal_b200.attention.caches.hybrid_cache import HybridCache, paged_bytes_per_token
    from vllm_metal_b200.lm.prenorm import PreNormModel
    from vllm_metal_b200.lm.registry import family_of

    cfg = default_prenorm_config()
    f = family_of(cfg)
    a = f.parse(cfg)
    assert f.component == "prenorm" and f.model_class(a) is PreNormModel and torch.float32 in f.dtypes
    c = HybridCache(a, 5, 16, 2, torch.bfloat16, "cpu")
    # runs: 0 | 1 2 | 1 2 | 1 2 | 3 4 5 6 -- a pass has a cache and a state of its own
    assert sorted(c.states) == [0, 1, 3, 5, 8, 10] and sorted(c.kv) == [2, 4, 6, 7, 9] and not c.latent and not c.previous
    assert c.states[1].matrix.shape == (3, 3, 40, 40) and c.states[1].last.shape == (3, 88)
    assert c.states[1].matrix.dtype == c.states[1].last.dtype == torch.float32
    assert [t.shape for t in c.kv[2]] == [(5, 16, 2, 24), (5, 16, 2, 40)]
    states = 4 * (5 * 24 * 24 + 3 * 3 * 40 * 40 + 2 * 32 * 32 + 64 * 64 + 6 * 88)
    assert HybridCache.state_bytes_per_slot(a, torch.bfloat16) == states
    assert c.nbytes == 5 * 16 * paged_bytes_per_token(a, torch.bfloat16) + 3 * states


def test_the_component_holds_every_symbol_its_models_call():
    from vllm_metal_b200.metal import EXPORTED_SYMBOLS
    from vllm_metal_b200.metal.build import sources
    from vllm_metal_b200.metal.hybrid_ops import PRENORM_SYMBOLS

    text = "\n".join(f.read_text() for f in sources("prenorm"))
    for name in (*PRENORM_SYMBOLS, "b200_residual_step", "b200_rope_norm_cache", "b200_recurrence", "b200_mixer_finish",
                 "b200_expert_route", "b200_expert_plan", "b200_expert_product", "b200_paged_attention", "b200_argmax",
                 "b200_advance_decode", "b200_last_error"):
        assert name in EXPORTED_SYMBOLS and re.search(rf"\b{name}\s*\(", text), name


def test_struct_layouts_match_the_header():
    """Fields of the ctypes mirrors in the header's order, with its types."""
    import ctypes

    from vllm_metal_b200.metal import hybrid_ops

    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    with open(os.path.join(root, "include", "b200_hybrid_ops.h"), encoding="utf-8") as f:
        text = re.sub(r"/\*.*?\*/", "", f.read(), flags=re.S)
    kinds = {"int64_t": "c_int64", "int32_t": "c_int32", "float": "c_float", "size_t": "c_size_t"}
    for name, mirror in (("residual_step", hybrid_ops.ResidualStepArgs), ("rope_norm_cache", hybrid_ops.RopeNormCacheArgs),
                         ("mixer_finish", hybrid_ops.MixerFinishArgs), ("recurrence", hybrid_ops.RecurrenceArgs)):
        body = re.search(rf"typedef struct b200_{name}_args \{{(.*?)\}} b200_{name}_args;", text, flags=re.S).group(1)
        fields = []
        for line in body.split(";"):
            if not line.strip():
                continue
            t, rest = re.match(r"\s*(?:const\s+)?(\w+)\s*(.*)", line.strip(), flags=re.S).groups()
            for v in rest.split(","):
                fields.append((v.strip().lstrip("*").strip(), ctypes.c_void_p if "*" in v else getattr(ctypes, kinds[t])))
        assert fields == list(mirror._fields_), name


def test_a_bottleneck_has_the_size_of_its_tensor(tmp_path):
    """The decays' bottleneck is in no configuration: weights of any rank load, another tensor of a wrong size does not."""
    from vllm_metal_b200.lm.prenorm import PreNormModel
    from vllm_metal_b200.lm.registry import family_of

    cfg = prenorm_config([wkv_layer(None)])
    tensors = random_checkpoint(cfg)
    for rank in (1, 7, 48):
        tensors["l0.mix.w1"], tensors["l0.mix.w2"] = torch.ones(rank, 88).bfloat16(), torch.ones(120, rank).bfloat16()
        m = PreNormModel.from_folder(family_of(cfg).parse(cfg), write_folder(tmp_path / str(rank), cfg, tensors), torch.bfloat16, "cpu")
        assert m.layers[0].mixer.decay_down.weight.shape == (-(-rank // 8) * 8, 88)
    tensors["l0.mix.w2"] = torch.ones(119, 48).bfloat16()
    with pytest.raises(ValueError, match="l0.mix.w2"):
        PreNormModel.from_folder(family_of(cfg).parse(cfg), write_folder(tmp_path / "bad", cfg, tensors), torch.bfloat16, "cpu")


# -- the oracle's mechanisms ------------------------------------------------------------------------------------

def test_oracle_grouped_norm_and_token_mix():
    x = np.array([[3.0, 4.0, 0.0, 2.0], [1.0, 1.0, 5.0, 5.0]])
    got = oracle.grouped_norm(x, [1.0, 2.0, 1.0, 1.0], 2, 0.0)
    r = math.sqrt(12.5)
    np.testing.assert_allclose(got, [[3 / r, 8 / r, 0, math.sqrt(2)], [1, 2, 1, 1]])
    np.testing.assert_allclose(oracle.grouped_norm(x, np.ones(4), 1, 0.0)[0], x[0] / math.sqrt(29 / 4))
    np.testing.assert_allclose(oracle.token_mix(x, [0.0, 1.0, 0.5, 0.25]), [[3, 0, 0, 1.5], [1, 4, 2.5, 4.25]])


def test_oracle_recurrence_is_the_sum_over_earlier_rows():
    rng = np.random.default_rng(0)
    t, h, n = 7, 2, 3
    r, k = rng.standard_normal((2, t, h, n))
    v, w, u = rng.standard_normal((t, h, 4)), rng.random((t, h, n)), rng.standard_normal((h, n))
    got = oracle.wkv(r, k, v, w, u)
    for a in range(h):
        for i in range(t):
            want = (r[i, a] * u[a] * k[i, a]).sum() * v[i, a]
            for j in range(i):
                want = want + (r[i, a] * np.prod(w[j + 1:i, a], axis=0) * k[j, a]).sum() * v[j, a]
            np.testing.assert_allclose(got[i, a], want, atol=1e-12)


def test_oracle_attention_takes_the_distance_off_the_scores():
    rng = np.random.default_rng(1)
    q, k, v = rng.standard_normal((9, 4, 3)), rng.standard_normal((9, 2, 3)), rng.standard_normal((9, 2, 5))
    slope = oracle.slopes(4)
    np.testing.assert_allclose(slope, [0.25, 0.0625, 2.0 ** -6, 2.0 ** -8])
    got = oracle.biased_attention(q, k, v, 0.7, slope, {"size": 4})
    for h in range(4):
        for i in range(9):
            js = range(max(0, i - 3), i + 1)
            s = np.exp([0.7 * k[j, h // 2] @ q[i, h] - slope[h] * (i - j) for j in js])
            np.testing.assert_allclose(got[i, h], s @ v[list(js), h // 2] / s.sum(), atol=1e-12)
    assert [j for j in range(12) if oracle.visible(9, j, {"size": 3})] == [7, 8, 9]
    assert [j for j in range(5) if oracle.visible(3, j, None)] == [0, 1, 2, 3]


def test_oracle_temperature_activation_and_routing():
    got = oracle.temperature([0, 8, 9, 18, 19, 1000], {"coef": 0.5, "every": 10})
    np.testing.assert_allclose(got, 1 + 0.5 * np.log([1, 1, 2, 2, 3, 101]))
    assert (oracle.temperature([0, 5], None) == 1).all()
    z = np.array([-2.0, -1e-3, 0.0, 3.0])
    p, q = math.log(1 + math.exp(0.3)), math.log(1 + math.exp(-0.4))
    np.testing.assert_allclose(oracle.xielu(z, [0.3, -0.4]), [(0.5 + q) * (math.exp(-2) + 1) - 1, (0.5 + q) * 5e-7 - 5e-4, 0, p * 9 + 1.5],
                               rtol=1e-3)
    chosen, w = oracle.route(np.log(np.array([[1.0, 6.0, 2.0, 3.0]])), 2)
    assert chosen.tolist() == [[1, 3]]
    np.testing.assert_allclose(w, [[2 / 3, 1 / 3]])
    assert oracle.route(np.zeros((1, 4)), 3)[0].tolist() == [[0, 1, 2]]


def test_oracle_order_of_a_loop():
    c = {"layers": [None] * 4, "loop": {"start": 1, "stop": 3, "times": 2}}
    assert oracle.order(c) == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (3, None)]
    assert oracle.order({"layers": [None] * 2}) == [(0, None), (1, None)]


@pytest.mark.parametrize("edit", ["mu", "before", "bonus", "decay", "w0", "tanh", "head_norm", "norm_weight", "gate", "scale", "window",
                                  "slope", "slope_shared", "temp_coef", "temp_every", "value_norm", "q_norm", "output_gate", "kv_heads",
                                  "groups", "eps", "act", "up_bias", "down_bias", "top", "router_bias", "weights_of_all", "expert",
                                  "embedding_scale", "loop_embedding", "loop_step", "loop_times"])
def test_a_planted_mistake_in_the_oracle_shows(edit, monkeypatch):
    """Every mechanism moves the logits of a small model: an oracle that gets one wrong is told apart."""
    cfg = default_prenorm_config()
    tensors = random_checkpoint(cfg)
    clear_routing(cfg)(tensors)
    t = to_oracle(tensors)
    toks = np.random.default_rng(0).integers(0, cfg["vocab"], 60).tolist()
    right = oracle.forward(cfg, t, toks)
    bad_cfg, bad = copy.deepcopy(cfg), dict(t)
    mixer, mlp = bad_cfg["layers"][2]["mixer"], bad_cfg["layers"][1]["mlp"]
    exact = {n: getattr(oracle, n) for n in ("wkv", "over_rms", "route", "order", "silu", "sigmoid", "biased_attention")}
    if edit == "mu":
        bad["l0.mix.mu.k"] = t["l0.mix.mu.v"]
    elif edit == "before":
        monkeypatch.setattr(oracle, "before", lambda h: np.concatenate([h[:1], h[:-1]]))
    elif edit == "bonus":
        bad["l0.mix.u"] = np.ones_like(t["l0.mix.u"])
    elif edit == "decay":  # the state decays before the row reads it
        monkeypatch.setattr(oracle, "wkv", lambda r, k, v, w, u: exact["wkv"](r * w, k, v, w, u))
    elif edit == "w0":
        bad["l1.mix.w0"] = np.zeros_like(t["l1.mix.w0"])
    elif edit == "tanh":
        bad["l0.mix.w1"] = np.zeros_like(t["l0.mix.w1"])
    elif edit == "head_norm":
        monkeypatch.setattr(oracle, "wkv", lambda r, k, v, w, u: exact["wkv"](r, k, v, w, u) * np.linspace(0.5, 2, v.shape[2]))
    elif edit == "norm_weight":
        bad["l1.mix.norm"] = np.ones_like(t["l1.mix.norm"])
    elif edit == "gate":
        bad["l4.mix.g"] = -t["l4.mix.g"]
    elif edit == "scale":
        mixer["scale"] = 0.2
    elif edit == "window":
        mixer["mask"]["size"] = 28
    elif edit == "slope":
        monkeypatch.setattr(oracle, "slopes", lambda heads: np.zeros(heads))
    elif edit == "slope_shared":  # by key/value head instead of query head
        monkeypatch.setattr(oracle, "slopes", lambda heads: 2.0 ** (-8.0 * np.arange(heads) / heads))
    elif edit == "temp_coef":
        mixer["q_temp"]["coef"] = 0.0
    elif edit == "temp_every":
        mixer["q_temp"]["every"] = 20
    elif edit == "value_norm":
        monkeypatch.setattr(oracle, "biased_attention", lambda q, k, v, *a: exact["biased_attention"](
            q, k, v * np.linspace(0.5, 2.0, len(v))[:, None, None], *a))
    elif edit == "q_norm":
        bad["l2.mix.q.norm"] = np.ones_like(t["l2.mix.q.norm"])
    elif edit == "output_gate":
        bad["l3.mix.g"] = np.zeros_like(t["l3.mix.g"])
    elif edit == "kv_heads":
        bad["l2.mix.q"] = np.roll(t["l2.mix.q"], 24, axis=0)
    elif edit == "groups":
        bad_cfg["norm"]["groups"] = 2
    elif edit == "eps":
        bad_cfg["norm"]["eps"] = 1e-1
    elif edit == "act":
        bad["l0.mlp.act"] = t["l0.mlp.act"][::-1]
    elif edit in ("up_bias", "down_bias"):
        name = f"l2.mlp.{edit[:-5]}.b"
        bad[name] = np.zeros_like(t[name])
    elif edit == "top":
        mlp["router"]["top"] = 2
    elif edit == "router_bias":
        bad["l1.mlp.router.b"] = np.zeros_like(t["l1.mlp.router.b"])
    elif edit == "weights_of_all":
        def of_all(z, top):
            e = np.exp(z - z.max(axis=1, keepdims=True))
            chosen = exact["route"](z, top)[0]
            return chosen, np.take_along_axis(e / e.sum(axis=1, keepdims=True), chosen, axis=1)

        monkeypatch.setattr(oracle, "route", of_all)
    elif edit == "expert":
        bad["l1.mlp.e3.up"], bad["l1.mlp.e4.up"] = t["l1.mlp.e4.up"], t["l1.mlp.e3.up"]
    elif edit == "embedding_scale":
        bad_cfg["embedding"]["scale"] = 3.3
    elif edit == "loop_embedding":  # every pass counts as the first
        monkeypatch.setattr(oracle, "order", lambda c: [(i, None if n is None else 0) for i, n in exact["order"](c)])
    elif edit == "loop_step":
        bad["loop.step"] = t["loop.step"][::-1]
    elif edit == "loop_times":
        bad_cfg["loop"]["times"] = 2
    err = np.sqrt(((oracle.forward(bad_cfg, bad, toks) - right) ** 2).mean(1)) / right.std()
    assert err[40:].max() > 1e-3, err.max()
    if edit == "window":
        assert (err[:28] == 0).all()  # while everything is still inside the window
