"""Host side of the sandwich-norm decoders with routed experts (no GPU): configuration, tensors, cache, component -- and the
oracle's mechanisms against closed forms."""

from __future__ import annotations

import copy
import math
import re

import numpy as np
import pytest
import torch

from oracle import kerolorn as oracle

from .hybrid_helpers import random_checkpoint, to_oracle
from .sandwich_helpers import clear_routing, default_sandwich_config, experts, sandwich_config, sandwich_layer


def test_configuration_reads_every_size_and_constant():
    from vllm_metal_b200.lm.hybrid_config import HybridArgs, RoutedArgs
    from vllm_metal_b200.lm.hybrid_random import tensor_shapes

    c = sandwich_config([sandwich_layer(), sandwich_layer(None, mask=None, rot=None),
                         sandwich_layer(experts(ff=9, n=5, top=5, scale=0.5, shared=None), mask={"size": 3})],
                        taps=5, logit_scale=-2.0, vocab=99, width=40, eps=1e-3)
    a = HybridArgs.parse(c)
    assert (a.vocab, a.width, a.eps, a.input_taps, a.logit_scale, a.num_layers) == (99, 40, 1e-3, 5, -2.0, 3)
    assert a.design.layout == "sandwich" and a.streams == 1
    m = a.layers[0].mixer
    assert (m.heads, m.kv_heads, m.dim, m.vdim, m.scale, m.window, m.keep_first) == (6, 2, 24, 40, 0.31, 29, 5)
    assert (m.rot.dims, m.rot.base, m.rot.factor, m.rot.original, m.rot.fast, m.rot.slow) == (16, 5000.0, 4.0, 96.0, 8.0, 0.5)
    assert a.layers[0].routed == RoutedArgs(7, 3, 40, 1.7, 56) and a.layers[2].routed == RoutedArgs(5, 5, 9, 0.5, 0)
    n = a.layers[1].mixer
    assert a.layers[1].routed is None and n.window == n.keep_first == n.rot.dims == 0 and n.rot.amplitude == 1.0
    assert (a.layers[2].mixer.window, a.layers[2].mixer.keep_first) == (3, 0)
    assert a.paged_layers() == {i: 2 * (24 + 40) for i in range(3)}
    s = tensor_shapes(a)
    assert s["l0.canon1"] == (40, 5) and s["l0.mix.temp"] == (6,) and s["l0.mix.k"] == (48, 40) and s["l0.mix.o"] == (40, 240)
    assert s["l0.mlp.e6.down"] == (40, 40) and s["l0.mlp.router"] == (7, 40) and s["l0.mlp.shared.sg"] == (1, 40)
    assert s["l2.mlp.e4.gate"] == (9, 40) and "l2.mlp.shared.up" not in s and "l0.mlp.e7.up" not in s
    assert "l1.norm1b" in s and "l1.norm2" not in s and "l1.norm2b" not in s and s["l2.norm2b"] == (40,)


@pytest.mark.parametrize("edit,message", [
    (lambda c: c["layers"][0].update(type="lightning"), "unknown mixer"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "'scale' is missing"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "key/value heads"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=26), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=3), "even"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("slow"), "'slow' is missing"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].update(factor=0.0), "must be positive"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(keep_first=-1), "keep_first"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "feed-forward kind"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=8), "8 of 7 experts"),
    (lambda c: c["layers"][0]["mlp"]["router"].pop("scale"), "'scale' is missing"),
    (lambda c: c["layers"][0]["mlp"]["expert"].update(ff=0), "ff must be"),
    (lambda c: c["layers"][0]["mlp"]["shared"].update(ff=0), "shared"),
    (lambda c: c["canon"].update(taps=0), "canon.taps"),
    (lambda c: c.pop("canon"), "'canon' is missing"),
    (lambda c: c.pop("logit_scale"), "'logit_scale' is missing"),
])
def test_configuration_errors_name_the_entry(edit, message):
    from vllm_metal_b200.lm.hybrid_config import ConfigError, HybridArgs

    c = sandwich_config([sandwich_layer(), sandwich_layer(None)])
    edit(c)
    with pytest.raises(ConfigError, match=message):
        HybridArgs.parse(c)


def test_registry_model_class_and_cache():
    from vllm_metal_b200.attention.caches.hybrid_cache import HybridCache, paged_bytes_per_token
    from vllm_metal_b200.lm.registry import family_of
    from vllm_metal_b200.lm.sandwich import SandwichModel

    cfg = default_sandwich_config()
    f = family_of(cfg)
    a = f.parse(cfg)
    assert f.component == "sandwich" and f.model_class(a) is SandwichModel and torch.float32 in f.dtypes
    c = HybridCache(a, 5, 16, 2, torch.bfloat16, "cpu")
    assert sorted(c.kv) == sorted(c.previous) == list(range(4)) and not c.latent and not c.states
    assert [t.shape for t in c.kv[0]] == [(5, 16, 2, 24), (5, 16, 2, 40)] and c.kv[3][1].shape == (5, 16, 4, 8)
    assert c.previous[2].shape == (3, 3, 88) and c.previous[2].dtype == torch.bfloat16
    assert paged_bytes_per_token(a, torch.bfloat16) == 2 * (3 * 2 * (24 + 40) + 4 * (16 + 8))
    assert HybridCache.state_bytes_per_slot(a, torch.bfloat16) == 4 * 3 * 88 * 2
    assert c.nbytes == 5 * 16 * paged_bytes_per_token(a, torch.bfloat16) + 3 * HybridCache.state_bytes_per_slot(a, torch.bfloat16)


def test_the_component_holds_every_symbol_its_models_call():
    from vllm_metal_b200.metal import EXPORTED_SYMBOLS
    from vllm_metal_b200.metal.build import sources
    from vllm_metal_b200.metal.hybrid_ops import SANDWICH_SYMBOLS

    text = "\n".join(f.read_text() for f in sources("sandwich"))
    for name in (*SANDWICH_SYMBOLS, "b200_embed_rows", "b200_mixer_finish", "b200_causal_conv", "b200_paged_attention", "b200_argmax",
                 "b200_advance_decode", "b200_last_error"):
        assert name in EXPORTED_SYMBOLS and re.search(rf"\b{name}\s*\(", text), name


def test_struct_layouts_match_the_header():
    """Fields of the ctypes mirrors in the header's order, with its types."""
    import os

    from vllm_metal_b200.metal import hybrid_ops

    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    with open(os.path.join(root, "include", "b200_hybrid_ops.h"), encoding="utf-8") as f:
        text = re.sub(r"/\*.*?\*/", "", f.read(), flags=re.S)
    kinds = {"int64_t": "c_int64", "int32_t": "c_int32", "float": "c_float", "size_t": "c_size_t"}
    import ctypes

    for name, mirror in (("residual_step", hybrid_ops.ResidualStepArgs), ("rope_norm_cache", hybrid_ops.RopeNormCacheArgs),
                         ("expert_product", hybrid_ops.ExpertProductArgs)):
        body = re.search(rf"typedef struct b200_{name}_args \{{(.*?)\}} b200_{name}_args;", text, flags=re.S).group(1)
        fields = []
        for line in body.split(";"):
            if not line.strip():
                continue
            t, rest = re.match(r"\s*(?:const\s+)?(\w+)\s*(.*)", line.strip(), flags=re.S).groups()
            for v in rest.split(","):
                fields.append((v.strip().lstrip("*").strip(), ctypes.c_void_p if "*" in v else getattr(ctypes, kinds[t])))
        assert fields == list(mirror._fields_), name


def test_frequencies_agree_with_the_oracle_and_keep_more_than_32_bits():
    from vllm_metal_b200.lm.hybrid_config import RotaryArgs

    for rot in ({"base": 1e4, "dims": 64}, {"base": 5e5, "dims": 6, "scaling": {"factor": 8.0, "original": 64, "fast": 4.0, "slow": 1.0}},
                {"base": 1e4, "dims": 48, "scaling": {"factor": 3.0, "original": 4096, "fast": 32.0, "slow": 1.0}},
                {"base": 20.0, "dims": 8, "scaling": {"factor": 1.5, "original": 7, "fast": 3.0, "slow": 3.0}}):
        a = RotaryArgs.parse(rot, "x")
        want, amplitude = oracle.frequencies(rot)
        np.testing.assert_allclose(a.frequencies(), want, rtol=1e-14)
        assert a.amplitude == amplitude
    # fast pairs keep their frequency, slow ones are divided by the factor
    f, plain = (oracle.frequencies({"base": 1e4, "dims": 64, **s})[0] for s in (
        {"scaling": {"factor": 4.0, "original": 2048, "fast": 32.0, "slow": 1.0}}, {}))
    assert f[0] == plain[0] and math.isclose(f[-1], plain[-1] / 4) and (np.diff(plain / f) >= -1e-12).all()


# -- the oracle's mechanisms ------------------------------------------------------------------------------------

def test_oracle_rotation_turns_neighbouring_pairs_and_passes_the_rest():
    x = np.random.default_rng(0).standard_normal((5, 2, 7))
    rot = {"base": 100.0, "dims": 4}
    got = oracle.rotate(x, [0, 1, 2, 30, 4], rot)
    assert np.array_equal(got[0], x[0]) and np.array_equal(got[:, :, 4:], x[:, :, 4:])
    for i in range(2):
        z = (x[3, 1, 2 * i] + 1j * x[3, 1, 2 * i + 1]) * np.exp(1j * 30 * 100.0 ** (-i / 2))
        np.testing.assert_allclose(got[3, 1, 2 * i:2 * i + 2], [z.real, z.imag])


def test_oracle_window_and_kept_tokens():
    m = {"size": 3, "keep_first": 2}
    assert [j for j in range(12) if oracle.visible(9, j, m)] == [0, 1, 7, 8, 9]
    assert [j for j in range(12) if oracle.visible(1, j, m)] == [0, 1]
    assert [j for j in range(12) if oracle.visible(3, j, m)] == [0, 1, 2, 3]
    assert [j for j in range(12) if oracle.visible(4, j, {"size": 1, "keep_first": 9})] == [0, 1, 2, 3, 4]
    assert [j for j in range(12) if oracle.visible(6, j, {"size": 2})] == [5, 6]
    assert [j for j in range(5) if oracle.visible(3, j, None)] == [0, 1, 2, 3]


def test_oracle_attention_shares_heads_and_scales_each():
    rng = np.random.default_rng(1)
    q, k, v = rng.standard_normal((9, 4, 3)), rng.standard_normal((9, 2, 3)), rng.standard_normal((9, 2, 5))
    scale, m = np.array([0.7, -0.2, 1.3, 0.0]), {"size": 4, "keep_first": 1}
    got = oracle.softmax_attention(q, k, v, scale, m)
    for h in range(4):
        for i in range(9):
            js = [j for j in range(9) if oracle.visible(i, j, m)]
            s = np.exp(scale[h] * k[js, h // 2] @ q[i, h])
            np.testing.assert_allclose(got[i, h], s @ v[js, h // 2] / s.sum(), atol=1e-12)


def test_oracle_convolution_and_routing():
    h = np.random.default_rng(2).standard_normal((6, 3))
    w = np.array([[0.5, 0.0, 2.0]] * 3)
    got = oracle.input_convolution(h, w)
    np.testing.assert_allclose(got[4], h[4] + 2 * h[4] + 0.5 * h[2])
    np.testing.assert_allclose(got[0], 3 * h[0])
    z = np.log(np.array([[1.0, 2.0, 3.0, 4.0]]))
    chosen, weights = oracle.route(z, [0.0, 0.35, 0.0, -0.05], 2, 3.0)
    assert chosen.tolist() == [[1, 3]]
    np.testing.assert_allclose(weights, [[0.6, 1.2]])   # scores without their corrections, not renormalised
    assert oracle.route(np.zeros((1, 4)), np.zeros(4), 3, 1.0)[0].tolist() == [[0, 1, 2]]


@pytest.mark.parametrize("edit", ["conv", "conv_side", "rot_base", "rot_dims", "scaling", "amplitude", "temp", "scale", "window",
                                  "keep_first", "norm1b", "norm2b", "top", "router_scale", "correction", "shared", "sg", "expert",
                                  "kv_heads", "logit_scale", "eps"])
def test_a_planted_mistake_in_the_oracle_shows(edit, monkeypatch):
    """Every mechanism moves the logits of a small model: an oracle that gets one wrong is told apart."""
    cfg = default_sandwich_config()
    tensors = random_checkpoint(cfg)
    clear_routing(cfg)(tensors)
    t = to_oracle(tensors)
    toks = np.random.default_rng(0).integers(0, cfg["vocab"], 60).tolist()
    right = oracle.forward(cfg, t, toks)
    bad_cfg, bad = copy.deepcopy(cfg), dict(t)
    mixer, mlp = bad_cfg["layers"][0]["mixer"], bad_cfg["layers"][0]["mlp"]
    if edit == "conv":
        bad["l2.canon1"] = np.zeros_like(t["l2.canon1"])
    elif edit == "conv_side":
        bad["l0.canon1"] = t["l0.canon1"][:, ::-1]
    elif edit == "rot_base":
        mixer["rot"]["base"] = 900.0
    elif edit == "rot_dims":
        mixer["rot"]["dims"] = 14
    elif edit == "scaling":
        mixer["rot"].pop("scaling")
    elif edit == "amplitude":
        exact = oracle.frequencies
        monkeypatch.setattr(oracle, "frequencies", lambda rot: (exact(rot)[0], 1.0))
    elif edit == "temp":
        bad["l1.mix.temp"] = np.ones_like(t["l1.mix.temp"])
    elif edit == "scale":
        mixer["scale"] = 0.2
    elif edit == "window":
        mixer["mask"]["size"] = 28
    elif edit == "keep_first":
        mixer["mask"]["keep_first"] = 4
    elif edit in ("norm1b", "norm2b"):
        bad[f"l0.{edit}"] = np.ones_like(t[f"l0.{edit}"])
    elif edit == "top":
        mlp["router"]["top"] = 2
    elif edit == "router_scale":
        mlp["router"]["scale"] = 1.0
    elif edit == "correction":
        bad["l0.mlp.correction"] = np.zeros_like(t["l0.mlp.correction"])
    elif edit == "shared":
        mlp.pop("shared")
    elif edit == "sg":
        bad["l3.mlp.shared.sg"] = np.zeros_like(t["l3.mlp.shared.sg"])
    elif edit == "expert":
        bad["l0.mlp.e3.up"], bad["l0.mlp.e4.up"] = t["l0.mlp.e4.up"], t["l0.mlp.e3.up"]
    elif edit == "kv_heads":
        bad["l0.mix.q"] = np.roll(t["l0.mix.q"], 24, axis=0)
    elif edit == "logit_scale":
        bad_cfg["logit_scale"] = 0.71
    elif edit == "eps":
        bad_cfg["norm"]["eps"] = 1e-1
    err = np.sqrt(((oracle.forward(bad_cfg, bad, toks) - right) ** 2).mean(1)) / right.std()
    assert err[40:].max() > 1e-3, err.max()
    if edit in ("window", "keep_first"):
        assert (err[:28 if edit == "window" else 33] == 0).all()  # while everything is still inside the window
