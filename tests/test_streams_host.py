"""Host side of the hyper-connected decoders (no GPU): configuration, loops, tensors, caches, components -- and the
oracle's mechanisms against closed forms."""

from __future__ import annotations

import copy
import re

import numpy as np
import pytest
import torch

from oracle import tatazen as oracle

from .hybrid_helpers import default_config, random_checkpoint, to_oracle
from .stream_helpers import default_stream_config, stream_config, stream_layer


def test_configuration_reads_every_size_and_unrolls_the_loop():
    from vllm_metal_b200.lm.hybrid_config import HybridArgs
    from vllm_metal_b200.lm.hybrid_random import tensor_shapes

    c = stream_config([stream_layer("parallel", ff=72), stream_layer("lightning", ff=None, decay=[0.0, 1.0, 0.5]),
                       stream_layer("lightning")], streams=5, loop=(0, 2, 3), vocab=99, width=40, eps=1e-3)
    a = HybridArgs.parse(c)
    assert (a.vocab, a.width, a.eps, a.streams, a.num_layers) == (99, 40, 1e-3, 5, 7)
    assert [x.weights for x in a.layers] == [0, 1, 0, 1, 0, 1, 2] and [x.ff for x in a.layers] == [72, 0] * 3 + [56]
    assert a.layers_of("parallel") == [0, 2, 4] and list(a.owners()) == [0, 1, 2]
    left, right = a.layers[0].mixer.left, a.layers[0].mixer.right
    assert (left.heads, left.kv_heads, left.dim, left.vdim, left.scale) == (6, 2, 24, 40, 0.31)
    assert (right.heads, right.dim, right.vdim, right.decay) == (2, 16, 56, (0.8, 0.99))
    assert a.layers[1].mixer.decay == (0.0, 1.0, 0.5)
    assert a.paged_layers() == {i: 2 * (24 + 40) for i in (0, 2, 4)}
    s = tensor_shapes(a)
    assert s["l0.mix.left.k"] == (48, 40) and s["l0.mix.left.o"] == (40, 240) and s["l0.mix.right.norm"] == (112,)
    assert s["l0.hc2.mix"] == (5, 5) and s["l0.rg2.b"] == (40,) and s["l1.shift"] == (40,) and s["l2.mlp.gate"] == (56, 40)
    assert "l1.norm2" not in s and "l1.rg2" not in s and "l3.norm1" not in s
    c.pop("loop")
    assert HybridArgs.parse(c).num_layers == 3


@pytest.mark.parametrize("edit,message", [
    (lambda c: c["layers"][0].update(type="mamba2"), "unknown mixer"),
    (lambda c: c["layers"][0]["mixer"].pop("left"), "'left' is missing"),
    (lambda c: c["layers"][0]["mixer"]["left"].pop("scale"), "left: 'scale' is missing"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=4), "key/value heads"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(scale=0.0), "scale"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(decay=[0.5]), "decay"),
    (lambda c: c["layers"][1]["mixer"].update(decay=[0.5, 0.5, 1.5]), "decay"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "feed-forward kind"),
    (lambda c: c.update(loop={"start": 1, "stop": 3, "times": 2}), "loop over layers"),
    (lambda c: c.update(loop={"start": 0, "stop": 1}), "'times' is missing"),
    (lambda c: c.update(streams=0), "streams"),
    (lambda c: c.pop("streams"), "'streams' is missing"),
])
def test_configuration_errors_name_the_entry(edit, message):
    from vllm_metal_b200.lm.hybrid_config import ConfigError, HybridArgs

    c = stream_config([stream_layer("parallel"), stream_layer("lightning")])
    edit(c)
    with pytest.raises(ConfigError, match=message):
        HybridArgs.parse(c)


def test_designs_do_not_share_mixers():
    from vllm_metal_b200.lm.hybrid_config import ConfigError, HybridArgs

    c = default_config()
    c["layers"][0] = stream_layer("lightning")
    with pytest.raises(ConfigError, match="unknown mixer"):
        HybridArgs.parse(c)


def test_registry_model_class_and_cache():
    from vllm_metal_b200.attention.caches.hybrid_cache import HybridCache, paged_bytes_per_token
    from vllm_metal_b200.lm.hybrid import HybridModel
    from vllm_metal_b200.lm.registry import family_of
    from vllm_metal_b200.lm.streams import StreamModel

    cfg = default_stream_config()
    f = family_of(cfg)
    a = f.parse(cfg)
    assert f.component == "streams" and f.model_class(a) is StreamModel
    other = family_of(default_config())
    assert other.component == "hybrid" and other.model_class(other.parse(default_config())) is HybridModel
    # layers: 0 | 1 2 | 1 2 | 3, every pass with a cache of its own
    assert [x.weights for x in a.layers] == [0, 1, 2, 1, 2, 3]
    c = HybridCache(a, 5, 16, 2, torch.bfloat16, "cpu")
    assert sorted(c.kv) == [1, 3, 5] and sorted(c.states) == sorted(c.previous) == list(range(6)) and not c.latent
    assert [t.shape for t in c.kv[3]] == [(5, 16, 2, 24), (5, 16, 2, 40)] and c.states[1].matrix.shape == (3, 2, 16, 56)
    assert c.previous[4].shape == (3, 1, 88) and c.previous[4].dtype == torch.bfloat16
    assert c.kv[1][0].data_ptr() != c.kv[3][0].data_ptr()
    assert paged_bytes_per_token(a, torch.bfloat16) == 3 * 2 * (24 + 40) * 2
    assert c.nbytes == 5 * 16 * paged_bytes_per_token(a, torch.bfloat16) + 3 * HybridCache.state_bytes_per_slot(a, torch.bfloat16)
    c.kv[5][1][1] = 1.0
    c.kv[5][1][2] = 2.0
    c.copy_blocks([(1, 2), (2, 1)])
    assert float(c.kv[5][1][1, 0, 0, 0]) == 2.0 and float(c.kv[5][1][2, 0, 0, 0]) == 1.0


def test_the_streams_component_holds_every_symbol_its_models_call():
    from vllm_metal_b200.metal import EXPORTED_SYMBOLS
    from vllm_metal_b200.metal.build import sources
    from vllm_metal_b200.metal.hybrid_ops import STREAM_SYMBOLS

    text = "\n".join(f.read_text() for f in sources("streams"))
    for name in (*STREAM_SYMBOLS, "b200_mixer_finish", "b200_causal_conv", "b200_recurrence", "b200_norm_rope_cache",
                 "b200_paged_attention", "b200_argmax", "b200_advance_decode", "b200_last_error"):
        assert name in EXPORTED_SYMBOLS and re.search(rf"\b{name}\s*\(", text), name


def test_the_component_asked_for_is_loaded_first(monkeypatch):
    from vllm_metal_b200 import metal
    from vllm_metal_b200.metal import build

    monkeypatch.setattr(build, "stale_artifacts", lambda component=None: [] if component else ["full"])
    monkeypatch.setattr(build, "build", lambda component=None: build.output_path(component))
    monkeypatch.setattr(build, "_wanted", [])
    for name in ("streams", "hybrid"):
        build.ensure(name)
        assert metal._component_library() == build.output_path(name)


def test_frequencies_keep_more_than_32_bits():
    from vllm_metal_b200.lm.streams import sinusoid_frequencies

    for width in (7, 64):
        f = sinusoid_frequencies(width).double().sum(1).numpy()
        want = 10000.0 ** (-2.0 * np.arange(-(-width // 2)) / width)
        np.testing.assert_allclose(f, want, rtol=1e-13)


# -- the oracle's mechanisms ------------------------------------------------------------------------------------

def test_oracle_lightning_equals_the_quadratic_form():
    rng = np.random.default_rng(0)
    q, k, v = rng.standard_normal((25, 3, 4)), rng.standard_normal((25, 3, 4)), rng.standard_normal((25, 3, 5))
    decay = [0.0, 1.0, 0.7]
    got = oracle.lightning_recurrence(q, k, v, decay)
    i = np.arange(25)
    for h in range(3):
        w = np.tril(np.where(i[:, None] >= i, float(decay[h]) ** np.maximum(i[:, None] - i, 0), 0.0) * (q[:, h] @ k[:, h].T))
        np.testing.assert_allclose(got[:, h], w @ v[:, h], atol=1e-12)


def test_oracle_attention_shares_heads_and_sees_the_past_only():
    rng = np.random.default_rng(1)
    q, k, v = rng.standard_normal((9, 4, 3)), rng.standard_normal((9, 2, 3)), rng.standard_normal((9, 2, 5))
    got = oracle.softmax_attention(q, k, v, 0.7)
    for h in range(4):
        for i in range(9):
            s = np.exp(0.7 * k[:i + 1, h // 2] @ q[i, h])
            np.testing.assert_allclose(got[i, h], s @ v[:i + 1, h // 2] / s.sum(), atol=1e-12)


def test_oracle_hyper_connections_reduce_to_the_plain_residual():
    rng = np.random.default_rng(2)
    x, y = rng.standard_normal((6, 8)), rng.standard_normal((6, 8))
    for s in (1, 3):
        streams = np.repeat(x[None], s, 0)
        np.testing.assert_allclose(oracle.read_streams(streams, np.full(s, 1 / s)), x)
        np.testing.assert_allclose(oracle.write_streams(streams, y, np.eye(s), np.ones(s)), streams + y)
    mix = rng.standard_normal((3, 3))
    streams = rng.standard_normal((3, 6, 8))
    got = oracle.write_streams(streams, y, mix, [1.0, 0.0, 2.0])
    np.testing.assert_allclose(got[1], mix[0, 1] * streams[0] + mix[1, 1] * streams[1] + mix[2, 1] * streams[2])
    np.testing.assert_allclose(oracle.token_shift(x, np.ones(8))[1:], x[:-1])
    assert np.array_equal(oracle.token_shift(x, np.zeros(8)), x)


@pytest.mark.parametrize("edit", ["position", "shift", "gate1", "gate2", "mix", "read", "write", "decay", "loop", "halves",
                                  "q_norm", "kv_heads", "scale", "out_gate", "eps"])
def test_a_planted_mistake_in_the_oracle_shows(edit, monkeypatch):
    """Every mechanism moves the logits of a small model: an oracle that gets one wrong is told apart."""
    cfg = default_stream_config()
    t = to_oracle(random_checkpoint(cfg))
    toks = np.random.default_rng(0).integers(0, cfg["vocab"], 40).tolist()
    right = oracle.forward(cfg, t, toks)
    bad_cfg, bad = copy.deepcopy(cfg), dict(t)
    if edit == "position":
        monkeypatch.setattr(oracle, "embed", lambda tokens, table: np.asarray(table)[tokens])
    elif edit == "shift":
        bad["l1.shift"] = np.zeros_like(t["l1.shift"])
    elif edit in ("gate1", "gate2"):
        name = f"l1.rg{edit[-1]}"
        bad[name] = np.zeros_like(t[name])
    elif edit == "mix":
        bad["l1.hc1.mix"] = t["l1.hc1.mix"].T
    elif edit == "read":
        bad["l2.hc1.in"] = t["l2.hc1.in"][::-1]
    elif edit == "write":
        bad["l2.hc2.out"] = np.ones_like(t["l2.hc2.out"])
    elif edit == "decay":
        bad_cfg["layers"][2]["mixer"]["decay"][2] = 0.98
    elif edit == "loop":
        bad_cfg["loop"]["times"] = 1
    elif edit == "halves":
        bad["l1.mix.left.out"], bad["l1.mix.right.out"] = t["l1.mix.right.out"], t["l1.mix.left.out"]
    elif edit == "q_norm":
        bad["l1.mix.left.q.norm"] = np.ones_like(t["l1.mix.left.q.norm"])
    elif edit == "kv_heads":
        bad["l1.mix.left.q"] = np.roll(t["l1.mix.left.q"], 24, axis=0)
    elif edit == "scale":
        bad_cfg["layers"][1]["mixer"]["left"]["scale"] = 0.2
    elif edit == "out_gate":
        bad["l3.mix.right.g"] = np.zeros_like(t["l3.mix.right.g"])
    elif edit == "eps":
        bad_cfg["norm"]["eps"] = 1e-1
    err = np.sqrt(((oracle.forward(bad_cfg, bad, toks) - right) ** 2).mean(1)) / right.std()
    assert err[12:].max() > 1e-2, err.max()
