"""Plain whole-sequence restatement of the "Kerolorn" decoder: sublayers between two norms, a short convolution on the
mixer's input, rotated-then-normed attention over a sliding window with kept first tokens, routed experts beside a gated
shared one.  numpy, float64, one function per mechanism, no cache, no batching: it takes the model folder's
``config.json`` dictionary and a ``{tensor name: array}`` dictionary and returns the logits of every position of one
sequence; a paged, chunked, batched implementation has to agree with it however the sequence was cut.

The frequency scaling follows Peng et al., "YaRN: Efficient Context Window Extension of Large Language Models"."""

from __future__ import annotations

import math

import numpy as np

F = np.float64


def linear(x, w):
    """Rows of ``x`` through a weight stored [out, in]."""
    return np.asarray(x, F) @ np.asarray(w, F).T


def sigmoid(z):
    e = np.exp(-np.abs(z))
    return np.where(z >= 0, 1.0, e) / (1.0 + e)


def silu(z):
    return z * sigmoid(z)


def over_rms(x, eps):
    """``x`` divided by its root mean square over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def rms_norm(x, w, eps):
    return over_rms(x, eps) * np.asarray(w, F)


def input_convolution(h, w):
    """``h`` [T, width] plus its causal per-channel convolution; ``w`` [width, taps], the last column meets the current
    token."""
    w = np.asarray(w, F)
    taps = w.shape[1]
    before = np.concatenate([np.zeros((taps - 1, h.shape[1]), F), h])
    y = np.array(h, F)
    for t in range(h.shape[0]):
        for j in range(taps):
            y[t] += w[:, j] * before[t + j]
    return y


def frequencies(rot):
    """Angle per position of every rotated pair and the factor on cosine and sine."""
    dims, base, scaling = rot["dims"], F(rot["base"]), rot.get("scaling")
    f = [float(base ** (-2.0 * i / dims)) for i in range(dims // 2)]
    if not scaling:
        return np.array(f, F), 1.0

    def turns_at(t):  # the (fractional) index whose pair turns t times over the original length
        return dims * math.log(scaling["original"] / (2.0 * math.pi * t)) / (2.0 * math.log(base))

    lo, hi = max(math.floor(turns_at(scaling["fast"])), 0), min(math.ceil(turns_at(scaling["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / scaling["factor"] * ramp + fi * (1.0 - ramp))
    return np.array(out, F), 0.1 * math.log(scaling["factor"]) + 1.0


def rotate(x, positions, rot):
    """``x`` [T, H, D]: the neighbouring pairs of the first ``dims`` dimensions are turned."""
    y = np.array(x, F)
    if not rot:
        return y
    freq, factor = frequencies(rot)
    for i, f in enumerate(freq):
        a = np.asarray(positions, F) * f
        c, s = (np.cos(a) * factor)[:, None], (np.sin(a) * factor)[:, None]
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        y[:, :, 2 * i], y[:, :, 2 * i + 1] = u * c - v * s, v * c + u * s
    return y


def visible(i, j, mask):
    """Whether position ``i`` sees position ``j`` (numbers or arrays)."""
    size = (mask or {}).get("size")
    if not size:
        return j <= i
    return (j <= i) & ((i - j < size) | (j < (mask.get("keep_first") or 0)))


def softmax_attention(q, k, v, scale, mask):
    """``q`` [T, H, D], ``k`` [T, G, D], ``v`` [T, G, V], ``scale`` [H]: [T, H, V]."""
    t, heads, _ = q.shape
    per = heads // k.shape[1]
    seen = visible(np.arange(t)[:, None], np.arange(t), mask)
    out = np.zeros((t, heads, v.shape[2]), F)
    for h in range(heads):
        s = np.where(seen, q[:, h] @ k[:, h // per].T * scale[h], -np.inf)
        w = np.exp(s - s.max(axis=1, keepdims=True))
        out[:, h] = w / w.sum(axis=1, keepdims=True) @ v[:, h // per]
    return out


def attention_mixer(h, m, p, eps):
    t, heads, groups, dim, vdim = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos, rot = np.arange(t), m.get("rot")
    q = over_rms(rotate(linear(h, p["q"]).reshape(t, heads, dim), pos, rot), eps)
    k = over_rms(rotate(linear(h, p["k"]).reshape(t, groups, dim), pos, rot), eps)
    v = linear(h, p["v"]).reshape(t, groups, vdim)
    scale = m["scale"] * np.asarray(p["temp"], F)
    return linear(softmax_attention(q, k, v, scale, m.get("mask")).reshape(t, heads * vdim), p["o"])


def gated_unit(h, p):
    return linear(silu(linear(h, p["gate"])) * linear(h, p["up"]), p["down"])


def route(z, correction, top, scale):
    """Logits [T, E]: the chosen experts [T, top], best first, and their weights."""
    e = np.exp(z - z.max(axis=1, keepdims=True))
    s = e / e.sum(axis=1, keepdims=True)
    chosen = np.argsort(-(s + np.asarray(correction, F)), axis=1, kind="stable")[:, :top]
    return chosen, np.take_along_axis(s, chosen, axis=1) * scale


def routed_experts(h, m, p):
    chosen, weights = route(linear_exact(h, p["router"]), p["correction"], m["router"]["top"], m["router"]["scale"])
    y = np.zeros_like(h)
    for e in range(m["router"]["experts"]):
        rows, places = np.nonzero(chosen == e)
        if len(rows):
            y[rows] += weights[rows, places][:, None] * gated_unit(h[rows], below(p, f"e{e}."))
    if m.get("shared"):
        y = y + sigmoid(linear_exact(h, p["shared.sg"])) * gated_unit(h, below(p, "shared."))
    return y


def linear_exact(x, w):
    """As ``linear``; products that a 16-bit run computes in 32 bits go through here."""
    return np.asarray(x, F) @ np.asarray(w, F).T


def below(tensors, prefix):
    return {k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)}


def run_layer(x, layer, p, eps):
    h = input_convolution(rms_norm(x, p["norm1"], eps), p["canon1"])
    x = x + rms_norm(attention_mixer(h, layer["mixer"], below(p, "mix."), eps), p["norm1b"], eps)
    if layer.get("mlp") is None:
        return x
    return x + rms_norm(routed_experts(rms_norm(x, p["norm2"], eps), layer["mlp"], below(p, "mlp.")), p["norm2b"], eps)


def forward(config, tensors, tokens, residuals=None):
    """Logits [T, vocab] of one whole sequence; ``residuals`` (a list) receives the stream after every layer."""
    eps = config["norm"]["eps"]
    x = np.asarray(tensors["embed"], F)[np.asarray(tokens)]
    for i, layer in enumerate(config["layers"]):
        x = run_layer(x, layer, below(tensors, f"l{i}."), eps)
        if residuals is not None:
            residuals.append(x.copy())
    return linear(rms_norm(x, tensors["final.norm"], eps), tensors["head"]) * config["logit_scale"]
