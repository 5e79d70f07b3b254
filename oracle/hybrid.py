"""Plain whole-sequence restatement of a decoder whose layers mix latent attention, Mamba-2 and mLSTM (design
"Mapuvik"): numpy, float64, one function per mechanism, no cache, no batching.  It takes the model folder's
``config.json`` dictionary and a ``{tensor name: array}`` dictionary and returns the logits of every position of one
sequence; a paged, chunked, batched implementation has to agree with it however the sequence was cut.

The recurrences follow the papers' token-by-token forms: Dao and Gu, "Transformers are SSMs: Generalized Models and
Efficient Algorithms Through Structured State Space Duality" (Mamba-2); Beck et al., "xLSTM: Extended Long Short-Term
Memory" (mLSTM); DeepSeek-AI, "DeepSeek-V2: A Strong, Economical, and Efficient Mixture-of-Experts Language Model"
(latent attention).
"""

from __future__ import annotations

import math

import numpy as np

F = np.float64


def linear(x, w):
    """Rows of ``x`` through a weight stored [out, in]."""
    return np.asarray(x, F) @ np.asarray(w, F).T


def sigmoid(z):
    return np.where(z >= 0, 1.0 / (1.0 + np.exp(-np.abs(z))), np.exp(-np.abs(z)) / (1.0 + np.exp(-np.abs(z))))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def log_sigmoid(z):
    return -softplus(-z)


_erf = np.vectorize(math.erf, otypes=[F])


def gelu_erf(z):
    return 0.5 * z * (1.0 + _erf(z / math.sqrt(2.0)))


def over_rms(x, eps):
    """``x`` divided by its root mean square over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def rms_norm_plain(x, w, eps):
    return over_rms(x, eps) * np.asarray(w, F)


def rms_norm_zero_centred(x, w, eps):
    """The stored weight is the distance from one."""
    return over_rms(x, eps) * (1.0 + np.asarray(w, F))


def rotate_interleaved(x, positions, dims, base):
    """``x`` [T, H, D]: the pairs (2i, 2i+1) of the first ``dims`` dimensions turned by ``position * base^(-2i/dims)``."""
    y = np.array(x, F)
    for i in range(dims // 2):
        a = np.asarray(positions, F) * F(base) ** (-2.0 * i / dims)
        c, s = np.cos(a)[:, None], np.sin(a)[:, None]
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        y[:, :, 2 * i], y[:, :, 2 * i + 1] = u * c - v * s, v * c + u * s
    return y


def visible(i, j, window):
    return j <= i and (window is None or i - j < window)


def latent_attention(h, m, p, eps):
    """``m``: the mixer's sizes, ``p``: its tensors, ``h`` [T, width]."""
    t, heads, dn, dr, dv, rank = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = np.arange(t)
    q = linear(h, p["q"]).reshape(t, heads, dn + dr)
    down = linear(h, p["dkv"])
    c = rms_norm_plain(down[:, :rank], p["dkv.norm"], eps)
    rot = m["rot"]
    k_rot = rotate_interleaved(down[:, None, rank:], pos, rot["dims"], rot["base"])[:, 0]
    q_rot = rotate_interleaved(q[:, :, dn:], pos, rot["dims"], rot["base"])
    k = linear(c, p["uk"]).reshape(t, heads, dn)
    v = linear(c, p["uv"]).reshape(t, heads, dv)
    window = (m.get("mask") or {}).get("size")
    out = np.zeros((t, heads, dv), F)
    for i in range(t):
        js = [j for j in range(t) if visible(i, j, window)]
        s = (np.einsum("hd,jhd->hj", q[i, :, :dn], k[js]) + q_rot[i] @ k_rot[js].T) * m["scale"]
        w = np.exp(s - s.max(axis=1, keepdims=True))
        out[i] = np.einsum("hj,jhd->hd", w / w.sum(axis=1, keepdims=True), v[js])
    y = out.reshape(t, heads * dv) * sigmoid(linear(h, p["g"]))
    return linear(y, p["o"])


def causal_conv(x, w, b):
    """Per-channel convolution; ``w`` [channels, taps], the last column meets the current token."""
    w, taps = np.asarray(w, F), w.shape[1]
    padded = np.concatenate([np.zeros((taps - 1, x.shape[1]), F), x])
    y = np.zeros_like(x)
    for k in range(taps):
        y += padded[k:k + x.shape[0]] * w[:, k]
    return y + np.asarray(b, F)


def mamba2_recurrence(x, b, c, dt, a_log, d):
    """``x`` [T, H, V], ``b`` / ``c`` [T, G, N], ``dt`` [T, H] (after softplus): the outputs [T, H, V]."""
    t, heads, vd = x.shape
    groups, n = b.shape[1:]
    y = np.zeros((t, heads, vd), F)
    for h in range(heads):
        g = h // (heads // groups)
        state = np.zeros((n, vd), F)
        rate = math.exp(float(a_log[h]))
        for i in range(t):
            state = math.exp(-rate * dt[i, h]) * state + dt[i, h] * np.outer(b[i, g], x[i, h])
            y[i, h] = state.T @ c[i, g] + float(d[h]) * x[i, h]
    return y


def mamba2(h, m, p, eps):
    t, heads, vd, n, groups = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = heads * vd
    z, xbc, dt = np.split(linear(h, p["in"]), [inner, 2 * inner + 2 * groups * n], axis=1)
    xbc = silu(causal_conv(xbc, p["conv"], p["conv.b"]))
    x, b, c = np.split(xbc, [inner, inner + groups * n], axis=1)
    dt = softplus(dt + np.asarray(p["dt_bias"], F))
    y = mamba2_recurrence(x.reshape(t, heads, vd), b.reshape(t, groups, n), c.reshape(t, groups, n), dt,
                          p["A_log"], p["D"]).reshape(t, inner)
    y = over_rms((y * silu(z)).reshape(t, m["norm_groups"], -1), eps).reshape(t, inner) * np.asarray(p["norm"], F)
    return linear(y, p["o"])


def mlstm_recurrence(q, k, v, log_i, log_f):
    """``q`` / ``k`` [T, H, K] (q already scaled), ``v`` [T, H, V], gates [T, H]: the outputs [T, H, V]."""
    t, heads, vd = v.shape
    y = np.zeros((t, heads, vd), F)
    for h in range(heads):
        s, n, m = np.zeros((q.shape[2], vd), F), np.zeros(q.shape[2], F), 0.0
        for i in range(t):
            new = max(log_f[i, h] + m, log_i[i, h])
            keep, add = math.exp(log_f[i, h] + m - new), math.exp(log_i[i, h] - new)
            s = keep * s + add * np.outer(k[i, h], v[i, h])
            n = keep * n + add * k[i, h]
            m = new
            y[i, h] = s.T @ q[i, h] / (max(abs(float(n @ q[i, h])), math.exp(-m)) + 1e-6)
    return y


def mlstm(h, m, p, eps):
    t, heads, kd, vd, cap = h.shape[0], m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q = linear(h, p["q"]).reshape(t, heads, kd) * kd ** -0.5
    k = linear(h, p["k"]).reshape(t, heads, kd)
    v = linear(h, p["v"]).reshape(t, heads, vd)
    log_i = cap * np.tanh((linear(h, p["i"]) + np.asarray(p["i.b"], F)) / cap)
    log_f = log_sigmoid(cap * np.tanh((linear(h, p["f"]) + np.asarray(p["f.b"], F)) / cap))
    y = over_rms(mlstm_recurrence(q, k, v, log_i, log_f), eps).reshape(t, heads * vd)
    return linear(y * np.asarray(p["norm"], F) * sigmoid(linear(h, p["g"])), p["o"])


MIXERS = {"latent_attention": latent_attention, "mamba2": mamba2, "mlstm": mlstm}


def feed_forward(h, p):
    return linear(gelu_erf(linear(h, p["up"])), p["down"])


def _below(tensors, prefix):
    return {k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)}


def forward(config, tensors, tokens, residuals=None):
    """Logits [T, vocab] of one whole sequence; ``residuals`` (a list) receives the stream after every layer."""
    eps = config["norm"]["eps"]
    x = np.asarray(tensors["embed"], F)[np.asarray(tokens)]
    for i, layer in enumerate(config["layers"]):
        own = f"l{layer.get('weights_of', i)}."
        h = rms_norm_zero_centred(x, tensors[own + "norm1"], eps)
        y = MIXERS[layer["type"]](h, layer["mixer"], _below(tensors, own + "mix."), eps)
        if layer.get("mlp") is not None:
            y = y + feed_forward(h, _below(tensors, own + "mlp."))
        x = x + y
        if residuals is not None:
            residuals.append(x.copy())
    return linear(rms_norm_zero_centred(x, tensors["final.norm"], eps), tensors["head"])
