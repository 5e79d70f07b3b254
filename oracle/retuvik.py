"""Plain whole-sequence restatement of the "Retuvik" decoder: pre-norm sublayers with grouped norms, RWKV-style time mixing
(a matrix state whose decay is a function of the input, per head and key channel) or windowed attention with a distance bias,
dense xIELU or routed feed-forwards, and a stretch of layers that runs several times.  numpy, float64, one function per
mechanism, no cache, no batching: it takes the model folder's ``config.json`` dictionary and a ``{tensor name: array}``
dictionary and returns the logits of every position of one sequence; a paged, chunked, batched implementation has to agree
with it however the sequence was cut."""

from __future__ import annotations

import numpy as np

F = np.float64


def linear(x, w):
    """Rows of ``x`` through a weight stored [out, in]."""
    return np.asarray(x, F) @ np.asarray(w, F).T


def linear_exact(x, w):
    """As ``linear``; products that a 16-bit run computes in 32 bits go through here."""
    return np.asarray(x, F) @ np.asarray(w, F).T


def sigmoid(z):
    e = np.exp(-np.abs(z))
    return np.where(z >= 0, 1.0, e) / (1.0 + e)


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def over_rms(x, eps):
    """``x`` divided by its root mean square over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def grouped_norm(x, w, groups, eps):
    """Every one of ``groups`` equal parts of a row over its own root mean square, times ``w``."""
    parts = over_rms(x.reshape(x.shape[0], groups, -1), eps)
    return parts.reshape(x.shape) * np.asarray(w, F)


def before(h):
    """The row before, zeros ahead of the first."""
    return np.concatenate([np.zeros_like(h[:1]), h[:-1]])


def token_mix(h, mu):
    return h + (before(h) - h) * np.asarray(mu, F)


def wkv(r, k, v, w, u):
    """``r``, ``k``, ``w`` [T, H, K], ``v`` [T, H, V], ``u`` [H, K]: [T, H, V]."""
    t, heads, dim = r.shape
    s = np.zeros((heads, dim, v.shape[2]), F)
    out = np.zeros_like(v)
    for i in range(t):
        new = k[i][:, :, None] * v[i][:, None, :]
        out[i] = np.einsum("hkv,hk->hv", s + u[:, :, None] * new, r[i])
        s = w[i][:, :, None] * s + new
    return out


def decay(mix, p):
    return np.exp(-np.exp(linear_exact(np.tanh(linear(mix, p["w1"])), p["w2"]) + np.asarray(p["w0"], F)))


def wkv_mixer(h, m, p, eps):
    t, heads, dim = h.shape[0], m["heads"], m["dim"]
    r, k, v = (linear(token_mix(h, p[f"mu.{s}"]), p[s]).reshape(t, heads, dim) for s in "rkv")
    gate = silu(linear(token_mix(h, p["mu.g"]), p["g"]))
    w = decay(token_mix(h, p["mu.w"]), p).reshape(t, heads, dim)
    o = over_rms(wkv(r, k, v, w, np.asarray(p["u"], F)), eps).reshape(t, heads * dim)
    return linear(o * np.asarray(p["norm"], F) * gate, p["o"])


def visible(i, j, mask):
    """Whether position ``i`` sees position ``j`` (numbers or arrays)."""
    size = (mask or {}).get("size")
    return (j <= i) & (i - j < size) if size else j <= i


def slopes(heads):
    return np.array([2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)], F)


def temperature(positions, q_temp):
    """The factor on the queries at ``positions``."""
    p = np.asarray(positions, F)
    if not q_temp:
        return np.ones_like(p)
    return 1.0 + q_temp["coef"] * np.log(np.floor((p + 1.0) / q_temp["every"]) + 1.0)


def biased_attention(q, k, v, scale, slope, mask):
    """``q`` [T, H, D], ``k`` [T, G, D], ``v`` [T, G, V], ``slope`` [H]: [T, H, V]."""
    t, heads, _ = q.shape
    per = heads // k.shape[1]
    i, j = np.arange(t)[:, None], np.arange(t)
    seen = visible(i, j, mask)
    out = np.zeros((t, heads, v.shape[2]), F)
    for h in range(heads):
        s = np.where(seen, q[:, h] @ k[:, h // per].T * scale - slope[h] * (i - j), -np.inf)
        w = np.exp(s - s.max(axis=1, keepdims=True))
        out[:, h] = w / w.sum(axis=1, keepdims=True) @ v[:, h // per]
    return out


def attention_mixer(h, m, p, eps):
    t, heads, groups, dim, vdim = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = over_rms(linear(h, p["q"]).reshape(t, heads, dim), eps) * np.asarray(p["q.norm"], F)
    q = q * temperature(np.arange(t), m.get("q_temp"))[:, None, None]
    k = over_rms(linear(h, p["k"]).reshape(t, groups, dim), eps) * np.asarray(p["k.norm"], F)
    v = over_rms(linear(h, p["v"]).reshape(t, groups, vdim), eps)
    o = biased_attention(q, k, v, m["scale"], slopes(heads), m.get("mask")).reshape(t, heads * vdim)
    return linear(o * sigmoid(linear(h, p["g"])), p["o"])


def xielu(z, act):
    p, q = (softplus(F(a)) for a in np.asarray(act, F))
    low = np.minimum(z, 0.0)
    return np.where(z > 0, p * z * z, (0.5 + q) * (np.expm1(low) - low)) + 0.5 * z


def dense(h, p):
    a = xielu(linear(h, p["up"]) + np.asarray(p["up.b"], F), p["act"])
    return linear(a, p["down"]) + np.asarray(p["down.b"], F)


def route(z, top):
    """Logits [T, E]: the ``top`` largest, best first, and the softmax over them alone."""
    chosen = np.argsort(-z, axis=1, kind="stable")[:, :top]
    c = np.take_along_axis(z, chosen, axis=1)
    w = np.exp(c - c.max(axis=1, keepdims=True))
    return chosen, w / w.sum(axis=1, keepdims=True)


def routed_experts(h, m, p):
    chosen, weights = route(linear_exact(h, p["router"]) + np.asarray(p["router.b"], F), m["router"]["top"])
    y = np.zeros_like(h)
    for e in range(m["router"]["experts"]):
        rows, places = np.nonzero(chosen == e)
        if len(rows):
            q = below(p, f"e{e}.")
            unit = linear(silu(linear(h[rows], q["gate"])) * linear(h[rows], q["up"]), q["down"])
            y[rows] += weights[rows, places][:, None] * unit
    return y


def below(tensors, prefix):
    return {k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)}


def run_layer(x, layer, p, groups, eps):
    mixer = {"wkv": wkv_mixer, "attention": attention_mixer}[layer["type"]]
    x = x + mixer(grouped_norm(x, p["norm1"], groups, eps), layer["mixer"], below(p, "mix."), eps)
    mlp = layer.get("mlp")
    if mlp is None:
        return x
    h, q = grouped_norm(x, p["norm2"], groups, eps), below(p, "mlp.")
    return x + (routed_experts(h, mlp, q) if mlp["kind"] == "moe" else dense(h, q))


def order(config):
    """The layers as they run: (number, pass) -- the pass where a layer is the first of one, else None."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop or loop["start"] == loop["stop"]:
        return [(i, None) for i in range(n)]
    start, stop, times = loop["start"], loop["stop"], loop["times"]
    runs = [(i, None) for i in range(start)]
    for t in range(times):
        runs += [(i, t if i == start else None) for i in range(start, stop)]
    return runs + [(i, None) for i in range(stop, n)]


def forward(config, tensors, tokens, residuals=None):
    """Logits [T, vocab] of one whole sequence; ``residuals`` (a list) receives the stream after every layer run."""
    eps, groups = config["norm"]["eps"], config["norm"]["groups"]
    first = np.asarray(tensors["embed"], F)[np.asarray(tokens)] * config["embedding"]["scale"]
    x = first
    for i, number in order(config):
        if number is not None:
            if number > 0:
                x = x + first
            x = x + np.asarray(tensors["loop.step"], F)[number]
        x = run_layer(x, config["layers"][i], below(tensors, f"l{i}."), groups, eps)
        if residuals is not None:
            residuals.append(x.copy())
    return linear(grouped_norm(x, tensors["final.norm"], groups, eps), tensors["head"])
