"""Gated linear recurrences and the short convolution on the device against the token-by-token oracle: both forms
(sequential, chunked), portions, slots that are used again, odd sizes."""

from __future__ import annotations

import numpy as np
import pytest
import torch

from oracle import hybrid as oracle

from .hybrid_helpers import segments

pytestmark = pytest.mark.gpu

TOL = {torch.float32: 2e-5, torch.bfloat16: 6e-3}  # of the outputs' largest magnitude; bf16: one rounding at the end


def close(got: torch.Tensor, want: np.ndarray, tol: float) -> None:
    err = np.abs(got.double().cpu().numpy() - want).max()
    assert err <= tol * max(1.0, np.abs(want).max()), (err, np.abs(want).max())


class Case:
    """Random operands of one long sequence per request and the oracle's outputs for all of it."""

    def __init__(self, kind, heads, groups, k, v, lens, dtype, seed=0, decay=1.0):
        rng = np.random.default_rng(seed)
        self.kind, self.heads, self.groups, self.k, self.v, self.lens, self.dtype = kind, heads, groups, k, v, lens, dtype
        self.taken = [0] * len(lens)
        r = lambda *s: torch.from_numpy(rng.standard_normal(s)).to(dtype)  # noqa: E731
        f = lambda *s: torch.from_numpy(rng.standard_normal(s)).float().cuda()  # noqa: E731
        self.rows = [{"q": r(n, groups, k), "k": r(n, groups, k), "v": r(n, heads, v), "a": 2 * r(n, heads),
                      "b": 2 * r(n, heads) + 2} for n in lens]
        self.bias_a, self.bias_b = f(heads), f(heads)
        self.rate, self.skip = decay * f(heads).exp(), f(heads)
        self.cap, self.q_scale = 5.0, (k ** -0.5 if kind == "mlstm" else 1.0)
        tiles = -(-v // 64)
        n = len(lens) + 2
        self.state = torch.full((n, heads, k, v), float("nan"), device="cuda")  # a fresh request must not read it
        self.norm = torch.full((n, heads, tiles, k), float("nan"), device="cuda")
        self.max = torch.full((n, heads, tiles), float("nan"), device="cuda")
        self.want = [self._oracle(x) for x in self.rows]

    def _oracle(self, x):
        d = {name: t.double().numpy() for name, t in x.items()}
        ba, bb = self.bias_a.double().cpu().numpy(), self.bias_b.double().cpu().numpy()
        if self.kind == "ssd":
            return oracle.mamba2_recurrence(d["v"], d["k"], d["q"], oracle.softplus(d["a"] + ba),
                                            np.log(self.rate.double().cpu().numpy()), self.skip.double().cpu().numpy())
        li = self.cap * np.tanh((d["a"] + ba) / self.cap)
        lf = oracle.log_sigmoid(self.cap * np.tanh((d["b"] + bb) / self.cap))
        return oracle.mlstm_recurrence(d["q"] * self.q_scale, d["k"], d["v"], li, lf)

    def step(self, ops, portions: dict[int, int], slots: dict[int, int], **kw):
        """The next ``portions[i]`` rows of requests ``i`` as one batch."""
        ids = list(portions)
        part = [{n: t[self.taken[i]:self.taken[i] + portions[i]] for n, t in self.rows[i].items()} for i in ids]
        for i in ids:
            self.taken[i] += portions[i]
        meta = segments([portions[i] for i in ids], [self.taken[i] for i in ids], [slots[i] for i in ids])
        cat = lambda n: torch.cat([p[n].reshape(p[n].shape[0], -1) for p in part]).cuda()  # noqa: E731
        gates = torch.cat([cat("a"), cat("b")], 1)
        a, b = gates.split(self.heads, 1)
        m = self.kind == "mlstm"
        out = ops.recurrence(self.kind, cat("q"), cat("k"), cat("v"), a, b if m else None, meta, self.state,
                             heads=self.heads, groups=self.groups, key_dim=self.k, value_dim=self.v, bias_a=self.bias_a,
                             bias_b=self.bias_b if m else None, rate=None if m else self.rate,
                             skip=None if m else self.skip, norm_state=self.norm if m else None,
                             max_state=self.max if m else None, q_scale=self.q_scale, gate_cap=self.cap if m else 0.0, **kw)
        want = np.concatenate([self.want[i][self.taken[i] - portions[i]:self.taken[i]] for i in ids])
        close(out, want.reshape(len(out), -1), TOL[self.dtype])


SHAPES = [("ssd", 6, 3, 24, 16), ("ssd", 4, 1, 128, 64), ("ssd", 2, 2, 72, 136), ("mlstm", 3, 3, 40, 24),
          ("mlstm", 2, 2, 128, 200), ("ssd", 4, 2, 64, 64), ("mlstm", 2, 2, 192, 72), ("mlstm", 1, 1, 256, 64),
          ("ssd", 1, 1, 320, 8), ("ssd", 3, 3, 5, 7), ("mlstm", 1, 1, 9, 65)]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("kind,heads,groups,k,v", SHAPES)
def test_whole_sequences_portions_and_single_rows_agree_with_the_oracle(ops, kind, heads, groups, k, v, dtype):
    c = Case(kind, heads, groups, k, v, [300, 231, 70, 3], dtype)
    slots = {0: 4, 1: 2, 2: 1, 3: 3}
    c.step(ops, {0: 230, 1: 1, 2: 64, 3: 2}, slots)      # chunk edges, a fresh single row, a portion of two
    c.step(ops, {2: 1, 0: 1, 1: 165}, slots)
    c.step(ops, {3: 1, 1: 5, 0: 4, 2: 5}, slots)          # on both sides of the token-by-token limit
    c.step(ops, {0: 65, 1: 60}, slots)


@pytest.mark.parametrize("kind,heads,groups,k,v", SHAPES[:9])
@pytest.mark.parametrize("chunk", [64, 128])
def test_chunked_and_sequential_forms_leave_the_same_state(ops, kind, heads, groups, k, v, chunk):
    if chunk == 128 and k % 64:
        pytest.skip("the tcgen05 form takes whole 64-wide slices of the key")
    a, b = (Case(kind, heads, groups, k, v, [390], torch.bfloat16) for _ in range(2))
    for n in (350, 40):
        a.step(ops, {0: n}, {0: 1}, chunk=chunk)
        b.step(ops, {0: n}, {0: 1}, force_sequential=True)
    torch.testing.assert_close(a.state[1], b.state[1], rtol=2e-4, atol=2e-5 * float(b.state[1].abs().max()))
    if kind == "mlstm":
        torch.testing.assert_close(a.norm[1], b.norm[1], rtol=2e-4, atol=2e-5 * float(b.norm[1].abs().max()))
        torch.testing.assert_close(a.max[1], b.max[1], rtol=1e-4, atol=1e-3)
    assert not ops.recurrence_failed()


@pytest.mark.parametrize("kind", ["ssd", "mlstm"])
def test_a_slot_that_changes_hands_starts_from_zero(ops, kind):
    c = Case(kind, 2, 2, 32, 64, [80, 80, 80], torch.bfloat16)
    c.step(ops, {0: 80}, {0: 1})
    c.step(ops, {1: 80}, {1: 1})   # the same slot, now another request: a chunked start
    c.step(ops, {2: 1}, {2: 1})    # and a single-row start
    c.step(ops, {2: 79}, {2: 1})


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_slow_decay_keeps_a_far_token_and_fast_decay_drops_it(ops, dtype):
    for decay in (1e-4, 30.0):
        c = Case("ssd", 2, 1, 16, 32, [400], dtype, decay=decay)
        for n in (257, 1, 2, 140):
            c.step(ops, {0: n}, {0: 1})


def test_mlstm_with_gates_at_their_caps(ops):
    c = Case("mlstm", 2, 2, 16, 16, [150], torch.float32)
    for x in c.rows:
        x["a"] = torch.sign(x["a"]) * 60
        x["b"] = torch.sign(x["b"]) * 60
    c.want = [c._oracle(x) for x in c.rows]
    for n in (100, 1, 49):
        c.step(ops, {0: n}, {0: 1})


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 7])
def test_causal_conv(ops, taps, dtype):
    ch, lens = 150, [50, 33, 9]
    rng = np.random.default_rng(taps)
    x = [torch.from_numpy(rng.standard_normal((n, ch))).to(dtype) for n in lens]
    w, b = rng.standard_normal((ch, taps)).astype(np.float32), rng.standard_normal(ch).astype(np.float32)
    want = [oracle.silu(oracle.causal_conv(t.double().numpy(), w, b)) for t in x]
    wt, bt = torch.from_numpy(w.T.copy()).cuda(), torch.from_numpy(b).cuda()
    state = torch.full((5, taps - 1, ch), float("nan"), dtype=dtype, device="cuda")
    taken, slots = [0, 0, 0], [2, 4, 1]
    for portions in ({0: 17, 1: 1, 2: 2}, {2: 1, 0: 1, 1: 2}, {1: 30, 0: 32, 2: 6}):
        ids = list(portions)
        for i in ids:
            taken[i] += portions[i]
        meta = segments([portions[i] for i in ids], [taken[i] for i in ids], [slots[i] for i in ids])
        rows = torch.cat([x[i][taken[i] - portions[i]:taken[i]] for i in ids]).cuda()
        wide = torch.zeros((len(rows), ch + 9), dtype=dtype, device="cuda")
        wide[:, 9:] = rows
        got = ops.causal_conv(wide[:, 9:], wt, bt, state, meta)
        close(got, np.concatenate([want[i][taken[i] - portions[i]:taken[i]] for i in ids]), TOL[dtype])
