"""The kernels of the pre-norm decoders one by one against the oracle: the step between sublayers with its mixes, the recurrence
with decays per key channel, normed heads and values, attention with a distance bias, activations and gates, routing."""

from __future__ import annotations

import numpy as np
import pytest
import torch

from oracle import retuvik as oracle

from .hybrid_helpers import segments

pytestmark = pytest.mark.gpu

BOTH = pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])


def f32(a) -> torch.Tensor:
    return torch.from_numpy(np.ascontiguousarray(a)).float().cuda()


def d(x: torch.Tensor) -> np.ndarray:
    return x.double().cpu().numpy()


def close(got: torch.Tensor, want: np.ndarray, tol: float) -> None:
    err = np.abs(d(got) - want).max()
    assert err <= tol * max(1.0, np.abs(want).max()), (err, np.abs(want).max())


# -- the step between two sublayers --------------------------------------------------------------------------------

@BOTH
@pytest.mark.parametrize("dim,groups,parts", [(88, 4, 3), (256, 4, 8), (96, 3, 1), (1000, 1, 2), (30, 5, 2), (4096, 8, 8), (37, 1, 5),
                                              (2560, 640, 6), (5000, 10, 2), (8196, 3, 4), (6, 6, 1), (2048, 2, 2)])
def test_residual_step_adds_what_it_is_given(ops, dim, groups, parts, dtype):
    rng = np.random.default_rng(dim)
    t, eps, vocab = 7, 1e-3, 11
    x = rng.standard_normal((t, dim)).astype(np.float32)
    op = lambda rows, scale: torch.from_numpy(scale * rng.standard_normal((rows, dim))).to(dtype).cuda()  # noqa: E731
    y, ys, table = op(t, 3.0), op(t * parts, 0.5), op(vocab, 1.0)
    weights = f32(rng.random((t, parts)))
    bias, add, norm = f32(rng.standard_normal(dim)), f32(rng.standard_normal(dim)), f32(rng.standard_normal(dim))
    ids = torch.tensor([0, 10, 3, 3, 5, 9, 1], dtype=torch.int32, device="cuda")
    rows_of = 2.5 * d(table)[ids.cpu().numpy()]
    tol = 2e-5 if dtype == torch.float32 else 8e-3
    mixed = np.einsum("tp,tpd->td", d(weights), d(ys).reshape(t, parts, dim))
    embed = (ids, table, 2.5, False)
    for result, r in ((None, 0), ({"y": y}, d(y)), ({"y": y, "bias": bias}, d(y) + d(bias)),
                      ({"y": ys, "part_weight": weights}, mixed)):
        for more, m in (({}, 0), ({"embed": embed}, rows_of), ({"embed": embed, "add": add}, rows_of + d(add)), ({"add": add}, d(add))):
            want = x + r + m
            h_want = oracle.grouped_norm(want, d(norm), groups, eps)
            kw = dict(eps=eps, dtype=dtype, groups=groups, **more)
            s = f32(x)
            close(ops.residual_step(s, result, norm, **kw), h_want, tol)
            close(s, want, 2e-5)
            s = f32(x)
            wide = ops.residual_step(s, result, norm, wide=True, **kw)
            assert wide.dtype == torch.float32
            close(wide, h_want, 2e-5)
            if not more:
                rows = torch.tensor([5, 0, 5], device="cuda")
                s = f32(x)
                close(ops.residual_step(s, result, norm, rows=rows, **kw), h_want[[5, 0, 5]], tol)
                assert np.array_equal(s.cpu().numpy(), x)
            if result is not None or more:
                s = f32(x)
                assert ops.residual_step(s, result, **{**kw, "groups": 1}) is None
                close(s, want, 2e-5)
    # a fresh stream begins with the embedding, whatever the memory held
    s = torch.full((t, dim), float("nan"), device="cuda")
    close(ops.residual_step(s, None, norm, eps=eps, dtype=dtype, groups=groups, embed=(ids, table, 2.5, True), add=add),
          oracle.grouped_norm(rows_of + d(add), d(norm), groups, eps), tol)
    close(s, rows_of + d(add), 2e-5)


def test_residual_step_refuses_what_does_not_fit(ops):
    x, w = torch.zeros((2, 24), device="cuda"), torch.ones(24, device="cuda")
    kw = dict(eps=1e-6, dtype=torch.float32)
    with pytest.raises(ValueError, match="groups"):
        ops.residual_step(x, None, w, groups=5, **kw)
    with pytest.raises(ValueError, match="embed"):
        ops.residual_step(x, None, w, embed=(torch.zeros(2, dtype=torch.int32, device="cuda"), torch.zeros((4, 16), device="cuda"), 1.0,
                                             False), **kw)
    with pytest.raises(ValueError, match="one row per request"):
        ops.residual_step(x, None, w, mix=(torch.ones((5, 24), device="cuda"), torch.zeros((3, 24), device="cuda")),
                          seg=segments([2], [2]), **kw)


@BOTH
@pytest.mark.parametrize("dim,mixes,groups", [(88, 5, 4), (37, 5, 1), (1040, 5, 5), (64, 1, 2), (24, 8, 3), (2048, 5, 4)])
def test_mixes_in_the_step_and_over_portions(ops, dim, mixes, groups, dtype):
    """Portions go through a kernel of their own, batches of single rows through the step itself; both keep the last row in the
    request's slot, which starts out as somebody else's."""
    rng = np.random.default_rng(3)
    mu, norm = f32(rng.random((mixes, dim))), f32(rng.standard_normal(dim))
    lens = [60, 33, 9]
    x = [rng.standard_normal((n, dim)).astype(np.float32) for n in lens]
    hs = [oracle.grouped_norm(a.astype(np.float64), d(norm), groups, 1e-6) for a in x]
    want = [np.stack([oracle.token_mix(h, m) for m in d(mu)]) for h in hs]
    state = torch.full((5, dim), float("nan"), device="cuda")
    taken, slots = [0, 0, 0], [2, 4, 1]
    kw = dict(eps=1e-6, dtype=dtype, groups=groups)
    for portions in ({0: 17, 1: 1, 2: 2}, {2: 1, 0: 1, 1: 1}, {1: 1}, {1: 29, 0: 2, 2: 5}, {0: 1, 2: 1}, {0: 38, 1: 1}):
        ids = list(portions)
        for i in ids:
            taken[i] += portions[i]
        seg = segments([portions[i] for i in ids], [taken[i] for i in ids], [slots[i] for i in ids])
        part = np.concatenate([x[i][taken[i] - portions[i]:taken[i]] for i in ids])
        if seg.max_q_len == 1:
            got = ops.residual_step(f32(part), None, norm, mix=(mu, state), seg=seg, **kw)
        else:
            got = ops.token_mix(ops.residual_step(f32(part), None, norm, wide=True, **kw), mu, state, seg, dtype)
        assert got.shape == (mixes, len(part), dim) and got.dtype == dtype
        close(got, np.concatenate([want[i][:, taken[i] - portions[i]:taken[i]] for i in ids], axis=1),
              1e-5 if dtype == torch.float32 else 5e-3)
        for i in ids:
            close(state[slots[i]], hs[i][taken[i] - 1], 1e-5)  # in 32 bits whatever the type


# -- the recurrence ----------------------------------------------------------------------------------------------

class Case:
    """Random operands of one long sequence per request and the oracle's outputs for all of it; ``z`` + bias = ln(-ln decay)."""

    def __init__(self, heads, dim, lens, dtype, seed=0, value_dim=None, level=-2.0, spread=1.5):
        rng = np.random.default_rng(seed)
        self.heads, self.dim, self.vdim, self.dtype, self.taken = heads, dim, value_dim or dim, dtype, [0] * len(lens)
        r = lambda *s: torch.from_numpy(rng.standard_normal(s)).to(dtype)  # noqa: E731
        self.rows = [{"q": r(n, heads, dim), "k": r(n, heads, dim), "v": r(n, heads, self.vdim),
                      "z": torch.from_numpy(level + spread * rng.standard_normal((n, heads, dim))).float()} for n in lens]
        self.bias, self.bonus = f32(0.3 * rng.standard_normal((heads, dim))), f32(rng.standard_normal((heads, dim)))
        self.state = torch.full((len(lens) + 2, heads, dim, self.vdim), float("nan"), device="cuda")  # a fresh request must not read it
        self.answer()

    def answer(self):
        self.want = []
        for x in self.rows:
            q, k, v, z = (x[n].double().numpy() for n in "qkvz")
            self.want.append(oracle.wkv(q, k, v, np.exp(-np.exp(z + d(self.bias))), d(self.bonus)))

    def step(self, ops, portions: dict[int, int], slots: dict[int, int], **kw):
        """The next ``portions[i]`` rows of requests ``i`` as one batch."""
        ids = list(portions)
        part = [{n: t[self.taken[i]:self.taken[i] + portions[i]] for n, t in self.rows[i].items()} for i in ids]
        for i in ids:
            self.taken[i] += portions[i]
        meta = segments([portions[i] for i in ids], [self.taken[i] for i in ids], [slots[i] for i in ids])
        cat = lambda n: torch.cat([p[n].reshape(p[n].shape[0], -1) for p in part]).cuda()  # noqa: E731
        out = ops.recurrence("wkv", cat("q"), cat("k"), cat("v"), cat("z"), None, meta, self.state, heads=self.heads, groups=self.heads,
                             key_dim=self.dim, value_dim=self.vdim, bias_a=self.bias, skip=self.bonus, **kw)
        want = np.concatenate([self.want[i][self.taken[i] - portions[i]:self.taken[i]] for i in ids])
        close(out, want.reshape(len(out), -1), 2e-5 if self.dtype == torch.float32 else 6e-3)
        return out


SHAPES = [(6, 24, None), (2, 64, None), (1, 128, None), (3, 5, None), (2, 200, None), (1, 72, 136), (4, 32, 8), (1, 64, 1), (1, 8, 200), (1, 1, 1)]


@BOTH
@pytest.mark.parametrize("heads,dim,vdim", SHAPES)
def test_recurrence_whole_sequences_portions_and_single_rows(ops, heads, dim, vdim, dtype):
    c = Case(heads, dim, [300, 231, 70, 3], dtype, value_dim=vdim)
    slots = {0: 4, 1: 2, 2: 1, 3: 3}
    c.step(ops, {0: 230, 1: 1, 2: 64, 3: 2}, slots)      # chunk edges, a fresh single row, a portion of two
    c.step(ops, {2: 1, 0: 1, 1: 165}, slots)
    c.step(ops, {3: 1, 1: 5, 0: 4, 2: 5}, slots)          # on both sides of the token-by-token limit
    c.step(ops, {0: 65, 1: 60}, slots)


@pytest.mark.parametrize("heads,dim,vdim", [s for s in SHAPES if s[1] % 8 == 0 and (s[2] or 8) % 8 == 0])
@pytest.mark.parametrize("level,spread", [(-2.0, 1.5), (-9.0, 0.5), (1.0, 2.0), (0.0, 4.0)])
def test_chunked_and_sequential_forms_leave_the_same_state(ops, heads, dim, vdim, level, spread):
    """Weak, strong and mixed decays: down to channels that forget within a row beside such that never do."""
    a, b = (Case(heads, dim, [390], torch.bfloat16, value_dim=vdim, level=level, spread=spread) for _ in range(2))
    for n in (350, 40):
        x, y = a.step(ops, {0: n}, {0: 1}), b.step(ops, {0: n}, {0: 1}, force_sequential=True)
        torch.testing.assert_close(x.float(), y.float(), rtol=1e-2, atol=1e-4 * float(y.float().abs().max()))
    torch.testing.assert_close(a.state[1], b.state[1], rtol=2e-4, atol=2e-5 * float(b.state[1].abs().max()))


@BOTH
def test_recurrence_with_decays_at_their_ends(ops, dtype):
    """exp(-exp(z)) from exactly 0 (exp(z) beyond every number) to exactly 1, row by row and channel by channel."""
    c = Case(2, 32, [200], dtype)
    z = c.rows[0]["z"]
    rng = np.random.default_rng(5)
    z[:] = torch.from_numpy(rng.choice([-200.0, -3.0, 0.0, 5.0, 200.0], z.shape, p=[0.6, 0.2, 0.1, 0.05, 0.05])).float()
    with np.errstate(over="ignore"):
        c.answer()
    for n in (130, 1, 3, 66):
        c.step(ops, {0: n}, {0: 1})


@BOTH
@pytest.mark.parametrize("at", [0, 1, 15, 16, 63, 64, 200])
def test_a_far_row_stays_and_counts_from_the_row_after_it(ops, dtype, at):
    """All keys but one are small and nothing decays: what that row wrote shows in every later row -- in its own through the
    bonus -- and in no earlier one."""
    c = Case(2, 16, [260], dtype, level=-30.0, spread=0.0)
    c.bonus.fill_(0.25)
    for x in c.rows:
        x["k"] *= 1e-3
        x["q"][:], x["k"][at], x["v"][at] = 1.0, 4.0, 4.0
    c.answer()
    for portions in ([260], [at + 1] + [1] * 3 + [2, 37], [at] * (at > 0) + [1, 1, 100]):
        c.taken, i = [0], 0
        while c.taken[0] < 260:
            n = min(portions[min(i, len(portions) - 1)], 260 - c.taken[0])
            out = c.step(ops, {0: n}, {0: 1})
            first = c.taken[0] - n
            for r in range(n):
                level = float(out[r].float().abs().mean())
                assert (level < 2) if first + r < at else (level > 30 if first + r == at else level > 150), (first + r, level)
            i += 1


def test_a_slot_that_changes_hands_starts_from_zero(ops):
    c = Case(2, 32, [80, 80, 80], torch.bfloat16)
    c.step(ops, {0: 80}, {0: 1})
    c.step(ops, {1: 80}, {1: 1})   # the same slot, now another request: a chunked start
    c.step(ops, {2: 1}, {2: 1})    # and a single-row start
    c.step(ops, {2: 79}, {2: 1})


def test_recurrence_refuses_what_does_not_fit(ops):
    c = Case(2, 16, [8], torch.bfloat16)
    c.rows[0]["z"] = c.rows[0]["z"].bfloat16()
    with pytest.raises(ValueError, match="gate_a"):
        c.step(ops, {0: 8}, {0: 1})
    c.taken, c.rows[0]["z"] = [0], torch.zeros(8, 2, 8)
    with pytest.raises(ValueError, match="gates must be"):
        c.step(ops, {0: 8}, {0: 1})


# -- gates and activations -----------------------------------------------------------------------------------------

@BOTH
@pytest.mark.parametrize("heads,dim,ff", [(4, 64, 384), (3, 24, 19), (2, 40, 1000), (1, 5, 7), (2, 1024, 4096)])
def test_head_norm_silu_gate_and_activations(ops, heads, dim, ff, dtype):
    rng = np.random.default_rng(ff)
    t, inner = 6, heads * dim
    r = lambda *s: torch.from_numpy(2 * rng.standard_normal(s)).to(dtype).cuda()  # noqa: E731
    y, g, z, w = r(t, inner), r(t, inner), r(t, ff), f32(rng.standard_normal(inner))
    tol = 1e-5 if dtype == torch.float32 else 8e-3
    cols = -(-inner // 8) * 8
    out = torch.full((t, cols), float("nan"), dtype=dtype, device="cuda")
    ops.mixer_finish(out, inner, y=y, post_gate=g, weight=w, group_size=dim, eps=1e-3, post="silu")
    normed = oracle.grouped_norm(d(y), d(w), heads, 1e-3)
    close(out[:, :inner], normed * oracle.silu(d(g)), tol)
    assert (out[:, inner:] == 0).all()
    ops.mixer_finish(out, inner, y=y, post_gate=g, weight=w, group_size=dim, eps=1e-3)
    close(out[:, :inner], normed * oracle.sigmoid(d(g)), tol)
    out[:, :inner] = y
    ops.mixer_finish(out, inner, y=out[:, :inner], post_gate=g)  # in place, no norm
    close(out[:, :inner], d(y) * oracle.sigmoid(d(g)), tol)
    act = torch.full((t, -(-ff // 8) * 8), float("nan"), dtype=dtype, device="cuda")
    z[0, :6] = torch.tensor([0.0, 1e-3, -1e-3, -30.0, 9.0, -1e-6]).to(dtype)[:min(6, ff)]
    for p, q in ((0.3, -0.4), (-2.0, 1.5)):
        ops.mixer_finish(act, 0, z, act="xielu", act_weights=(float(oracle.softplus(p)), float(0.5 + oracle.softplus(q))))
        close(act[:, :ff], oracle.xielu(d(z), [p, q]), tol)
        assert (act[:, ff:] == 0).all()
    ops.mixer_finish(act, 0, z, act="tanh")
    close(act[:, :ff], np.tanh(d(z)), tol)


# -- normed heads and values -----------------------------------------------------------------------------------

@BOTH
@pytest.mark.parametrize("heads,groups,dim,vdim", [(6, 2, 24, 40), (5, 1, 64, 64), (2, 2, 25, 9), (32, 4, 128, 96), (3, 1, 8, 200), (1, 1, 500, 3)])
@pytest.mark.parametrize("temp", [{"coef": 0.5, "every": 16}, {"coef": -0.1, "every": 1}, None])
def test_head_norms_temperature_and_cache_write(ops, heads, groups, dim, vdim, temp, dtype):
    rng = np.random.default_rng(0)
    t, bs, eps = 9, 16, 1e-3
    up = lambda n: -(-n // 8) * 8  # noqa: E731
    cols = [heads * dim, groups * dim, groups * vdim]
    at = np.concatenate([[0], np.cumsum([up(c) for c in cols])])
    stacked = torch.from_numpy(0.3 * rng.standard_normal((t, at[-1]))).to(dtype).cuda()
    q, k, v = (stacked[:, a:a + c].unflatten(1, (-1, s)) for a, c, s in zip(at, cols, (dim, dim, vdim)))
    kc = torch.zeros((4, bs, groups, dim), dtype=dtype, device="cuda")
    vc = torch.zeros((4, bs, groups, vdim), dtype=dtype, device="cuda")
    slots = torch.tensor([16, 17, 63, 31, 32, -1, 48, 5, 64], device="cuda")
    pos = torch.tensor([0, 14, 15, 16, 30, 31, 4095, 1000003, 47], dtype=torch.int32, device="cuda")
    qn, kn = f32(rng.standard_normal(dim)), f32(rng.standard_normal(dim))
    want_q = oracle.over_rms(d(q), eps) * d(qn) * oracle.temperature(d(pos), temp)[:, None, None]
    want_k, want_v = oracle.over_rms(d(k), eps) * d(kn), oracle.over_rms(d(v), eps)
    ops.rope_norm_cache(q, k, v, kc, vc, slots, pos, None, 1.0, eps, q_norm=qn, k_norm=kn, norm_values=True,
                        temperature=(temp["coef"], temp["every"]) if temp else (0.0, 1.0))
    tol = 2e-6 if dtype == torch.float32 else 8e-3
    close(q, want_q, tol)
    used = torch.zeros(4 * bs, dtype=torch.bool)
    for i, s in enumerate(slots.tolist()):
        if 0 <= s < 4 * bs:
            close(kc[s // bs, s % bs], want_k[i], tol)
            close(vc[s // bs, s % bs], want_v[i], tol)
            used[s] = True
    assert float(kc.view(4 * bs, -1)[~used.cuda()].abs().max()) == 0 == float(vc.view(4 * bs, -1)[~used.cuda()].abs().max())


# -- attention with a distance bias ------------------------------------------------------------------------------

class Paged:
    def __init__(self, heads, groups, dim, vdim, lens, dtype, block_size=16, seed=0, slopes=None):
        rng = np.random.default_rng(seed)
        r = lambda *s: torch.from_numpy(rng.standard_normal(s)).to(dtype)  # noqa: E731
        self.heads, self.groups, self.vdim, self.dtype, self.bs = heads, groups, vdim, dtype, block_size
        self.q, self.k, self.v = ([r(n, h, s) for n in lens] for h, s in ((heads, dim), (groups, dim), (groups, vdim)))
        self.slopes = oracle.slopes(heads) if slopes is None else np.asarray(slopes, np.float64)
        pages = [-(-n // block_size) for n in lens]
        ids = rng.permutation(np.arange(1, 1 + sum(pages) + 3))
        self.tables = [list(map(int, ids[sum(pages[:i]):sum(pages[:i + 1])])) for i in range(len(lens))]
        # what other requests left in the pages
        self.kc = torch.full((len(ids) + 1, block_size, groups, dim), float("nan"), dtype=dtype)
        self.vc = torch.full((len(ids) + 1, block_size, groups, vdim), float("nan"), dtype=dtype)

    def run(self, ops, counts, lens, scale, window, **kw):
        """The last ``counts[i]`` of the first ``lens[i]`` tokens of every request as one batch."""
        kc, vc = self.kc.clone(), self.vc.clone()
        for i, n in enumerate(lens):
            p = np.arange(n)
            at = np.asarray(self.tables[i])[p // self.bs], p % self.bs
            kc[at], vc[at] = self.k[i][:n], self.v[i][:n]
        kc, vc = kc.cuda(), vc.cuda()
        meta = segments(counts, lens, tables=[t[:-(-n // self.bs)] for t, n in zip(self.tables, lens)], block_size=self.bs)
        q = torch.cat([self.q[i][n - c:n] for i, (c, n) in enumerate(zip(counts, lens))]).cuda()
        out = torch.full((len(q), self.heads, self.vdim), float("nan"), dtype=self.dtype, device="cuda")
        keep = kw.get("keep_first", 0)
        ops.paged_attention_primitive(q, kc, vc, self.groups, scale, 0.0, meta.block_tables, meta.seq_lens, meta.cu_seqlens_q,
                                      self.bs, max(lens), window, out, wide_weights=True, plain_softmax=True, min_q_len=min(counts),
                                      slopes=f32(self.slopes), **kw)
        want = [self.rows(i, c, n, scale, window, keep) for i, (c, n) in enumerate(zip(counts, lens))]
        close(out, np.concatenate(want), 1e-5 if self.dtype == torch.float32 else 5e-3)

    def rows(self, i, c, n, scale, window, keep):
        q, k, v = (x[i][:n].double().numpy() for x in (self.q, self.k, self.v))
        mask = {"size": max(window, 0)}
        if c > 3 and not keep:
            return oracle.biased_attention(q, k, v, scale, self.slopes, mask)[n - c:]
        out = []
        for r in range(n - c, n):
            js = np.arange(r + 1)
            js = js[oracle.visible(r, js, mask) | (js < keep)]
            per = self.heads // self.groups
            s = np.stack([k[js, h // per] @ q[r, h] * scale - self.slopes[h] * (r - js) for h in range(self.heads)])
            w = np.exp(s - s.max(axis=1, keepdims=True))
            w /= w.sum(axis=1, keepdims=True)
            out.append(np.stack([w[h] @ v[js, h // per] for h in range(self.heads)]))
        return np.stack(out)


WINDOWS = [41, 16, 17, 1, 128, 129, 300, -1]
SIZES = [(6, 2, 24, 40), (10, 1, 64, 64), (4, 2, 128, 128), (2, 2, 5, 9), (18, 1, 32, 16), (12, 1, 80, 176), (1, 1, 48, 48)]


@BOTH
@pytest.mark.parametrize("heads,groups,dim,vdim", SIZES)
@pytest.mark.parametrize("window", WINDOWS)
def test_distance_bias_in_prompts_portions_and_decoding(ops, heads, groups, dim, vdim, window, dtype):
    p = Paged(heads, groups, dim, vdim, [290, 40, 130, 17], dtype)
    scale = 1.5 * dim ** -0.5
    p.run(ops, [290, 40, 130, 17], [290, 40, 130, 17], scale, window)
    p.run(ops, [1, 1, 1, 1], [290, 16, 129, 1], scale, window)
    p.run(ops, [2, 16, 1, 15], [257, 33, 128, 17], scale, window)  # portions on both sides of the tile kernel's limit


@BOTH
@pytest.mark.parametrize("block_size", [8, 32, 64])
def test_distance_bias_on_other_pages(ops, block_size, dtype):
    p = Paged(4, 2, 64, 64, [300, 65], dtype, block_size)
    for window in (41, -1):
        for counts in ([300, 65], [1, 1], [70, 3]):
            p.run(ops, counts, [300, 65], 0.2, window)


@BOTH
@pytest.mark.parametrize("window", [1000, 530, -1])
def test_distance_bias_over_split_keys(ops, window, dtype):
    """Flat slopes, so that far keys count."""
    p = Paged(4, 1, 64, 64, [2100, 700, 33], dtype, slopes=[1e-3, 0.0, 4e-3, 0.02])
    for lens in ([2100, 700, 33], [2065, 529, 16], [2049, 33, 1]):
        p.run(ops, [1, 1, 1], lens, 0.2, window, _force_partitions=2)
        p.run(ops, [1, 1, 1], lens, 0.2, window)
    if dtype == torch.bfloat16:
        p.run(ops, [1, 1, 1], [2100, 700, 33], 0.2, window, _kernel=1, _force_partitions=2)
        p.run(ops, [20, 17, 16], [2100, 700, 33], 0.2, window, _kernel=3)


@BOTH
@pytest.mark.parametrize("heads,groups,dim,vdim", [(6, 2, 24, 40), (10, 1, 64, 64), (2, 2, 5, 9)])
def test_one_outstanding_key_just_inside_and_outside_the_window(ops, heads, groups, dim, vdim, dtype):
    """The key every query asks for lies first or last of what is visible, or one past it, and at pages' edges."""
    for size, n, at in [(30, 150, at) for at in (0, 15, 16, 119, 120, 121, 127, 128, 148, 149)] + [(48, 160, at) for at in (111, 112)]:
        p = Paged(heads, groups, dim, vdim, [n], dtype, seed=at, slopes=np.full(heads, 0.01))
        p.q[0][:, :, 0], p.k[0][:, :, 0] = 8.0, 0.0
        p.k[0][at, :, 0] = 6.0
        for counts, lens in (([n], [n]), ([1], [n]), ([3], [n]), ([1], [max(1, at)]), ([1], [min(n, at + size)]),
                             ([1], [min(n, at + size + 1)]), ([2], [min(n, at + size + 1)])):
            p.run(ops, counts, lens, 0.5, size)


@BOTH
def test_distance_bias_beside_kept_first_tokens(ops, dtype):
    p = Paged(6, 2, 64, 64, [290, 40], dtype, slopes=[0.01, 0.0, 0.3, 1e-3, 0.02, 2.0])
    p.run(ops, [1, 1], [290, 40], 0.2, 41, keep_first=7)
    p.run(ops, [3, 2], [290, 40], 0.2, 17, keep_first=20)


def test_distance_bias_is_refused_where_it_does_not_belong(ops):
    p = Paged(2, 1, 64, 64, [20], torch.bfloat16)
    p.slopes = np.zeros(3)
    with pytest.raises(ValueError, match="slopes"):
        p.run(ops, [1], [20], 1.0, -1)
    q = torch.zeros((1, 2, 64), device="cuda").bfloat16()
    c = torch.zeros((2, 16, 1, 64), device="cuda").bfloat16()
    i = lambda *x: torch.tensor(x, dtype=torch.int32, device="cuda")  # noqa: E731
    with pytest.raises(ValueError, match="softcap"):
        ops.paged_attention_primitive(q, c, c, 1, 1.0, 30.0, i([1]).view(1, 1), i(1), i(0, 1), 16, 1, -1, torch.empty_like(q),
                                      slopes=torch.zeros(2, device="cuda"))


# -- routing -------------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("t,n,top", [(1, 1, 1), (5, 7, 3), (64, 64, 8), (33, 100, 7), (300, 16, 16), (9, 1000, 40)])
def test_routing_over_the_chosen(ops, t, n, top):
    rng = np.random.default_rng(n)
    z = f32(3 * rng.standard_normal((t, n + 5)))
    b = f32(rng.standard_normal(n))
    for bias in (b, None):
        chosen, weights = ops.expert_route(z, bias, n, top, 1.0, True)
        want, w = oracle.route(d(z[:, :n] + bias if bias is not None else z[:, :n]), top)
        assert np.array_equal(chosen.cpu().numpy(), want)
        close(weights, w, 2e-6)
    # logits so far apart that a softmax over all of them would leave nothing of the others
    z = torch.zeros((t, n), device="cuda") - 200.0 * torch.arange(n, device="cuda")
    chosen, weights = ops.expert_route(z, None, n, top, 1.0, True)
    assert chosen.tolist() == [list(range(top))] * t
    close(weights, np.eye(top)[:1].repeat(t, 0), 0)
