"""The kernels of the sandwich-norm decoders one by one against the oracle: the step between sublayers with its convolution,
rotated and normed heads, attention over a window with kept first tokens, routing, expert products."""

from __future__ import annotations

import numpy as np
import pytest
import torch

from oracle import kerolorn as oracle

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
@pytest.mark.parametrize("dim,parts", [(88, 3), (256, 8), (1000, 1), (30, 2), (4096, 8), (37, 5), (2560, 6), (5000, 2), (8196, 4), (1, 1)])
def test_residual_step(ops, dim, parts, dtype):
    rng = np.random.default_rng(dim)
    t, eps = 7, 1e-3
    x = rng.standard_normal((t, dim)).astype(np.float32)
    op = lambda rows, scale: torch.from_numpy(scale * rng.standard_normal((rows, dim))).to(dtype).cuda()  # noqa: E731
    y, ys, extra = op(t, 3.0), op(t * parts, 0.5), op(t, 2.0)
    weights, gates = f32(rng.random((t, parts))), f32(rng.standard_normal((t, 3)))
    post, pre = f32(rng.standard_normal(dim)), f32(rng.standard_normal(dim))
    tol = 2e-5 if dtype == torch.float32 else 8e-3
    mixed = np.einsum("tp,tpd->td", d(weights), d(ys).reshape(t, parts, dim))
    routed = {"y": ys, "part_weight": weights, "norm": post}
    for result, r in ((None, None), ({"y": y, "norm": post}, d(y)), (routed, mixed),
                      (dict(routed, extra=extra, extra_gate=gates[:, 1]), mixed + oracle.sigmoid(d(gates[:, 1:2])) * d(extra))):
        want = x + (0 if r is None else oracle.rms_norm(r, d(post), eps))
        s = f32(x)
        h = ops.residual_step(s, result, pre, eps=eps, dtype=dtype)
        close(s, want, 2e-5)
        close(h, oracle.rms_norm(want, d(pre), eps), tol)
        rows = torch.tensor([5, 0, 5], device="cuda")
        s = f32(x)
        h = ops.residual_step(s, result, pre, eps=eps, dtype=dtype, rows=rows)
        assert np.array_equal(s.cpu().numpy(), x)
        close(h, oracle.rms_norm(want, d(pre), eps)[[5, 0, 5]], tol)
        if result is not None:
            s = f32(x)
            assert ops.residual_step(s, result, eps=eps, dtype=dtype) is None
            close(s, want, 2e-5)


@BOTH
@pytest.mark.parametrize("taps,dim", [(1, 88), (2, 37), (3, 256), (4, 88), (7, 40), (16, 24)])
def test_convolution_in_the_step_and_over_portions(ops, taps, dim, dtype):
    """Portions go through the convolution kernel, batches of single rows through the step itself; both keep the last inputs in
    the request's slot, which starts out as somebody else's."""
    rng = np.random.default_rng(3)
    w = f32(rng.standard_normal((taps, dim)))
    and_input = w.clone()
    and_input[-1] += 1.0
    norm = f32(rng.standard_normal(dim))
    lens = [60, 33, 9]
    x = [rng.standard_normal((n, dim)).astype(np.float32) for n in lens]
    want = [oracle.input_convolution(oracle.rms_norm(a.astype(np.float64), d(norm), 1e-6), d(w).T) for a in x]
    state = torch.full((5, taps - 1, dim), float("nan"), dtype=dtype, device="cuda")
    taken, slots = [0, 0, 0], [2, 4, 1]
    for portions in ({0: 17, 1: 1, 2: 2}, {2: 1, 0: 1, 1: 1}, {1: 1}, {1: 29, 0: 2, 2: 5}, {0: 1, 2: 1}, {0: 38, 1: 1}):
        ids = list(portions)
        for i in ids:
            taken[i] += portions[i]
        seg = segments([portions[i] for i in ids], [taken[i] for i in ids], [slots[i] for i in ids])
        part = lambda a: np.concatenate([a[i][taken[i] - portions[i]:taken[i]] for i in ids])  # noqa: E731
        if seg.max_q_len == 1:
            got = ops.residual_step(f32(part(x)), None, norm, eps=1e-6, dtype=dtype, conv=(w, state), seg=seg)
        else:
            h = ops.residual_step(f32(part(x)), None, norm, eps=1e-6, dtype=dtype)
            got = ops.causal_conv(h, and_input, None, state, seg, silu=False)
        close(got, part(want), 1e-5 if dtype == torch.float32 else 1.2e-2)


# -- rotated, normed heads -----------------------------------------------------------------------------------------

ROTS = [{"base": 1e4, "dims": 8}, {"base": 5e5, "dims": 24, "scaling": {"factor": 8.0, "original": 512, "fast": 16.0, "slow": 1.0}}, None]


@BOTH
@pytest.mark.parametrize("heads,groups,dim,vdim", [(6, 2, 24, 40), (5, 1, 64, 64), (2, 2, 25, 9), (32, 4, 128, 96), (3, 1, 200, 8), (1, 1, 500, 3)])
@pytest.mark.parametrize("rot", ROTS)
def test_rotation_norm_and_cache_write(ops, heads, groups, dim, vdim, rot, dtype):
    from vllm_metal_b200.lm.hybrid_config import RotaryArgs

    rng = np.random.default_rng(0)
    t, bs, eps = 9, 16, 1e-3
    up = lambda n: -(-n // 8) * 8  # noqa: E731
    cols = [heads * dim, groups * dim, groups * vdim]
    at = np.concatenate([[0], np.cumsum([up(c) for c in cols])])
    stacked = torch.from_numpy(0.3 * rng.standard_normal((t, at[-1]))).to(dtype).cuda()
    q, k, v = (stacked[:, a:a + c].unflatten(1, (-1, s)) for a, c, s in zip(at, cols, (dim, dim, vdim)))
    v_before = v.clone()
    kc = torch.zeros((4, bs, groups, dim), dtype=dtype, device="cuda")
    vc = torch.zeros((4, bs, groups, vdim), dtype=dtype, device="cuda")
    slots = torch.tensor([16, 17, 63, 31, 32, -1, 48, 5, 64], device="cuda")
    pos = torch.tensor([0, 1, 15, 511, 4095, 7, 130001, 1000003, 2], dtype=torch.int32, device="cuda")
    temp = f32(rng.standard_normal(heads))
    args = RotaryArgs.parse(rot, "")
    f = torch.tensor(args.frequencies(), dtype=torch.float64)
    freq = torch.stack([f.float(), (f - f.float().double()).float()], 1).contiguous().cuda()
    turned = [oracle.rotate(d(x), d(pos), rot) if rot else d(x) for x in (q, k)]
    want_q, want_k = (oracle.over_rms(x, eps) for x in turned)
    ops.rope_norm_cache(q, k, v, kc, vc, slots, pos, freq, args.amplitude, eps, temp)
    tol = 2e-6 if dtype == torch.float32 else 8e-3
    close(q, want_q * d(temp)[None, :, None], tol)
    used = torch.zeros(4 * bs, dtype=torch.bool)
    for i, s in enumerate(slots.tolist()):
        if 0 <= s < 4 * bs:
            close(kc[s // bs, s % bs], want_k[i], tol)
            assert torch.equal(vc[s // bs, s % bs], v_before[i])
            used[s] = True
    assert float(kc.view(4 * bs, -1)[~used.cuda()].abs().max()) == 0 == float(vc.view(4 * bs, -1)[~used.cuda()].abs().max())


# -- attention over a window with kept first tokens ----------------------------------------------------------------

class Paged:
    def __init__(self, heads, groups, dim, vdim, lens, dtype, block_size=16, seed=0):
        rng = np.random.default_rng(seed)
        r = lambda *s: torch.from_numpy(rng.standard_normal(s)).to(dtype)  # noqa: E731
        self.heads, self.groups, self.vdim, self.dtype, self.bs = heads, groups, vdim, dtype, block_size
        self.q, self.k, self.v = ([r(n, h, s) for n in lens] for h, s in ((heads, dim), (groups, dim), (groups, vdim)))
        pages = [-(-n // block_size) for n in lens]
        ids = rng.permutation(np.arange(1, 1 + sum(pages) + 3))
        self.tables = [list(map(int, ids[sum(pages[:i]):sum(pages[:i + 1])])) for i in range(len(lens))]
        # what other requests left in the pages
        self.kc = torch.full((len(ids) + 1, block_size, groups, dim), float("nan"), dtype=dtype)
        self.vc = torch.full((len(ids) + 1, block_size, groups, vdim), float("nan"), dtype=dtype)

    def run(self, ops, counts, lens, scale, mask, **kw):
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
        size, keep = mask
        ops.paged_attention_primitive(q, kc, vc, self.groups, scale, 0.0, meta.block_tables, meta.seq_lens, meta.cu_seqlens_q,
                                      self.bs, max(lens), size, out, wide_weights=True, plain_softmax=True, min_q_len=min(counts),
                                      keep_first=keep, **kw)
        want = [self.rows(i, c, n, scale, mask) for i, (c, n) in enumerate(zip(counts, lens))]
        close(out, np.concatenate(want), 1e-5 if self.dtype == torch.float32 else 5e-3)

    def rows(self, i, c, n, scale, mask):
        """The last ``c`` of ``n`` rows: all of them from the oracle's attention, few one by one."""
        q, k, v = (x[i][:n].double().numpy() for x in (self.q, self.k, self.v))
        m, out = {"size": max(mask[0], 0), "keep_first": mask[1]}, []
        if c > 3:
            return oracle.softmax_attention(q, k, v, np.full(self.heads, scale), m)[n - c:]
        for r in range(n - c, n):
            js = np.nonzero(oracle.visible(r, np.arange(r + 1), m))[0]
            per = self.heads // self.groups
            s = np.stack([k[js, h // per] @ q[r, h] * scale for h in range(self.heads)])
            w = np.exp(s - s.max(axis=1, keepdims=True))
            w /= w.sum(axis=1, keepdims=True)
            out.append(np.stack([w[h] @ v[js, h // per] for h in range(self.heads)]))
        return np.stack(out)


MASKS = [(41, 7), (16, 0), (17, 1), (1, 3), (5, 64), (128, 16), (129, 131), (64, 5), (33, 400), (300, 12), (-1, 9)]
SIZES = [(6, 2, 24, 40), (10, 1, 64, 64), (4, 2, 128, 128), (2, 2, 5, 9), (18, 1, 32, 16), (12, 1, 80, 176)]


@BOTH
@pytest.mark.parametrize("heads,groups,dim,vdim", SIZES)
@pytest.mark.parametrize("mask", MASKS)
def test_window_with_kept_tokens_in_prompts_portions_and_decoding(ops, heads, groups, dim, vdim, mask, dtype):
    p = Paged(heads, groups, dim, vdim, [290, 40, 130, 17], dtype)
    scale = 1.5 * dim ** -0.5
    p.run(ops, [290, 40, 130, 17], [290, 40, 130, 17], scale, mask)
    p.run(ops, [1, 1, 1, 1], [290, 16, 129, 1], scale, mask)
    p.run(ops, [2, 16, 1, 15], [257, 33, 128, 17], scale, mask)  # portions on both sides of the tile kernel's limit


@BOTH
@pytest.mark.parametrize("block_size", [8, 32, 64])
def test_other_pages(ops, block_size, dtype):
    p = Paged(4, 2, 64, 64, [300, 65], dtype, block_size)
    for mask in ((41, 7), (70, 33)):
        for counts in ([300, 65], [1, 1], [70, 3]):
            p.run(ops, counts, [300, 65], 0.2, mask)


@BOTH
@pytest.mark.parametrize("mask", [(1000, 40), (1203, 1), (530, 700), (5000, 3)])
def test_split_keys(ops, mask, dtype):
    """Partitions over the kept tiles and the window's, counted without the gap between them."""
    p = Paged(4, 1, 64, 64, [2100, 700, 33], dtype)
    for lens in ([2100, 700, 33], [2065, 529, 16], [2049, 33, 1]):
        p.run(ops, [1, 1, 1], lens, 0.2, mask, _force_partitions=2)
        p.run(ops, [1, 1, 1], lens, 0.2, mask)
    if dtype == torch.bfloat16:
        p.run(ops, [1, 1, 1], [2100, 700, 33], 0.2, mask, _kernel=1, _force_partitions=2)
        p.run(ops, [20, 17, 16], [2100, 700, 33], 0.2, mask, _kernel=3)


@BOTH
@pytest.mark.parametrize("heads,groups,dim,vdim", [(6, 2, 24, 40), (10, 1, 64, 64), (2, 2, 5, 9)])
def test_one_outstanding_key_just_inside_and_outside_every_edge(ops, heads, groups, dim, vdim, dtype):
    """The key every query asks for lies first or last of what is visible, or one past it, and at pages' edges."""
    for (size, keep), n, at in [((30, 6), 150, at) for at in (0, 5, 6, 15, 16, 119, 120, 121, 127, 128, 148, 149)] + \
            [((48, 16), 160, at) for at in (15, 16, 111, 112)] + [((20, 33), 200, at) for at in (31, 32, 33, 179, 180)]:
        p = Paged(heads, groups, dim, vdim, [n], dtype, seed=at)
        p.q[0][:, :, 0], p.k[0][:, :, 0] = 8.0, 0.0
        p.k[0][at, :, 0] = 6.0
        for counts, lens in (([n], [n]), ([1], [n]), ([3], [n]), ([1], [max(1, at)]), ([1], [min(n, at + size)]),
                             ([1], [min(n, at + size + 1)]), ([2], [min(n, at + size + 1)])):
            p.run(ops, counts, lens, 0.5, (size, keep))


def test_attention_refuses_a_negative_count_of_kept_tokens(ops):
    with pytest.raises(ValueError, match="keep_first"):
        Paged(2, 1, 64, 64, [20], torch.bfloat16).run(ops, [1], [20], 1.0, (4, -1))


# -- routed experts ------------------------------------------------------------------------------------------------

@pytest.mark.parametrize("t,n,top", [(1, 1, 1), (5, 7, 3), (64, 64, 8), (33, 100, 7), (300, 16, 16), (9, 1000, 10)])
def test_routing(ops, t, n, top):
    rng = np.random.default_rng(n)
    z = f32(2 * rng.standard_normal((t, n + 5)))
    c = f32(rng.standard_normal(n) / n)
    for correction in (c, None):
        chosen, weights = ops.expert_route(z, correction, n, top, 2.5)
        want, w = oracle.route(d(z[:, :n]), d(c) if correction is not None else np.zeros(n), top, 2.5)
        assert np.array_equal(chosen.cpu().numpy(), want)
        close(weights, w, 2e-6)
    chosen, _ = ops.expert_route(torch.zeros((t, n), device="cuda"), None, n, top, 1.0)
    assert chosen.tolist() == [list(range(top))] * t  # ties go to the lower number


@pytest.mark.parametrize("t,n,top,tile", [(1, 5, 2, 32), (64, 64, 8, 32), (300, 16, 4, 64), (2000, 7, 3, 128), (50, 1000, 20, 32)])
def test_plan(ops, t, n, top, tile):
    rng = np.random.default_rng(t)
    chosen = np.stack([rng.permutation(n)[:top] if n < 200 else rng.choice(n // 2, top, replace=False) for _ in range(t)])
    pairs, first, tiles, rows = ops.expert_plan(torch.from_numpy(chosen).int().cuda(), n, tile)
    pairs, first, tiles = (x.cpu().numpy() for x in (pairs, first, tiles))
    counts = np.bincount(chosen.ravel(), minlength=n)
    assert rows == tile and np.array_equal(first, np.concatenate([[0], np.cumsum(counts)]))
    assert np.array_equal(tiles, np.concatenate([[0], np.cumsum(-(-counts // tile))]))
    for e in range(n):
        assert sorted(pairs[first[e]:first[e + 1]]) == np.nonzero(chosen.ravel() == e)[0].tolist()


def test_the_sort_sees_the_choices_of_the_launch_before_it(ops):
    """Routing and sorting back to back into memory that still holds other choices, as a step of the model runs them."""
    rng = np.random.default_rng(0)
    zs = [f32(rng.standard_normal((200, 48))) for _ in range(6)]
    stale = [torch.randint(0, 48, (200, 5), dtype=torch.int32, device="cuda") for _ in range(4)]
    del stale
    got = []
    for z in zs * 5:
        chosen, _ = ops.expert_route(z @ torch.eye(48, device="cuda"), None, 48, 5, 1.0)
        pairs, first, _, _ = ops.expert_plan(chosen, 48, 32)
        got.append((chosen.clone(), pairs.clone(), first.clone()))
    for chosen, pairs, first in got:
        assert torch.equal(first.diff(), torch.bincount(chosen.flatten(), minlength=48).int())
        assert torch.equal(chosen.flatten()[pairs.long()], torch.arange(48, device="cuda").repeat_interleave(first.diff()).int())


def products(ops, t, width, ff, n, top, shared, dtype, tile, kernel, seed=0):
    """Both products of random experts against one matrix product per pair."""
    rng = np.random.default_rng(seed)
    r = lambda *s: torch.from_numpy(rng.standard_normal(s) * s[-1] ** -0.5).to(dtype).cuda()  # noqa: E731
    up8 = lambda c: -(-c // 8) * 8  # noqa: E731
    x = torch.from_numpy(rng.standard_normal((t, width))).to(dtype).cuda()
    w_in = r(n, 2 * ff, width)
    w_out = torch.full((n, width, up8(ff)), float("nan"), dtype=dtype, device="cuda")  # the padding is nobody's
    w_out[:, :, :ff] = r(n, width, ff)
    s_in = s_out = None
    if shared:
        s_in, s_out = r(2 * shared, width), torch.full((width, up8(shared)), float("nan"), dtype=dtype, device="cuda")
        s_out[:, :shared] = r(width, shared)
    # uneven on purpose: expert 0 is popular, the last one never chosen where there is a choice
    score = rng.random((t, n)) + np.linspace(0.8, 0, n)
    if top < n:
        score[:, -1] = -1
    chosen = np.argsort(-score, axis=1)[:, :top]
    plan = ops.expert_plan(torch.from_numpy(np.ascontiguousarray(chosen)).int().cuda(), n, tile)
    act, s_act = ops.expert_product(x, w_in, plan, top, t, gated=True, shared_weight=s_in, kernel=kernel)
    unit = lambda a, w, f: oracle.silu(a @ w[:f].T) * (a @ w[f:].T)  # noqa: E731
    xd, tol = d(x), 1e-5 if dtype == torch.float32 else 6e-3
    pairs = plan[0].cpu().numpy()
    close(act, np.stack([unit(xd[p // top], d(w_in[chosen.flat[p]]), ff) for p in pairs]), tol)
    y, s_y = ops.expert_product(act, w_out, plan, top, t, gated=False, k=ff, shared_x=s_act, shared_weight=s_out,
                                shared_k=shared, kernel=kernel)
    want = np.empty((t * top, width))
    acts = d(act)
    for i, p in enumerate(pairs):
        want[p] = d(w_out[chosen.flat[p], :, :ff]) @ acts[i]
    close(y, want, tol)
    if shared:
        close(s_act, unit(xd, d(s_in), shared), tol)
        close(s_y, d(s_act) @ d(s_out[:, :shared]).T, tol)
    assert not ops.expert_product_failed()
    return act, y


@BOTH
@pytest.mark.parametrize("t,width,ff,n,top,shared", [(1, 88, 40, 7, 3, 56), (5, 37, 19, 4, 1, 9), (40, 64, 33, 5, 5, 0), (3, 24, 1, 1, 1, 1),
                                                     (70, 130, 100, 3, 2, 257)])
def test_products_of_any_size(ops, t, width, ff, n, top, shared, dtype):
    products(ops, t, width, ff, n, top, shared, dtype, 32, 1)


@pytest.mark.parametrize("tile", [32, 64, 128])
@pytest.mark.parametrize("t,width,ff,n,top,shared", [
    (1, 88, 40, 7, 3, 56), (2, 64, 8, 3, 1, 0), (64, 512, 264, 16, 4, 136), (300, 136, 96, 5, 2, 128), (33, 1032, 200, 9, 9, 8),
    (700, 256, 128, 6, 3, 520), (129, 72, 384, 2, 1, 0), (17, 8, 8, 300, 5, 16)])
def test_products_on_tensor_cores(ops, t, width, ff, n, top, shared, tile):
    products(ops, t, width, ff, n, top, shared, torch.bfloat16, tile, 2)


def test_a_rows_results_do_not_depend_on_the_others(ops):
    """The same rows in another batch and another tile: the same bits."""
    rng = np.random.default_rng(9)
    r = lambda *s: torch.from_numpy(rng.standard_normal(s) * s[-1] ** -0.5).bfloat16().cuda()  # noqa: E731
    x, w_in, w_out = 8 * r(90, 256), r(6, 2 * 136, 256), r(6, 256, 136)
    chosen = torch.from_numpy(np.stack([rng.permutation(6)[:2] for _ in range(90)])).int().cuda()

    def run(rows, tile):
        plan = ops.expert_plan(chosen[rows].contiguous(), 6, tile)
        act, _ = ops.expert_product(x[rows].contiguous(), w_in, plan, 2, len(rows), gated=True, kernel=2)
        return ops.expert_product(act, w_out, plan, 2, len(rows), gated=False, kernel=2)[0].view(len(rows), 2, -1)

    whole = run(list(range(90)), 128)
    for rows, tile in (([5], 32), ([89, 3, 40], 64), (list(range(60, 0, -1)), 32)):
        assert torch.equal(run(rows, tile), whole[rows])


def test_products_refuse_what_they_cannot_do(ops):
    x, w = torch.zeros((4, 60), device="cuda").bfloat16(), torch.zeros((2, 8, 60), device="cuda").bfloat16()
    plan = ops.expert_plan(torch.zeros((4, 1), dtype=torch.int32, device="cuda"), 2, 64)
    with pytest.raises(ValueError, match="tcgen05"):
        ops.expert_product(x, w, plan, 1, 4, gated=True, kernel=2)
    with pytest.raises(ValueError, match="tiles of 32"):
        ops.expert_product(x, w, plan, 1, 4, gated=True)
    with pytest.raises(ValueError, match="disagree"):
        ops.expert_product(x[:, :8], w, plan, 1, 4, gated=True)
    with pytest.raises(ValueError, match="experts"):
        ops.expert_route(torch.zeros((2, 4), device="cuda"), None, 4, 5, 1.0)
    with pytest.raises(RuntimeError, match="CUDA"):
        ops.expert_route(torch.zeros((2, 4)), None, 4, 2, 1.0)
