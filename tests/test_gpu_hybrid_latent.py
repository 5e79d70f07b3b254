"""Latent attention on the device: the cache row, both attention forms (latent space, expanded), windows, splits, pages."""

from __future__ import annotations

import numpy as np
import pytest
import torch

from oracle import hybrid as oracle

from .hybrid_helpers import LATENT, segments

pytestmark = pytest.mark.gpu


def plain_attention(q, rows, start, scale, window, rank):
    """``q [n, H, width]`` of positions ``start ..`` over latent rows ``[L, width]``: outputs ``[n, H, rank]``."""
    out = np.zeros((q.shape[0], q.shape[1], rank))
    for i in range(q.shape[0]):
        p = start + i
        js = [j for j in range(len(rows)) if oracle.visible(p, j, window if window > 0 else None)]
        s = q[i] @ rows[js].T * scale
        w = np.exp(s - s.max(axis=1, keepdims=True))
        out[i] = (w / w.sum(axis=1, keepdims=True)) @ rows[js][:, :rank]
    return out


class Pool:
    """Latent rows of several requests scattered over shuffled pages; free rows hold NaN."""

    def __init__(self, lens, width, dtype, block_size, seed=0):
        rng = np.random.default_rng(seed)
        pages = [-(-n // block_size) for n in lens]
        perm = rng.permutation(sum(pages) + 3)
        self.block_size, self.tables, at = block_size, [], 0
        self.cache = torch.full(((sum(pages) + 3) * block_size, width), float("nan"), dtype=dtype)
        self.rows = []
        for n, k in zip(lens, pages):
            table = perm[at:at + k].tolist()
            at += k
            r = torch.from_numpy(rng.standard_normal((n, width))).to(dtype)
            for p in range(n):
                self.cache[table[p // block_size] * block_size + p % block_size] = r[p]
            self.tables.append(table)
            self.rows.append(r)
        self.cache = self.cache.cuda()


@pytest.mark.parametrize("dtype,kernel,splits", [(torch.float32, 1, 0), (torch.bfloat16, 1, 0), (torch.bfloat16, 2, 0),
                                                  (torch.bfloat16, 2, 3), (torch.bfloat16, 2, 7), (torch.bfloat16, 3, 0),
                                                  (torch.bfloat16, 3, 1), (torch.bfloat16, 3, 4)])
@pytest.mark.parametrize("heads,rank,rot,window,bs", [(5, 48, 16, 0, 16), (32, 512, 64, 96, 16), (3, 64, 16, 33, 8),
                                                       (40, 80, 32, 7, 32), (16, 320, 64, 0, 64)])
def test_latent_space_attention(ops, dtype, kernel, splits, heads, rank, rot, window, bs):
    ctx, q_lens = [301, 1, 64, 97, 33], [1, 1, 3, 9, 33]
    pool = Pool(ctx, rank + rot, dtype, bs)
    meta = segments(q_lens, ctx, block_size=bs, tables=pool.tables)
    rng = np.random.default_rng(3)
    q = torch.from_numpy(rng.standard_normal((sum(q_lens), heads, rank + rot))).to(dtype)
    scale = 2.0 * (rank + rot) ** -0.5
    got = ops.latent_attention(q.cuda(), pool.cache, meta, scale, window, rank, max(q_lens), kernel=kernel,
                               force_splits=splits).double().cpu().numpy()
    at = 0
    for i, n in enumerate(q_lens):
        want = plain_attention(q[at:at + n].double().numpy(), pool.rows[i].double().numpy(), ctx[i] - n, scale, window, rank)
        tol = 3e-5 if dtype == torch.float32 else 1e-2
        assert np.abs(got[at:at + n] - want).max() <= tol * np.abs(want).max(), (i, n)
        at += n
    assert not ops.latent_attention_failed()


@pytest.mark.parametrize("dtype,kernel", [(torch.float32, 1), (torch.bfloat16, 2), (torch.bfloat16, 3)])
def test_one_key_just_inside_and_just_outside_the_window(ops, dtype, kernel):
    """One key outweighs all others; it must count for the last position that sees it and for none after."""
    rank, rot, heads, bs, window = 32, 16, 2, 16, 45
    for key in (0, 15, 16, 31, 47):
        n = key + window + 4
        pool = Pool([n], rank + rot, dtype, bs)
        rows = torch.zeros((n, rank + rot))
        rows[key, 0], rows[key, 1] = 30.0, 5.0
        for p in range(n):
            pool.cache[pool.tables[0][p // bs] * bs + p % bs] = rows[p].to(dtype).cuda()
        q = torch.zeros((n, heads, rank + rot), dtype=dtype)
        q[:, :, 0] = 1.0
        out = ops.latent_attention(q.cuda(), pool.cache, segments([n], [n], block_size=bs, tables=pool.tables), 1.0,
                                   window, rank, n, kernel=kernel)[:, :, 1].float().cpu().numpy()
        sees = np.array([oracle.visible(p, key, window) for p in range(n)])
        assert (out[sees] > 4.9).all() and (out[~sees] == 0.0).all(), key
        one = segments([1], [n], block_size=bs, tables=pool.tables)  # decoding: the last position alone
        last = ops.latent_attention(q[:1].cuda(), pool.cache, one, 1.0, window, rank, 1, kernel=kernel)[0, :, 1]
        assert float(last.abs().max()) == 0.0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rot_dims", [0, 4, 8])
def test_cache_row_and_query_columns(ops, dtype, rot_dims):
    t, heads, dim, rot, rank, eps = 37, 3, 12, 8, 20, 1e-4
    rng = np.random.default_rng(1)
    q = torch.from_numpy(rng.standard_normal((t, heads * (dim + rot)))).to(dtype)
    down = torch.from_numpy(3 * rng.standard_normal((t, rank + rot))).to(dtype)
    w = torch.from_numpy(rng.standard_normal(rank)).float()
    pos = np.arange(1000, 1000 + t)
    slots = rng.permutation(64)[:t]
    freq = torch.tensor([700.0 ** (-2.0 * i / max(1, rot_dims)) for i in range(rot_dims // 2)]).cuda()
    cache = torch.zeros((64, rank + rot), dtype=dtype, device="cuda")
    out = {}
    for nope, offset, cols in ((False, rank, rank + rot), (True, dim, 32)):
        out[nope] = torch.full((t, heads, cols), 7.0, dtype=dtype, device="cuda")
        ops.latent_prep(q.cuda(), down.cuda(), w.cuda(), torch.from_numpy(pos.astype(np.int32)).cuda(),
                        torch.from_numpy(slots).cuda(), freq, cache, out[nope], heads=heads, dim=dim, rot_dim=rot,
                        kv_rank=rank, eps=eps, rot_offset=offset, copy_nope=nope)
    d = down.double().numpy()
    c = oracle.rms_norm_plain(d[:, :rank], w.double().numpy(), eps)
    kr = oracle.rotate_interleaved(d[:, None, rank:], pos, rot_dims, 700.0)[:, 0]
    qd = q.double().numpy().reshape(t, heads, dim + rot)
    qr = oracle.rotate_interleaved(qd[:, :, dim:], pos, rot_dims, 700.0)
    tol = 2e-4 if dtype == torch.float32 else 2e-2
    np.testing.assert_allclose(cache[torch.from_numpy(slots).cuda()].double().cpu().numpy(), np.concatenate([c, kr], 1),
                               atol=tol, rtol=tol)
    np.testing.assert_allclose(out[False][:, :, rank:].double().cpu().numpy(), qr, atol=tol, rtol=tol)
    assert bool((out[False][:, :, :rank] == 7.0).all())  # somebody else's columns
    full = out[True].double().cpu().numpy()
    np.testing.assert_allclose(full[:, :, :dim + rot], np.concatenate([qd[:, :, :dim], qr], 2), atol=tol, rtol=tol)
    assert (full[:, :, dim + rot:] == 0.0).all()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rows,heads,n,k", [(1, 3, 40, 24), (70, 2, 136, 72), (5, 4, 33, 13)])
def test_head_linear(ops, dtype, rows, heads, n, k):
    g = torch.Generator().manual_seed(0)
    x = torch.randn((rows, heads, k), generator=g).to(dtype)
    w = torch.randn((heads, n, k), generator=g).to(dtype)
    gate = torch.randn((rows, heads * n), generator=g).to(dtype)
    want = torch.einsum("thk,hnk->thn", x.double(), w.double())
    for use in (False, True):
        y = torch.zeros((rows, heads, n), dtype=dtype, device="cuda")
        ops.head_linear(x.cuda(), w.cuda(), y, gate.cuda() if use else None)
        ref = want * torch.sigmoid(gate.double()).view_as(want) if use else want
        torch.testing.assert_close(y.double().cpu(), ref, atol=1e-5 if dtype == torch.float32 else 3e-2,
                                   rtol=1e-5 if dtype == torch.float32 else 1e-2)


@pytest.mark.parametrize("window", [0, 50, 1])
@pytest.mark.parametrize("dims", [{}, {"dim": 96, "rot_dim": 32, "vdim": 128, "kv_rank": 64, "heads": 2}])
def test_expanded_and_latent_space_forms_agree(window, dims):
    """The same layer, the same batch, both forms; the longer requests continue at an odd position."""
    from vllm_metal_b200.attention.caches.hybrid_cache import HybridCache
    from vllm_metal_b200.lm.hybrid_config import HybridArgs
    from vllm_metal_b200.lm.mixers import LatentAttentionMixer

    from .hybrid_helpers import layer, make_config, random_checkpoint

    m = {**LATENT, **dims, "mask": {"size": window} if window else None}
    m["rot"] = {"base": 5000.0, "dims": m["rot_dim"]}
    cfg = make_config([layer("latent_attention", ff=None, **m)])
    args = HybridArgs.parse(cfg)
    tensors = random_checkpoint(cfg)
    mixer = LatentAttentionMixer(args.layers[0].mixer, args.width, args.eps,
                                 lambda name, shape: tensors["l0.mix." + name].reshape(shape), torch.bfloat16, "cuda")
    h = torch.randn((230, args.width), dtype=torch.bfloat16, device="cuda")
    parts = {k: h @ w.cuda().t() for k, w in mixer.weights.items()}
    inner = m["heads"] * m["vdim"]
    results = []
    for limit in (16, 1 << 30):
        type(mixer).expand_from = property(lambda self, limit=limit: limit)
        try:
            cache = HybridCache(args, 40, 16, 4, torch.bfloat16)
            y1, y2 = (torch.zeros((n, inner), dtype=torch.bfloat16, device="cuda") for n in (130, 100))
            tables = [[3, 9, 1, 7, 30, 22, 21, 20, 19, 11, 12], [5, 2, 8, 14, 15]]
            take = lambda lo, hi: {k: v[lo:hi].contiguous() for k, v in parts.items()}  # noqa: E731
            mixer.run(take(0, 130), None, segments([1, 129], [1, 129], tables=tables[::-1]), cache, 0, y1, 0)
            mixer.run(take(130, 230), None, segments([2, 36, 62], [3, 165, 62],
                                                     tables=[tables[1], tables[0], [33, 34, 35, 36]]), cache, 0, y2, 0)
            results.append(torch.cat([y1, y2]).float())
        finally:
            type(mixer).expand_from = _EXPAND_FROM
    torch.testing.assert_close(results[0], results[1], atol=2e-2 * float(results[1].abs().max()), rtol=0)


def _expand_from():
    from vllm_metal_b200.lm.mixers import LatentAttentionMixer

    return LatentAttentionMixer.__dict__["expand_from"]


_EXPAND_FROM = _expand_from()
