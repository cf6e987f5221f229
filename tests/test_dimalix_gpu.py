"""The Dimalix design on the GPU against the plain implementation (tests/plain_dimalix.py).

Mechanisms alone (the kernels driven directly, with inputs made so that a single key, an edge, a correction or a group
decides the result), then whole models of several small configurations through the trace replay (whole prompts,
token-by-token decoding, portions down to two tokens, mixed batches with pages and slots used again) and through
``LLMEngine.generate`` and the programs.
"""
from __future__ import annotations

import json
import os

import numpy as np
import pytest
import torch

import helpers
import plain_dimalix as pd
from test_nigilorn_gpu import DTYPES, TD, LatentCase, Pages, Step, bf16_round, dev, host, ints, portions, split

pytestmark = pytest.mark.gpu


# ------------------------------------------------------------------------------------------ queries, keys and values
def rotate_halves(u, positions, freq):
    """u [T, heads, d]: of the first 2 * len(freq) dimensions, i turns with i + len(freq)."""
    n = len(freq)
    ang = np.asarray(positions, dtype=np.float64)[:, None] * np.asarray(freq)[None, :]
    c, s = np.cos(ang)[:, None, :], np.sin(ang)[:, None, :]
    out = u.copy()
    out[..., :n], out[..., n:2 * n] = u[..., :n] * c - u[..., n:2 * n] * s, u[..., n:2 * n] * c + u[..., :n] * s
    return out


ROTS = [  # head size, rotated dimensions, base, scaling
    (16, 16, 100.0, None), (24, 10, 9000.0, dict(factor=4.0, original=300, low=1.0, high=4.0)),
    (40, 40, 2e5, dict(factor=8.0, original=2048, low=1.0, high=3.0)), (12, 6, 30.0, dict(factor=2.0, original=20, low=1.0, high=4.0)),
    (10, 2, 7.0, dict(factor=3.0, original=64, low=2.0, high=2.0)), (8, 0, 10.0, None), (128, 128, 1e4, None)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("own_values", [False, True])
@pytest.mark.parametrize("bias", [True, False])
@pytest.mark.parametrize("d,dims,base,scaling", ROTS)
def test_norm_over_the_whole_projection_then_rotation(d, dims, base, scaling, bias, own_values, dtype):
    """Queries and cached keys normed with all heads together before they turn; values that are the keys as projected, or
    columns of their own; heads of very unequal size, so that a norm per head would show; positions far out; both pairings."""
    from swifttransformer_b200 import ops
    rng = np.random.default_rng(d + dims)
    H, G, ps, eps = 6, 2, 4, 3e-2
    vd = 12 if own_values else d
    freq = pd.rotation_frequencies(dict(dims=dims, base=base, scaling=scaling))
    start, T = 1003, 9
    width = (H + G) * d + (G * vd if own_values else 0)
    loud = np.repeat([1.0, 9.0, 0.1, 3.0, 0.5, 1.0], d)
    proj = bf16_round(rng.normal(size=(T + 1, width)) * np.concatenate([loud, np.repeat([4.0, 0.2], d), np.ones(width - (H + G) * d)]))
    b = rng.normal(size=width).astype(np.float32).astype(np.float64) if bias else np.zeros(width)
    qn, kn = (1 + 0.3 * rng.normal(size=n * d).astype(np.float32).astype(np.float64) for n in (H, G))
    st = Step([(1, start, T)], pad_tokens=1)
    table = np.full((2, (start + T) // ps + 1), -1, dtype=np.int32)
    need = np.arange(start // ps, (start + T - 1) // ps + 1)
    table[1, need] = rng.permutation(len(need))
    pos = np.arange(start, start + T)
    v_off = (H + G) * d if own_values else H * d
    for neighbours in (True, False):
        pool = torch.zeros((len(need), 1, G * ps * (d + vd)), dtype=TD[dtype], device="cuda")
        q = torch.zeros((T + 1, H * d), dtype=TD[dtype], device="cuda")
        status = torch.zeros(1, dtype=torch.int32, device="cuda")
        ops.gqa_prepare_whole_norm(dev(proj, TD[dtype]), 0, H * d, v_off, dev(b) if bias else None, dev(freq) if dims else None,
                                   dims, 0.0, 1, q, pool, 0, st.positions, st.seq, st.slots, ints(table), H, G, d, vd, ps,
                                   status, dev(qn), dev(kn), eps, neighbours=neighbours)
        assert int(status.item()) == 0
        full = proj[:T] + b
        if neighbours:
            turn = lambda u: pd.rotate_neighbours(u, pos, dict(dims=dims, base=base, scaling=scaling))
        else:
            turn = lambda u: rotate_halves(u, pos, freq)
        rq = turn(pd.rms_norm(full[:, :H * d], qn, eps).reshape(T, H, d))
        rk = turn(pd.rms_norm(full[:, H * d:(H + G) * d], kn, eps).reshape(T, G, d))
        rv = full[:, v_off:v_off + G * vd].reshape(T, G, vd)
        tol = 2e-4 if dtype == "float32" else 1.5e-2                     # float angles at positions in the thousands
        assert np.abs(host(q)[:T].reshape(T, H, d) - rq).max() < tol * np.abs(rq).max() and np.all(host(q)[T] == 0)
        flat = host(pool)[:, 0]
        keys, vals = flat[:, :G * ps * d].reshape(-1, G, ps, d), flat[:, G * ps * d:].reshape(-1, G, ps, vd)
        for t in range(T):
            page, at = table[1, (start + t) // ps], (start + t) % ps
            assert np.abs(keys[page, :, at] - rk[t]).max() < tol * np.abs(rk).max()
            assert np.abs(vals[page, :, at] - rv[t]).max() < (1e-6 if dtype == "float32" else 5e-3) * np.abs(rv).max()


# ------------------------------------------------------------------------------------------ attention in chunks
def seen_mask(T, chunk, window, keep):
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    near = np.ones((T, T), bool)
    if chunk:
        near &= i // chunk == j // chunk
    if window:
        near &= i - j < window
    return (j <= i) & (near | (j < keep))


class ChunkCase:
    """Grouped attention over the keys of a query's own chunk (and, where a case says so, of a window inside it and the
    request's first keys); unused rows of the pool hold large numbers."""

    def __init__(self, lengths, H, G, d, vd, ps, chunk, seed, dtype, window=0, keep=0):
        rng = np.random.default_rng(seed)
        self.H, self.G, self.d, self.vd, self.ps, self.dtype = H, G, d, vd, ps, dtype
        self.chunk, self.window, self.keep = chunk, window, keep
        self.pages, self.lengths = Pages(lengths, ps, rng), list(lengths)
        self.q = [bf16_round(rng.normal(size=(n, H, d))) for n in lengths]
        self.k = [bf16_round(rng.normal(size=(n, G, d))) for n in lengths]
        self.v = [bf16_round(rng.normal(size=(n, G, vd))) for n in lengths]
        self.scale = 0.9 / np.sqrt(d)

    def write(self):
        G, ps, d, vd, P = self.G, self.ps, self.d, self.vd, self.pages.n_pages
        keys, vals = np.full((P, G, ps, d), 3e4), np.full((P, G, ps, vd), 3e4)
        for i in range(len(self.lengths)):
            for p, page, at in self.pages.each(i):
                keys[page, :, at], vals[page, :, at] = self.k[i][p], self.v[i][p]
        flat = np.concatenate([keys.reshape(P, -1), vals.reshape(P, -1)], axis=1)
        pool = np.full((P, 2, flat.shape[1]), 3e4)
        pool[:, 1] = flat
        self.pool = dev(pool, TD[self.dtype])

    def reference(self, i):
        seen = seen_mask(self.lengths[i], self.chunk, self.window, self.keep)
        return pd.attend(self.q[i], self.k[i], self.v[i], seen, self.scale).reshape(self.lengths[i], -1)

    def passed(self, i, pos):
        """The table when the request's next query stands at ``pos``: pages no later query sees are gone."""
        table = self.pages.table.copy()
        first = pos // self.chunk * self.chunk if self.chunk else 0
        if self.window:
            first = max(first, pos - self.window + 1)
        kept = (self.keep + self.ps - 1) // self.ps
        table[self.pages.slot[i], kept:max(kept, first // self.ps)] = -1
        return table

    def kernels(self):
        from swifttransformer_b200 import ops
        probe = torch.zeros(1, dtype=TD[self.dtype], device="cuda")
        fast = ops.gqa_attention_fast_applies(probe, self.H, self.G, self.d, self.vd)
        return ["plain", "items"] + (["tiles", "single"] if fast else [])

    def run(self, entries, kernel, pad_tokens=0, table=None):
        from swifttransformer_b200 import ops
        H, G, d, vd = self.H, self.G, self.d, self.vd
        st = Step([(self.pages.slot[i], s, n) for i, s, n in entries], pad_tokens=pad_tokens)
        q = dev(np.concatenate([self.q[i][s:s + n].reshape(n, -1) for i, s, n in entries] + [np.full((pad_tokens, H * d), 50.0)]),
                TD[self.dtype])
        out = torch.full((st.n_rows, H * vd), 77.0, dtype=TD[self.dtype], device="cuda")
        status = torch.zeros(1, dtype=torch.int32, device="cuda")
        bt = ints(self.pages.table if table is None else table)
        tail = (H, G, d, vd, self.ps, self.scale, self.window, self.keep, None, None, 0, 1.0)
        kw = dict(status=status, chunk=self.chunk)
        args, rows = (q, self.pool, 1, out), (st.positions, st.seq, st.slots, bt)
        if kernel == "plain":
            ops.gqa_attention_plain(*args, *rows, *tail, **kw)
        elif kernel in ("items", "single"):
            items = ints(list(range(st.n))[::-1] + [-1, -1])
            fn = ops.gqa_attention_plain if kernel == "items" else ops.gqa_attention_single
            fn(*args, *rows, *tail, items=items, n_items=st.n + 2, **kw)
        else:
            tr = ops.attention_prefill_tile_rows()
            tiles = [(k, off) for k, (_, _, n) in enumerate(entries) for off in range(0, n, tr)][::-1] + [(0, 1 << 24)]
            ops.gqa_attention_tiles(*args, ints(tiles), len(tiles), tr, st.q_start, st.start_pos, st.slots, bt, *tail, **kw)
        return split(out, entries, st, status)


CHUNKS = [  # H, G, d, vd, page size, chunk, window, first keys
    (6, 2, 16, 16, 8, 21, 0, 0), (4, 4, 32, 8, 16, 64, 0, 0), (8, 1, 64, 64, 4, 1, 0, 0), (3, 3, 12, 20, 16, 7, 0, 0),
    (16, 4, 40, 48, 32, 130, 0, 0), (9, 1, 8, 8, 8, 40, 0, 0), (20, 2, 24, 24, 8, 1000, 0, 0), (2, 1, 128, 128, 16, 100, 0, 0),
    (4, 2, 32, 32, 8, 50, 13, 0), (4, 1, 16, 16, 16, 70, 30, 3), (2, 2, 96, 96, 8, 33, 0, 5)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", CHUNKS)
def test_chunked_attention_whole_batched_in_portions_and_decoded(shape, dtype):
    H, G, d, vd, ps, chunk, window, keep = shape
    c = ChunkCase((150, 1, 37, 203), H, G, d, vd, ps, chunk, H + d, dtype, window, keep)
    c.write()
    refs = [c.reference(i) for i in range(len(c.lengths))]
    top = max(np.abs(r).max() for r in refs)
    tol = (1e-5 if dtype == "float32" else 2e-2) * top
    for kernel in c.kernels():
        whole = c.run([(i, 0, n) for i, n in enumerate(c.lengths)], kernel, pad_tokens=3)
        for i, r in enumerate(refs):
            assert np.abs(whole[i] - r).max() < tol, (kernel, i)
        assert np.abs(c.run([(3, 0, 203)], kernel)[3] - whole[3]).max() < tol
        for start, n in portions(203, (70, 2, 5, 33, 2)):
            got = c.run([(0, 120, 1), (3, start, n)], kernel, table=c.passed(3, start))
            assert np.abs(got[3] - refs[3][start:start + n]).max() < tol, (kernel, start, n)
            assert np.abs(got[0] - refs[0][120:121]).max() < tol
        edges = [p for e in range(chunk, 203, chunk) for p in (e - 1, e)][:40] if chunk > 1 else []
        for pos in sorted({0, 1, ps - 1, ps, 100, 202} | set(edges)):
            got = c.run([(3, pos, 1), (2, 36, 1)], kernel, pad_tokens=1, table=c.passed(3, pos))
            assert np.abs(got[3] - refs[3][pos:pos + 1]).max() < tol, (kernel, pos)
            assert np.abs(got[2] - refs[2][36:37]).max() < tol


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind,shape,size", [("grouped", (4, 2, 32, 32, 8), 24), ("grouped", (3, 1, 20, 20, 16), 100),
                                             ("grouped", (2, 2, 64, 64, 16), 64), ("latent", (4, 32, 8, 8), 24),
                                             ("latent", (3, 48, 16, 16), 100)])
def test_one_loud_key_just_inside_and_just_outside(kind, shape, size, dtype):
    """A key that takes all the weight wherever it is seen: the result is its value up to the last position of its chunk (of
    its window), and knows nothing of it one position further; in prompt rows and decoded tokens, at the borders of chunks
    and pages and at the request's first tokens."""
    T = 230
    for loud in (0, 1, size - 1, size, 2 * size - 1, shape[-1] - 1, shape[-1], 50):
        if kind == "grouped":
            c = ChunkCase((T,), *shape, size, loud + 1, dtype)
            first_out, passed = (loud // size + 1) * size, lambda p: c.passed(0, p)
        else:
            c = LatentCase((T,), *shape, size, loud + 1, dtype)
            first_out, passed = loud + size, lambda p: c.pages.without_passed_pages(0, p, size)
        vector = np.ones(c.k[0].shape[-1]) * 3.0
        c.k[0][loud] = vector
        c.q[0][:] = bf16_round(c.q[0] * 0.1 + vector * (12.0 / (9.0 * vector.size) / c.scale))
        c.write()
        ref = c.reference(0)
        tol = (2e-5 if dtype == "float32" else 2e-2) * np.abs(ref).max()
        for kernel in c.kernels():
            assert np.abs(c.run([(0, 0, T)], kernel)[0] - ref).max() < tol, (kernel, loud)
            for pos in [p for p in (loud, first_out - 1, first_out, first_out + 1) if p < T]:
                one = c.run([(0, pos, 1)], kernel, table=passed(pos))[0]
                assert np.abs(one - ref[pos]).max() < tol, (kernel, loud, pos)
            two = c.run([(0, first_out - 1, 2)], kernel, table=passed(first_out - 1))[0] if first_out < T else None
            assert two is None or np.abs(two - ref[first_out - 1:first_out + 1]).max() < tol, (kernel, loud)
        if first_out < T and kind == "grouped":
            value = np.repeat(c.v[0][loud], c.H // c.G, axis=0).reshape(-1)
            assert np.abs(ref[first_out - 1] - value).max() < 0.2 * np.abs(value).max()      # the edge itself shows
            assert np.abs(ref[first_out] - value).max() > 0.3 * np.abs(value).max()


# ------------------------------------------------------------------------------------------ routing and experts
ROUTERS = [  # experts, identity outputs, top, groups (count, keep)
    (10, 2, 3, (4, 2)), (6, 0, 6, None), (13, 3, 2, (16, 5)), (7, 2, 1, (3, 1)), (56, 8, 8, (8, 3)), (8, 2, 4, (2, 1)), (1, 0, 1, None),
    (1, 3, 2, (2, 2)), (69, 1, 5, (35, 20)), (30, 3, 7, (3, 2))]


@pytest.mark.parametrize("shift", [0.0, -3.0])
@pytest.mark.parametrize("E,identity,top,groups", ROUTERS)
def test_choice_by_corrected_scores(E, identity, top, groups, shift):
    """From a product's logits and from the hidden rows; corrections that change most choices, also where every choice
    score is negative (an expert outside the kept groups must not count as nought)."""
    from swifttransformer_b200 import ops
    rng = np.random.default_rng(E * top + identity)
    T, W, n = 90, 24, E + identity
    wr, h = bf16_round(rng.normal(size=(n, W)) * 0.4), bf16_round(rng.normal(size=(T, W)))
    b = (rng.normal(size=n) * 1.5 / n + shift).astype(np.float32)
    router = dict(experts=E, identity=identity, top=top, **({"groups": dict(count=groups[0], keep=groups[1])} if groups else {}))
    z = h @ wr.T
    chosen, weights = pd.route(z, b.astype(np.float64), router)
    if n > top and shift == 0.0:
        assert not np.array_equal(chosen, pd.route(z, np.zeros(n), router)[0])
    pos = ints(list(range(T - 1)) + [-1])
    rule = dict(renorm=True, scores="softmax", groups=groups, correction=dev(b), group_score="max")
    wide = np.concatenate([z, np.full((T, 3), 9.0)], axis=1)
    for experts, got in (ops.moe_choose(dev(wide), n, top, pos, **rule), ops.moe_route(dev(h), dev(wr), top, pos, None, **rule)[:2],
                         ops.moe_route(dev(h, torch.bfloat16), dev(wr), top, pos, None, **rule)[:2]):
        e = experts.cpu().numpy()
        same = (e[:-1] == chosen[:-1]).all(axis=1)
        assert same.mean() > 0.97 and np.all(e[-1] == -1)          # (32-bit sums at a shift of 3 make a few near ties)
        assert shift or same.all()
        assert np.abs(host(got)[:-1][same] - weights[:-1][same]).max() < 1e-5


def test_group_score_is_the_largest_choice_score():
    """The group with the single largest choice score wins over the one whose two largest add up to more; with the sum of
    two the other one would."""
    from swifttransformer_b200 import ops
    z = np.log(np.array([[0.35, 0.02, 0.03, 0.3, 0.28, 0.02]]))
    experts, w = ops.moe_choose(dev(z), 6, 2, None, renorm=True, groups=(2, 1), group_score="max")
    assert experts.cpu().tolist() == [[0, 2]] and np.allclose(host(w), [[0.35 / 0.38, 0.03 / 0.38]], atol=1e-6)
    experts, _ = ops.moe_choose(dev(z), 6, 2, None, renorm=True, groups=(2, 1), group_score="top2")
    assert experts.cpu().tolist() == [[3, 4]]
    # corrections lift a group whose scores are small; the weights are the bare scores
    fix = dev(np.array([-1.0, -1.0, -1.0, -1.0, -1.0, -0.5]))
    experts, w = ops.moe_choose(dev(z), 6, 2, None, renorm=True, groups=(3, 1), group_score="max", correction=fix)
    assert experts.cpu().tolist() == [[5, 4]] and np.allclose(host(w), [[0.02 / 0.3, 0.28 / 0.3]], atol=1e-6)


class PartCtx:
    def __init__(self, T):
        self.positions = ints(list(range(T)) + [-1])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T", [5, 70])
@pytest.mark.parametrize("E,identity,top,groups,ff", [(10, 2, 3, (4, 2), 24), (4, 0, 2, None, 20), (5, 3, 1, (2, 1), 64), (2, 6, 4, (2, 1), 16)])
def test_experts_some_of_which_are_the_identity(E, identity, top, groups, ff, T, dtype):
    """A mixture alone: its sum as a tensor, and unsummed for a block that forms it."""
    from swifttransformer_b200.parts.base import FEED_FORWARDS
    rng = np.random.default_rng(E * ff + T)
    W, n = 40, E + identity
    w = {"router": bf16_round(rng.normal(size=(n, W))), "correction": bf16_round(rng.normal(size=n) * 0.3)}
    for e in range(E):
        w[f"e{e}.gate"], w[f"e{e}.up"] = (bf16_round(rng.normal(size=(ff, W)) * 0.4) for _ in range(2))
        w[f"e{e}.down"] = bf16_round(rng.normal(size=(W, ff)) * 0.3)
    h = bf16_round(rng.normal(size=(T, W)))
    router = dict(experts=E, identity=identity, top=top, **({"groups": dict(count=groups[0], keep=groups[1])} if groups else {}))
    ref = pd.experts_ff(h, w, "", {"router": router})
    if identity:
        chosen, _ = pd.route(h @ w["router"].T, w["correction"], router)
        assert (chosen >= E).any()
    part = FEED_FORWARDS.build("routed_experts", hidden=W, inner=ff, num_experts=E, top=top, activation="silu",
                               expert_names=[{k: f"e{e}.{k}" for k in ("gate", "up", "down")} for e in range(E)],
                               router_name="router", renormalise=True, groups=groups, group_score="max",
                               correction_name="correction", identity=identity)
    part.bind({k: dev(v, torch.float32 if k in ("router", "correction") else TD[dtype]) for k, v in w.items()})
    rows = dev(np.concatenate([h, np.zeros((1, W))]), TD[dtype])
    tol = (2e-5 if dtype == "float32" else 2e-2) * np.abs(ref).max()
    for got in (part.forward(rows, PartCtx(T)).value, part.forward_unsummed(rows, PartCtx(T)).total()):
        assert got.dtype == torch.float32 and np.abs(host(got)[:T] - ref).max() < tol


# ------------------------------------------------------------------------------------------ sums, scales and norms
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [20, 64, 33, 192, 2048, 2056, 4100, 8192, 9001])
def test_scaled_sum_of_two_results_and_two_norms_in_one_kernel(width, dtype):
    """x + e + (s1 a + s2 f) in place with each part present or absent, f given or summed from experts, both norms or one or
    none, all rows or chosen ones; padding rows are left alone."""
    from swifttransformer_b200 import ops
    rng = np.random.default_rng(width)
    T, eps, top, n_real = 9, 1e-3, 3, 4
    f32 = lambda *s: rng.normal(size=s).astype(np.float32).astype(np.float64)
    x, a, f, e = f32(T, width), f32(T, width), f32(T, width), f32(T, width)
    s1, s2, w1, w2 = (1 + 0.4 * f32(width) for _ in range(4))
    experts = rng.integers(0, n_real + 2, size=(T, top)).astype(np.int32)
    experts[2] = n_real                                     # all identity
    experts[3] = 1                                          # none
    weights = np.abs(f32(T, top))
    order = ops.moe_sort(ints(experts), n_real)
    place = order.place.cpu().numpy().reshape(T, top)
    y, h = bf16_round(f32(T * top, width)), bf16_round(f32(T, width))
    summed = np.zeros((T, width))
    for t in range(T):
        for k in range(top):
            summed[t] += weights[t, k] * (y[place[t, k]] if experts[t, k] < n_real else h[t])
    items = ops.ExpertSum(dev(y, TD[dtype]), order, dev(weights), ints(experts), n_real, dev(h, TD[dtype]))
    assert np.abs(host(items.total()) - summed).max() < 1e-5 * np.abs(summed).max()
    pos = ints(list(range(T - 1)) + [-1])
    rows = [5, 0, 5, 7]
    for use_a, use_f, use_e, norms, chosen in [(1, 1, 0, 2, 0), (1, 2, 0, 2, 0), (1, 2, 1, 2, 0), (1, 0, 0, 1, 0), (0, 0, 0, 2, 0), (0, 0, 1, 1, 0),
                                               (1, 2, 0, 0, 0), (1, 1, 1, 0, 0), (0, 1, 0, 2, 0), (1, 2, 0, 1, 1), (1, 0, 1, 1, 1)]:
        new = x + (e if use_e else 0) + (s1 * a if use_a else 0) + (s2 * (f if use_f == 1 else summed) if use_f else 0)
        xd = dev(x)
        n = len(rows) if chosen else T
        outs = [torch.full((n, width), 5.0, dtype=TD[dtype], device="cuda") if i < norms else None for i in range(2)]
        ops.scaled_sum_norms(xd, eps, dev(a) if use_a else None, dev(s1) if use_a else None, dev(f) if use_f == 1 else None,
                             dev(s2) if use_f else None, dev(e) if use_e else None, items if use_f == 2 else None,
                             dev(w1) if norms > 0 else None, outs[0], dev(w2) if norms > 1 else None, outs[1],
                             None if chosen else pos, ints(rows) if chosen else None)
        got, case = host(xd), (use_a, use_f, use_e, norms, chosen)
        if chosen:
            assert np.abs(got - x).max() < 1e-6, case
        else:
            assert np.abs(got[:-1] - new[:-1]).max() < 2e-5 * np.abs(new).max() and np.abs(got[-1] - x[-1]).max() < 1e-6, case
        for o, w in zip(outs, (w1, w2)):
            if o is None:
                continue
            ref = pd.rms_norm(new, w, eps)
            tol = (2e-5 if dtype == "float32" else 5e-3) * np.abs(ref).max()
            if chosen:
                assert np.abs(host(o) - ref[rows]).max() < tol, case
            else:
                assert np.abs(host(o)[:-1] - ref[:-1]).max() < tol and np.all(host(o)[-1] == 5.0), case


def test_embedding_rows_are_added_in_float():
    """The opening of a later pass, behind a block that left scaled results and behind one that left nothing."""
    from swifttransformer_b200.parts.base import BLOCKS
    from swifttransformer_b200.parts.block import ResidualStream
    rng = np.random.default_rng(3)
    x, x0, a = (rng.normal(size=(5, 24)).astype(np.float32) for _ in range(3))
    again = BLOCKS.build("reentry_add")
    for pending in (True, False):
        s = ResidualStream(dev(x), torch.bfloat16, embedded=dev(x0))
        if pending:
            s.scaled_pending = (dev(a), dev(np.full(24, 2.0)), None, None)
        again.forward(s, None, None)
        s.fold()
        assert np.abs(host(s.x) - (x + x0 + (2.0 * a if pending else 0))).max() < 1e-6 and s.carry is None


# ------------------------------------------------------------------------------------------ whole models
def rot(dims, base, factor=None, original=64, low=1.0, high=4.0):
    r = {"dims": dims, "base": base}
    if factor:
        r["scaling"] = {"factor": factor, "original": original, "low": low, "high": high}
    return r


def lat(heads, dim, rot_dim, vdim, kr, scale, size, r, mlp):
    mx = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kr, scale=scale)
    mx.update({"mask": {"size": size}} if size else {}, **({"rot": r} if r else {}))
    return {"type": "latent_attention", "mixer": mx, "mlp": mlp}


def att(heads, kv, dim, scale, size, r, mlp):
    mx = dict(heads=heads, kv_heads=kv, dim=dim, vdim=dim, scale=scale)
    mx.update({"mask": {"size": size}} if size else {}, **({"rot": r} if r else {}))
    return {"type": "attention", "mixer": mx, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, identity=0, groups=None):
    r = {"experts": experts, "top": top, **({"identity": identity} if identity else {})}
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": r}


# (``over``: the share of positions that may be further off in bfloat16 because a token went to another expert)
CONFIGS = {
    # sizes that are multiples of nothing; a stretch in the middle that runs three times; chunks and windows of several
    # sizes that pass over prompts and decoded tokens; a layer without feed-forward
    "mix": dict(cfg=dict(architecture="Dimalix", vocab=300, width=44, norm={"eps": 1e-5}, embedding={"scale": 3.0},
                         loop={"start": 1, "stop": 3, "times": 3}, layers=[
        att(4, 2, 14, 0.8, 9, rot(6, 50.0, 2.0, 40), dense(40)),
        lat(3, 10, 6, 7, 22, 0.3, 12, rot(6, 100.0), moe(7, 3, 20, 2, (3, 2))),
        att(3, 3, 6, 0.9, 33, None, None),
        lat(2, 5, 4, 9, 13, 0.4, 40, rot(2, 20.0), dense(30)),
        att(6, 2, 10, 0.5, 50, rot(10, 300.0, 8.0, 100), moe(4, 1, 12, 1))]), seed=51, std=0.1, page_size=8, over=0.35),
    # sizes that the tensor-core kernels take; the first layers run twice; masks longer than a tile of queries; in it
    # the only layer that chooses between experts is the last one, so that nothing carries a choice on
    "fast": dict(cfg=dict(architecture="Dimalix", vocab=200, width=64, norm={"eps": 3e-6}, embedding={"scale": 8.0},
                          loop={"start": 0, "stop": 2, "times": 2}, layers=[
        lat(8, 16, 8, 24, 64, 0.2, 40, rot(8, 1e4), moe(4, 4, 32)),
        att(8, 2, 32, 0.25, 130, rot(32, 3e5, 2.0, 512), dense(96)),
        lat(4, 32, 16, 8, 32, 0.2, 150, rot(16, 500.0), None),
        att(8, 4, 16, 0.3, 48, rot(16, 1000.0, 4.0, 64, 2.0, 8.0), moe(14, 4, 16, 2, (8, 4)))]), seed=52, std=0.12,
                 page_size=16, over=0.15),
    # one head, one expert, nothing that repeats, a stretch that runs once, no mask, no rotation, a chunk of one, a window of one
    "lone": dict(cfg=dict(architecture="Dimalix", vocab=64, width=20, norm={"eps": 1e-4}, loop={"start": 0, "stop": 5, "times": 1}, layers=[
        att(1, 1, 4, 0.5, 1, rot(2, 3.0), moe(1, 1, 8)),
        lat(1, 4, 2, 6, 5, 0.5, 0, None, dense(16)),
        att(3, 1, 6, 0.5, 0, None, moe(2, 2, 4, 1)),
        lat(2, 3, 0, 4, 9, 0.5, 1, None, moe(1, 1, 8, 2, (3, 2))),
        att(9, 1, 8, 0.5, 16, rot(4, 7.0, 2.0, 30, 1.0, 1.0), None)]), seed=53, std=0.25, page_size=4, over=0.1),
}


def louder(name, t, std):
    """Random weights under which faults show: layer scales far from one and of either sign, biases and corrections as
    large as what they are added to, loud queries, keys and routers."""
    f = t.float()
    if name.endswith((".ls1", ".ls2")):
        return (f - 1.0) * 5 + 0.5
    if name.endswith(".router"):
        return f * 3
    if name.endswith(".correction"):
        return f / std * 0.2
    if name.endswith(".b"):
        return f * 4
    if name.endswith((".mix.q", ".mix.k", ".mix.dkv")):
        return f * 2
    return f


def write_model(path, cfg_dict, seed, std):
    from swifttransformer_b200.config import DimalixConfig, save_config
    from swifttransformer_b200.models import build_model_def
    from swifttransformer_b200.weights.random_init import random_tensors
    from swifttransformer_b200.weights.safetensors_io import write_safetensors
    cfg = DimalixConfig.from_dict(cfg_dict)
    save_config(cfg, path)
    tensors = [(s.name, louder(s.name, t, std).to(torch.bfloat16))
               for s, t in random_tensors(build_model_def(cfg).param_specs(), seed, std, "cpu")]
    write_safetensors(os.path.join(path, "model.safetensors"), tensors)
    return path


@pytest.fixture(scope="module")
def model_dirs(tmp_path_factory):
    root = tmp_path_factory.mktemp("dimalix")
    return {name: write_model(str(root / name), c["cfg"], c["seed"], c["std"]) for name, c in CONFIGS.items()}


_PLAIN = {}


def plain_logits(model_dir, tokens):
    key = (model_dir, tuple(tokens))
    if key not in _PLAIN:
        if model_dir not in _PLAIN:
            _PLAIN[model_dir] = pd.load_model(model_dir)
        cfg, w = _PLAIN[model_dir]
        _PLAIN[key] = pd.forward(cfg, w, tokens)
    return _PLAIN[key]


def requests_for(name, lengths=(210, 1, 23, 97, 64)):
    vocab = CONFIGS[name]["cfg"]["vocab"]
    return {f"r{i}": helpers.random_tokens(vocab, n, seed=10 * i + len(name)) for i, n in enumerate(lengths)}


def compare(model_dir, reqs, got, dtype, what, over=0.1):
    """float32: every position within rounding.  bfloat16: rounding of the activations can hand a token to another
    expert where two scores nearly tie, so over all requests of a run the share ``over`` of the positions may lie further
    off; the typical one must be close and none wild."""
    tol = {"float32": 3e-5, "bfloat16": 5e-2}[dtype]
    errs = []
    for rid, toks in reqs.items():
        ref = plain_logits(model_dir, toks)
        assert got[rid].shape == ref.shape, (what, rid)
        scale = np.abs(ref).max()
        if dtype == "float32":
            bad = helpers.first_bad(got[rid], ref, tol * scale)
            assert bad is None, (f"{what}/{dtype}: request {rid} first differs at position {bad[0]} of {len(toks)} by "
                                 f"{bad[1]:.3e} of {scale:.3e}")
        errs.append(np.abs(got[rid] - ref).max(axis=1) / scale)
    err = np.concatenate(errs)
    if dtype == "bfloat16":
        assert np.median(err) < tol / 2 and (err > tol).mean() <= over and err.max() < 30 * tol, \
            f"{what}/{dtype}: median {np.median(err):.3e}, over {(err > tol).mean():.3f}, worst {err.max():.3e} at {int(np.argmax(err))}"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(CONFIGS))
@pytest.mark.parametrize("schedule", ["whole", "decode", "portions", "mixed"])
def test_replay_matches_plain(model_dirs, name, dtype, schedule):
    from swifttransformer_b200.engine.replay import TraceSession
    reqs = requests_for(name)
    steps = {"whole": helpers.trace_whole, "decode": lambda r: helpers.trace_decode_tail(r, tail=60),
             "portions": helpers.trace_portions, "mixed": lambda r: helpers.trace_mixed(r, seed=1, max_live=3)}[schedule](reqs)
    s = TraceSession(model_dirs[name], dtype, helpers.live_token_need(steps), page_size=CONFIGS[name]["page_size"], max_requests=3)
    got = helpers.replay(s, steps)
    compare(model_dirs[name], reqs, got, dtype, f"{name}/{schedule}", CONFIGS[name]["over"])
    s.cache.check()
    assert all(g.pool.num_held == 0 for g in s.cache.groups)


def test_residual_stream_after_every_layer_run(model_dirs):
    from swifttransformer_b200.engine.replay import TraceSession
    for name in CONFIGS:
        toks = helpers.random_tokens(CONFIGS[name]["cfg"]["vocab"], 29, seed=5)
        s = TraceSession(model_dirs[name], "float32", 64, page_size=CONFIGS[name]["page_size"], max_requests=1)
        s.runner.use_cuda_graphs = False
        got, order = [], s.model.layer_order
        s.model.after_layer = lambda i, stream: got.append(stream.x.cpu().numpy().copy()) if order[i].cache >= 0 else None
        s.run_step([dict(id="a", tokens=toks, want=[28])], ["a"])
        cfg, w = pd.load_model(model_dirs[name])
        _, ref = pd.forward(cfg, w, toks, return_layers=True)
        assert len(got) == len(ref)
        for i in range(len(ref)):
            assert np.abs(got[i] - ref[i]).max() < 2e-5 * np.abs(ref[i]).max(), (name, i)


def test_a_far_key_among_hundreds(model_dirs, tmp_path):
    """Two prompts that differ in their first token only.  In the model the two layers have no mask and a loud first
    token (its row of the embedding table), which every later position looks at: hundreds of tokens further the logits of
    the two still differ by far more than the tolerance, in a prompt, in portions and decoded."""
    from swifttransformer_b200.engine.replay import TraceSession
    from swifttransformer_b200.weights.safetensors_io import write_safetensors
    cfg = dict(architecture="Dimalix", vocab=80, width=48, norm={"eps": 1e-5}, embedding={"scale": 1.0}, layers=[
        att(4, 2, 16, 0.3, 0, None, dense(32)), lat(4, 16, 8, 16, 32, 0.3, 0, rot(4, 1e6), dense(32))])
    path = write_model(str(tmp_path / "far"), cfg, 7, 0.3)
    raw, w = pd.load_model(path)
    for t in (0, 1):
        w["embed"][t] *= 40.0                       # (the norms make a lone loud row no louder as a key, but its residual is)
    w["l0.mix.k"] *= 0.05
    w["l0.mix.k.b"] *= 0.05
    w["l0.mix.q.b"] *= 3.0
    write_safetensors(os.path.join(path, "model.safetensors"),
                      [(n, torch.tensor(t, dtype=torch.float32).to(torch.bfloat16)) for n, t in w.items()])
    _, w = pd.load_model(path)
    toks = helpers.random_tokens(80, 420, seed=8)
    toks = [t if t > 1 else t + 2 for t in toks]
    refs = {}
    for first in (0, 1):
        reqs = {f"p{first}": [first] + toks}
        refs[first] = pd.forward(raw, w, [first] + toks)
        for steps in (helpers.trace_whole(reqs), helpers.trace_portions(reqs), helpers.trace_decode_tail(reqs, tail=100)):
            s = TraceSession(path, "float32", 448, max_requests=1)
            got = helpers.replay(s, steps)[f"p{first}"]
            assert np.abs(got - refs[first]).max() < 3e-5 * np.abs(refs[first]).max()
    apart = np.abs(refs[0][300:] - refs[1][300:]).max(axis=1) / np.abs(refs[0]).max()
    assert apart.min() > 1e-3, apart.min()


@pytest.mark.parametrize("dtype", DTYPES)
def test_recorded_and_eager_steps_agree(model_dirs, dtype):
    from swifttransformer_b200.engine.replay import TraceSession
    reqs = requests_for("fast", lengths=(170, 9))
    steps = helpers.trace_mixed(reqs, seed=2, max_live=2, chunk=90)
    outs = []
    for graphs in (True, False):
        s = TraceSession(model_dirs["fast"], dtype, helpers.live_token_need(steps), max_requests=2)
        s.runner.use_cuda_graphs = graphs
        outs.append(helpers.replay(s, steps))
        assert (s.runner.graph_steps + s.runner.padded_graph_steps > 0) == graphs
    for rid in reqs:
        tol = 1e-5 if dtype == "float32" else 3e-2
        err = np.abs(outs[0][rid] - outs[1][rid]).max(axis=1) / np.abs(outs[1][rid]).max()
        assert err.max() < tol, (rid, int(np.argmax(err)), float(err.max()))


@pytest.mark.parametrize("dtype", DTYPES)
def test_unequal_requests_together_and_each_alone(model_dirs, dtype):
    from swifttransformer_b200.engine.replay import TraceSession
    reqs = requests_for("fast", lengths=(130, 1, 7, 66))
    s = TraceSession(model_dirs["fast"], dtype, 384, max_requests=4)
    together = s.run_step([dict(id=r, tokens=t, want=list(range(len(t)))) for r, t in reqs.items()], list(reqs)).cpu().numpy()
    at = 0
    for rid, toks in reqs.items():
        alone = s.run_step([dict(id=rid, tokens=toks, want=list(range(len(toks))))], [rid]).cpu().numpy()
        err = np.abs(together[at:at + len(toks)] - alone).max(axis=1) / np.abs(alone).max()
        assert err.max() < (1e-5 if dtype == "float32" else 5e-2), (rid, int(np.argmax(err)), float(err.max()))
        at += len(toks)


@pytest.mark.parametrize("name", ["mix", "fast"])
def test_long_decoding_with_pages_and_slots_used_again(model_dirs, name):
    """Three requests after one another through the same single slot and a pool that holds only one of them, each
    decoded token by token for 300 steps after a short prompt: chunks and windows pass over decoded tokens and their
    pages come back."""
    from swifttransformer_b200.engine.replay import TraceSession
    s = TraceSession(model_dirs[name], "float32", 384, page_size=CONFIGS[name]["page_size"], max_requests=1)
    for k in range(3):
        toks = helpers.random_tokens(CONFIGS[name]["cfg"]["vocab"], 330, seed=40 + k)
        rows = [s.run_step([dict(id=k, tokens=toks[:30], want=list(range(30)))]).cpu().numpy().copy()]
        for t in range(30, 330):
            rows.append(s.run_step([dict(id=k, tokens=[toks[t]], want=[0])], [k] if t == 329 else []).cpu().numpy().copy())
        s.check()
        ref = plain_logits(model_dirs[name], toks)
        bad = helpers.first_bad(np.concatenate(rows), ref, 3e-5 * np.abs(ref).max())
        assert bad is None, (k, bad)
    assert all(g.pool.num_held == 0 for g in s.cache.groups)


def test_windows_and_chunks_give_their_pages_back(model_dirs):
    """A model whose every attention has a mask holds, however long the request grows, only what its masks span."""
    from swifttransformer_b200.engine.replay import TraceSession
    s = TraceSession(model_dirs["mix"], "float32", 2048, page_size=8, max_requests=1)
    toks = helpers.random_tokens(300, 600, seed=9)
    s.run_step([dict(id=0, tokens=toks[:500], want=[])])
    assert max(g.pool.num_held for g in s.cache.groups) <= 50 // 8 + 2
    assert min(g.pool.num_held for g in s.cache.groups) <= 9 // 8 + 2
    got = s.run_step([dict(id=0, tokens=toks[500:], want=[99])]).cpu().numpy()
    ref = plain_logits(model_dirs["mix"], toks)
    assert np.abs(got[0] - ref[599]).max() < 3e-5 * np.abs(ref).max()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mix", "fast"])
def test_greedy_generation_through_the_engine(model_dirs, name, dtype):
    from swifttransformer_b200.engine.engine import LLMEngine
    from swifttransformer_b200.sampling.sampler import SamplingParams
    vocab = CONFIGS[name]["cfg"]["vocab"]
    prompts = [helpers.random_tokens(vocab, n, seed=n) for n in (5, 31, 1, 18, 44, 9)]
    eng = LLMEngine(model_dirs[name], dtype=dtype, page_size=CONFIGS[name]["page_size"], num_pages=24,
                    max_num_seqs=3, max_batch_tokens=48, chunk_size=20, max_seq_len=256)
    outs = eng.generate(prompts, SamplingParams(max_new_tokens=12, temperature=0.0))
    cfg, w = pd.load_model(model_dirs[name])
    off = 0
    for prompt, out in zip(prompts, outs):
        toks = list(prompt)
        tokens = list(out.output if hasattr(out, "output") else out)
        assert len(tokens) == 12
        for k, tok in enumerate(tokens):
            logits = pd.forward(cfg, w, toks)[-1]
            best = int(np.argmax(logits))
            if tok != best:
                assert dtype == "bfloat16", (name, k, tok, best)
                off += bool(logits[best] - logits[tok] > 0.08 * np.abs(logits).max())      # (another expert was chosen)
            toks.append(tok)
    assert off <= CONFIGS[name]["over"] * 12 * len(prompts), (name, off)


# ------------------------------------------------------------------------------------------ the programs
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def test_run_gpt_takes_a_dimalix_folder(model_dirs, tmp_path):
    import subprocess
    import sys
    vocab = CONFIGS["mix"]["cfg"]["vocab"]
    prompts = [helpers.random_tokens(vocab, n, 70 + n) for n in (6, 21)]
    inp = tmp_path / "in.txt"
    inp.write_text("\n".join(" ".join(map(str, p)) for p in prompts) + "\n")
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "run_gpt"), model_dirs["mix"], "any", "fp32", str(inp),
                        "--max_decoding_step", "5", "--num_total_blocks", "64"], capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    cfg, w = pd.load_model(model_dirs["mix"])
    lines = [l for l in r.stdout.splitlines() if l.startswith("[")]
    assert len(lines) == 2
    for line, p in zip(lines, prompts):
        got = [int(t) for t in line.split(")")[1].split("(")[0].split()]
        assert got == pd.greedy(cfg, w, p, 5)


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_run_program_with_four_slots(model_dirs, tmp_path, dtype):
    """bin/trace_run with its defaults (four request slots, pages of 16): six requests, at most four live, so slots and
    pages are handed out again; every wanted row against the plain implementation."""
    import subprocess
    import sys
    name = "fast"
    reqs = requests_for(name, lengths=(50, 1, 33, 170, 18, 40))
    steps = helpers.trace_mixed(reqs, seed=3, max_live=4)
    out = tmp_path / "out"
    p = subprocess.Popen([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", model_dirs[name], "--dtype", dtype,
                          "--out", str(out), "--max-tokens", str(helpers.live_token_need(steps))],
                         stdin=subprocess.PIPE, stdout=subprocess.PIPE, stderr=subprocess.PIPE, text=True)
    got = {rid: [] for rid in reqs}
    vocab = CONFIGS[name]["cfg"]["vocab"]
    for i, st in enumerate(steps):
        p.stdin.write(json.dumps(dict(st, step=i)) + "\n")
        p.stdin.flush()
        assert p.stdout.readline().strip() == f"done {i}", p.stderr.read()[-2000:]
        arr = np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(-1, vocab)
        k = 0
        for e in st["entries"]:
            got[e["id"]].append(arr[k:k + len(e["want"])])
            k += len(e["want"])
        assert k == len(arr)
    p.stdin.close()
    assert p.wait(timeout=120) == 0
    compare(model_dirs[name], reqs, {rid: np.concatenate(v) for rid, v in got.items()}, dtype, "trace_run",
            CONFIGS[name]["over"])
