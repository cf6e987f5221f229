"""The Nigilorn design on the GPU against the plain implementation (tests/plain_nigilorn.py).

Mechanisms alone (the kernels driven directly, with inputs made so that a single key, an edge, a state or a group
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
import plain_nigilorn as pn

pytestmark = pytest.mark.gpu

DTYPES = ["float32", "bfloat16"]
TD = {"float32": torch.float32, "bfloat16": torch.bfloat16}


def dev(a, dtype=torch.float32):
    return torch.tensor(np.asarray(a), dtype=dtype, device="cuda")


def ints(a):
    return torch.tensor(np.asarray(a), dtype=torch.int32, device="cuda")


def host(t):
    return t.float().cpu().numpy().astype(np.float64)


def bf16_round(a):
    return torch.tensor(np.asarray(a), dtype=torch.float32).to(torch.bfloat16).double().numpy()


class Step:
    """The index arrays of one step for (slot, start, n) entries, with padding tokens at position -1 and padding
    requests behind, as the step function lays them out."""

    def __init__(self, entries, pad_tokens=0, pad_requests=0):
        pos, seq, q_start, slots, starts = [], [], [0], [], []
        for i, (slot, start, n) in enumerate(entries):
            pos += list(range(start, start + n))
            seq += [i] * n
            q_start.append(q_start[-1] + n)
            slots.append(slot)
            starts.append(start)
        self.n = len(pos)
        pos += [-1] * pad_tokens
        seq += [0] * pad_tokens
        q_start += [self.n] * pad_requests
        slots += [0] * pad_requests
        starts += [0] * pad_requests
        self.lens = np.array([n for _, _, n in entries], dtype=np.int32)
        self.n_rows, self.n_seqs = len(pos), len(entries) + pad_requests
        self.positions, self.seq, self.q_start, self.slots = ints(pos), ints(seq), ints(q_start), ints(slots)
        self.start_pos = ints(starts)


def portions(total, sizes):
    out, pos, k = [], 0, 0
    while pos < total:
        n = min(sizes[k % len(sizes)], total - pos)
        out.append((pos, n))
        pos += n
        k += 1
    return out


# ------------------------------------------------------------------------------------------ rotations
ROTS = [  # head size, rotated dimensions, base, scaling
    (16, 16, 100.0, None),
    (24, 10, 9000.0, dict(factor=4.0, original=300, fast=8.0, slow=1.0)),
    (40, 40, 2e5, dict(factor=8.0, original=2048, fast=32.0, slow=2.0)),
    (12, 4, 30.0, dict(factor=2.0, original=20, fast=50.0, slow=40.0)),     # the ramp's two ends fall together
    (8, 2, 7.0, dict(factor=3.0, original=64, fast=1.0, slow=1.0)),
]


@pytest.mark.parametrize("d,dims,base,scaling", ROTS)
def test_frequencies_of_stretched_contexts(d, dims, base, scaling):
    from swifttransformer_b200.parts.base import POSITION_ENCODINGS
    enc = POSITION_ENCODINGS.build("rotary_pairs", dims=dims, base=base, scaling=scaling)
    freq, amp = pn.rotation_frequencies(dict(dims=dims, base=base, scaling=scaling))
    assert np.allclose(enc.frequencies(), freq, rtol=1e-12) and abs(enc.amplitude - amp) < 1e-12
    if scaling:
        plain, _ = pn.rotation_frequencies(dict(dims=dims, base=base))
        assert amp > 1.0 and np.all(freq <= plain) and np.all(freq >= plain / scaling["factor"] - 1e-15)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("norm", [True, False])
@pytest.mark.parametrize("d,dims,base,scaling", ROTS)
def test_queries_and_keys_turn_in_neighbouring_pairs(d, dims, base, scaling, norm, dtype):
    """Queries and cached keys from a fused projection: rotation with amplitude, then the division by the root mean
    square; positions far out; the values pass."""
    from swifttransformer_b200 import ops
    rng = np.random.default_rng(d * dims)
    H, G, vd, ps, eps = 4, 2, 6, 4, 3e-2
    rot = dict(dims=dims, base=base, scaling=scaling)
    freq, amp = pn.rotation_frequencies(rot)
    start, T = 1003, 9
    width = H * d + G * (d + vd)
    proj = bf16_round(rng.normal(size=(T + 1, width)))
    st = Step([(1, start, T)], pad_tokens=1)
    table = np.full((2, (start + T) // ps + 1), -1, dtype=np.int32)
    need = np.arange(start // ps, (start + T - 1) // ps + 1)
    table[1, need] = rng.permutation(len(need))
    pool = torch.zeros((len(need), 1, G * ps * (d + vd)), dtype=TD[dtype], device="cuda")
    q = torch.zeros((T + 1, H * d), dtype=TD[dtype], device="cuda")
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    ops.gqa_prepare(dev(proj, TD[dtype]), 0, H * d, (H + G) * d, None, dev(freq), dims, 0.0, 1, q, pool, 0, st.positions,
                    st.seq, st.slots, ints(table), H, G, d, vd, ps, status, norm_eps=eps if norm else 0.0, neighbours=True,
                    rot_amp=amp)
    assert int(status.item()) == 0
    pos = np.arange(start, start + T)
    unit = (lambda u: pn.rms_unit(u, eps)) if norm else (lambda u: u)
    rq = unit(pn.rotate_neighbours(proj[:T, :H * d].reshape(T, H, d), pos, rot))
    rk = unit(pn.rotate_neighbours(proj[:T, H * d:(H + G) * d].reshape(T, G, d), pos, rot))
    tol = (2e-4 if dtype == "float32" else 1.5e-2)        # float angles at positions in the thousands
    assert np.abs(host(q)[:T].reshape(T, H, d) - rq).max() < tol * np.abs(rq).max() and np.all(host(q)[T] == 0)
    flat = host(pool)[:, 0]
    keys, vals = flat[:, :G * ps * d].reshape(-1, G, ps, d), flat[:, G * ps * d:].reshape(-1, G, ps, vd)
    for t in range(T):
        page, at = table[1, (start + t) // ps], (start + t) % ps
        assert np.abs(keys[page, :, at] - rk[t]).max() < tol * np.abs(rk).max()
        assert np.abs(vals[page, :, at] - proj[t, (H + G) * d:].reshape(G, vd)).max() < 1e-6


# ------------------------------------------------------------------------------------------ attention over pages
class Pages:
    """Block tables of several requests whose pages are dealt out of order, with spare pages nobody owns."""

    def __init__(self, lengths, ps, rng):
        per = [(n + ps - 1) // ps for n in lengths]
        self.lengths, self.ps, self.n_pages = list(lengths), ps, sum(per) + 3
        order = rng.permutation(self.n_pages)
        self.table = np.full((len(lengths) + 1, max(per) + 1), -1, dtype=np.int32)
        self.slot = [len(lengths) - i for i in range(len(lengths))]
        at = 0
        for i, c in enumerate(per):
            self.table[self.slot[i], :c] = order[at:at + c]
            at += c

    def without_passed_pages(self, i, pos, window):
        """The table once a window has passed: what a query at ``pos`` cannot see any more is gone."""
        table = self.table.copy()
        if window:
            table[self.slot[i], :max(0, pos - window + 1) // self.ps] = -1
        return table

    def each(self, i):
        for p in range(self.lengths[i]):
            yield p, self.table[self.slot[i], p // self.ps], p % self.ps


class GroupedCase:
    """Grouped attention with one gate number per head; unused rows of the pool hold large numbers."""

    def __init__(self, lengths, H, G, d, vd, ps, window, seed, dtype):
        rng = np.random.default_rng(seed)
        self.H, self.G, self.d, self.vd, self.ps, self.window, self.dtype = H, G, d, vd, ps, window, dtype
        self.pages, self.lengths = Pages(lengths, ps, rng), list(lengths)
        self.q = [bf16_round(rng.normal(size=(n, H, d))) for n in lengths]
        self.k = [bf16_round(rng.normal(size=(n, G, d))) for n in lengths]
        self.v = [bf16_round(rng.normal(size=(n, G, vd))) for n in lengths]
        self.gate = [bf16_round(rng.normal(size=(n, H))) for n in lengths]
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
        o = pn.attend(self.q[i], self.k[i], self.v[i], pn.seen_window(self.lengths[i], self.window or None), self.scale)
        return (o * pn.sigmoid(self.gate[i])[:, :, None]).reshape(self.lengths[i], -1)

    def kernels(self):
        from swifttransformer_b200 import ops
        probe = torch.zeros(1, dtype=TD[self.dtype], device="cuda")
        fast = ops.gqa_attention_fast_applies(probe, self.H, self.G, self.d, self.vd)
        return ["plain", "items"] + (["tiles", "single"] if fast else [])

    def run(self, entries, kernel, pad_tokens=0, table=None):
        from swifttransformer_b200 import ops
        H, G, d, vd = self.H, self.G, self.d, self.vd
        st = Step([(self.pages.slot[i], s, n) for i, s, n in entries], pad_tokens=pad_tokens)
        cut = lambda rows, fill: np.concatenate([rows[i][s:s + n].reshape(n, -1) for i, s, n in entries]
                                                + [np.full((pad_tokens, rows[0][0].size), fill)])
        q = dev(cut(self.q, 50.0), TD[self.dtype])
        wide = torch.zeros((st.n_rows, H + 13), dtype=TD[self.dtype], device="cuda")     # gate logits at an odd column
        wide[:, 3:3 + H] = dev(cut(self.gate, 0.0), TD[self.dtype])
        out = torch.full((st.n_rows, H * vd), 77.0, dtype=TD[self.dtype], device="cuda")
        status = torch.zeros(1, dtype=torch.int32, device="cuda")
        bt = ints(self.pages.table if table is None else table)
        tail = (H, G, d, vd, self.ps, self.scale, self.window, 0, None, wide, 3, 1.0)
        kw = dict(status=status, gate_heads=True)
        args = (q, self.pool, 1, out)
        rows = (st.positions, st.seq, st.slots, bt)
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


class LatentCase:
    """Attention in the latent space under a window: keys and values are the cached latents."""

    def __init__(self, lengths, H, kr, rot, ps, window, seed, dtype):
        rng = np.random.default_rng(seed)
        self.H, self.kr, self.rot, self.ps, self.window, self.dtype = H, kr, rot, ps, window, dtype
        self.pages, self.lengths = Pages(lengths, ps, rng), list(lengths)
        self.q = [bf16_round(rng.normal(size=(n, H, kr + rot))) for n in lengths]
        self.k = [bf16_round(rng.normal(size=(n, 1, kr + rot))) for n in lengths]
        self.scale = 0.9 / np.sqrt(kr + rot)

    def write(self):
        P, ps, kd = self.pages.n_pages, self.ps, self.kr + self.rot
        rows = np.full((P, ps, kd), 3e4)
        for i in range(len(self.lengths)):
            for p, page, at in self.pages.each(i):
                rows[page, at] = self.k[i][p, 0]
        pool = np.full((P, 2, ps * kd), 3e4)
        pool[:, 1] = rows.reshape(P, -1)
        self.pool = dev(pool, TD[self.dtype])

    def reference(self, i):
        seen = pn.seen_window(self.lengths[i], self.window or None)
        return pn.attend(self.q[i], self.k[i], self.k[i][..., :self.kr], seen, self.scale).reshape(self.lengths[i], -1)

    def kernels(self):
        from swifttransformer_b200 import ops
        probe = torch.zeros(1, dtype=TD[self.dtype], device="cuda")
        fast = ops.latent_attention_mma_applies(probe, self.kr, self.rot)
        return ["plain"] + (["mma", "mma1", "mma7"] if fast else [])

    def run(self, entries, kernel, pad_tokens=0, table=None):
        from swifttransformer_b200 import ops
        st = Step([(self.pages.slot[i], s, n) for i, s, n in entries], pad_tokens=pad_tokens, pad_requests=1)
        q = np.concatenate([self.q[i][s:s + n].reshape(n, -1) for i, s, n in entries]
                           + [np.full((pad_tokens, self.q[0][0].size), 50.0)])
        out = torch.full((st.n_rows, self.H * self.kr), 77.0, dtype=TD[self.dtype], device="cuda")
        status = torch.zeros(1, dtype=torch.int32, device="cuda")
        bt = ints(self.pages.table if table is None else table)
        kw = {} if kernel == "plain" else dict(q_start=st.q_start, start_pos=st.start_pos, n_seqs=st.n_seqs,
                                               n_splits={"mma": None, "mma1": 1, "mma7": 7}[kernel])
        ops.latent_attention(dev(q, TD[self.dtype]), self.pool, 1, out, st.positions, st.seq, st.slots, bt, self.H, self.kr,
                             self.rot, self.ps, self.scale, status=status, kernel=kernel[:3] if kernel != "plain" else kernel,
                             window=self.window, **kw)
        return split(out, entries, st, status)


def split(out, entries, st, status):
    assert int(status.item()) == 0, entries
    o = host(out)
    assert np.all(o[st.n:] == 77.0)
    res, at = {}, 0
    for i, s, n in entries:
        res[i] = o[at:at + n]
        at += n
    return res


GROUPED = [  # H, G, d, vd, page size, window
    (6, 2, 16, 24, 8, 21), (4, 4, 32, 8, 16, 0), (8, 1, 64, 72, 4, 64), (3, 3, 12, 20, 16, 7), (16, 4, 40, 48, 32, 130),
    (1, 1, 8, 8, 8, 1), (20, 2, 24, 16, 8, 50), (2, 1, 128, 160, 16, 100)]
LATENT = [  # H, kr, rot, page size, window
    (5, 32, 8, 8, 21), (3, 48, 16, 16, 0), (16, 64, 32, 4, 64), (2, 20, 6, 16, 7), (7, 160, 24, 32, 130), (1, 16, 0, 8, 1),
    (70, 32, 8, 16, 33), (4, 512, 64, 16, 40)]


def make_case(kind, shape, lengths, seed, dtype):
    if kind == "grouped":
        H, G, d, vd, ps, window = shape
        return GroupedCase(lengths, H, G, d, vd, ps, window, seed, dtype)
    H, kr, rot, ps, window = shape
    return LatentCase(lengths, H, kr, rot, ps, window, seed, dtype)


SHAPES = [("grouped", s) for s in GROUPED] + [("latent", s) for s in LATENT]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind,shape", SHAPES)
def test_windowed_attention_whole_batched_in_portions_and_decoded(kind, shape, dtype):
    c = make_case(kind, shape, (150, 1, 37, 203), seed=shape[0] + shape[1], dtype=dtype)
    c.write()
    refs = [c.reference(i) for i in range(len(c.lengths))]
    top = max(np.abs(r).max() for r in refs)
    tol = (1e-5 if dtype == "float32" else 2e-2) * top
    for kernel in c.kernels():
        whole = c.run([(i, 0, n) for i, n in enumerate(c.lengths)], kernel, pad_tokens=3)
        for i, r in enumerate(refs):
            assert np.abs(whole[i] - r).max() < tol, (kernel, i)
        alone = c.run([(3, 0, 203)], kernel)
        assert np.abs(alone[3] - whole[3]).max() < tol
        for start, n in portions(203, (70, 2, 5, 33, 2)):
            table = c.pages.without_passed_pages(3, start, c.window)
            got = c.run([(0, 120, 1), (3, start, n)], kernel, table=table)
            assert np.abs(got[3] - refs[3][start:start + n]).max() < tol, (kernel, start, n)
            assert np.abs(got[0] - refs[0][120:121]).max() < tol
        for pos in (0, 1, c.ps - 1, c.ps, 100, 201, 202):
            got = c.run([(3, pos, 1), (2, 36, 1)], kernel, pad_tokens=1, table=c.pages.without_passed_pages(3, pos, c.window))
            assert np.abs(got[3] - refs[3][pos:pos + 1]).max() < tol, (kernel, pos)
            assert np.abs(got[2] - refs[2][36:37]).max() < tol


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind,shape", [("grouped", (4, 2, 32, 16, 8, 24)), ("latent", (4, 32, 8, 8, 24)),
                                        ("grouped", (3, 1, 16, 8, 16, 100)), ("latent", (3, 48, 16, 16, 100))])
def test_one_loud_key_just_inside_and_just_outside_the_window(kind, shape, dtype):
    """A key that takes all the weight wherever it is seen: the result is its value inside the window and knows nothing
    of it one position further; in prompt rows and decoded tokens, at page borders and at the request's first tokens."""
    T = 160
    window, ps = shape[-1], shape[-2]
    for loud in (0, 1, ps - 1, ps, 3 * ps, 50):
        c = make_case(kind, shape, (T,), seed=loud + 1, dtype=dtype)
        vector = np.ones(c.k[0].shape[-1]) * 3.0
        c.k[0][loud] = vector
        c.q[0][:] = bf16_round(c.q[0] * 0.1 + vector * (12.0 / (9.0 * vector.size) / c.scale))
        c.write()
        ref = c.reference(0)
        last_in, first_out = min(T - 1, loud + window - 1), loud + window
        value = np.tile((c.v[0][loud] if kind == "grouped" else c.k[0][loud][:, :c.kr]), (c.H // (c.G if kind == "grouped" else 1), 1))
        tol = (2e-5 if dtype == "float32" else 2e-2) * np.abs(ref).max()
        for kernel in c.kernels():
            whole = c.run([(0, 0, T)], kernel)[0]
            assert np.abs(whole - ref).max() < tol
            for pos in [p for p in (loud, last_in, first_out, first_out + 1) if p < T]:
                one = c.run([(0, pos, 1)], kernel, table=c.pages.without_passed_pages(0, pos, window))[0]
                assert np.abs(one - ref[pos]).max() < tol, (kernel, loud, pos)
        if first_out < T and kind == "latent":
            # the edge itself shows: the loud key's value is (nearly) the result at the last position that sees it
            assert np.abs(ref[last_in].reshape(c.H, -1) - value).max() < 0.2 * np.abs(value).max()
            assert np.abs(ref[first_out].reshape(c.H, -1) - value).max() > 0.5 * np.abs(value).max()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,d,rot,e,kr,dims,window", [(3, 12, 6, 10, 20, 6, 9), (4, 32, 16, 24, 48, 16, 30), (2, 8, 8, 8, 16, 8, 0)])
def test_latent_mixer_with_direct_queries(H, d, rot, e, kr, dims, window, dtype):
    """The mixer with a cache of its own: projections, rotated parts, latent cache, window and output, in portions and
    decoded, and the columns of its first product that belong to its block."""
    from swifttransformer_b200.cache.manager import CacheManager
    from swifttransformer_b200.parts.base import MIXERS, POSITION_ENCODINGS
    rng = np.random.default_rng(H * d)
    W, T, eps, ps = 40, 61, 1e-5, 4
    scaling = dict(factor=2.0, original=40, fast=6.0, slow=1.0)
    mx = dict(heads=H, dim=d, rot_dim=rot, vdim=e, kv_rank=kr, scale=0.3, rot=dict(dims=dims, base=500.0, scaling=scaling))
    if window:
        mx["mask"] = {"size": window}
    w = {"q": rng.normal(size=(H * (d + rot), W)) * 0.3, "dkv": rng.normal(size=(kr + rot, W)) * 0.3,
         "dkv.norm": 1 + 0.1 * rng.normal(size=kr), "uk": rng.normal(size=(H * d, kr)) * 0.3,
         "uv": rng.normal(size=(H * e, kr)) * 0.3, "o": rng.normal(size=(W, H * e)) * 0.3}
    w = {k: bf16_round(v) for k, v in w.items()}
    h, extra = bf16_round(rng.normal(size=(T, W))), bf16_round(rng.normal(size=(W, W)) * 0.2)
    m = MIXERS.build("latent_attention", hidden=W, num_heads=H, dim=d, rot=rot, vdim=e, kv_rank=kr, q_rank=0, scale=0.3,
                     eps=eps, names={k: k for k in ("q", "dkv", "uk", "uv", "o")} | {"kv_norm": "dkv.norm"}, window=window,
                     qk_position=POSITION_ENCODINGS.build("rotary_pairs", **mx["rot"]), float_out=True)
    assert m.take_rows(dev(extra, TD[dtype]))
    m.bind({k: dev(v, torch.float32 if v.ndim == 1 else TD[dtype]) for k, v in w.items()})
    ref, ref_extra = pn.latent_attention(h, w, "", mx, eps), h @ extra.T
    tol = 2e-5 if dtype == "float32" else 3e-2
    for cuts in ([(0, T)], portions(T, (7, 2, 1, 13, 1))):
        cache = CacheManager([m.cache_spec()], TD[dtype], "cuda", page_size=ps, num_pages=24, max_seqs=2, max_seq_len=96)
        slot, got = cache.alloc_slot(), []
        for start, n in cuts:
            assert cache.reserve(slot, start, start + n)
            g = cache.groups[0]
            for at, page in g.take_updates():
                g.block_table.view(-1)[at] = page
            st = Step([(slot, start, n)], pad_tokens=1, pad_requests=1)

            class Ctx:
                positions, seq_of_token, slots, q_start, start_pos, n_seqs = (st.positions, st.seq, st.slots, st.q_start,
                                                                              st.start_pos, st.n_seqs)
                status = torch.zeros(1, dtype=torch.int32, device="cuda")
                scratch_f32 = staticmethod(lambda n: torch.empty(n, dtype=torch.float32, device="cuda"))
            rows = dev(np.concatenate([h[start:start + n], np.zeros((1, W))]), TD[dtype])
            delta = m.forward(rows, Ctx, cache.entries()[0].view())
            assert int(Ctx.status.item()) == 0 and delta.value.dtype == torch.float32
            got.append(host(delta.value)[:n])
            assert np.abs(host(delta.extra)[:n] - ref_extra[start:start + n]).max() < tol * np.abs(ref_extra).max()
            cache.commit(slot, start + n)
        err = np.abs(np.concatenate(got) - ref).max(axis=1)
        assert err.max() < tol * np.abs(ref).max(), (cuts[:3], int(np.argmax(err)), float(err.max()))


# ------------------------------------------------------------------------------------------ convolution and scan
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("channels,taps", [(20, 4), (33, 2), (64, 1), (12, 8), (128, 5), (8, 3)])
def test_convolution_inside_a_mixer(channels, taps, dtype):
    """Bias and activation, first columns of a wider projection; unequal requests in one step, in portions shorter and
    longer than the filter, token by token, in steps long enough for several tokens per thread; padding and other slots
    are left alone."""
    from swifttransformer_b200 import ops
    rng = np.random.default_rng(channels + taps)
    lens = (330, 9, 41)
    xs = [bf16_round(rng.normal(size=(n, channels))) for n in lens]
    w, b = rng.normal(size=(channels, taps)), rng.normal(size=channels)
    refs = [pn.silu(pn.causal_conv(x, w.astype(np.float32).astype(np.float64), b)) for x in xs]
    tol = (2e-5 if dtype == "float32" else 1e-2) * max(np.abs(r).max() for r in refs)
    plans = [[[(0, 0, 330), (1, 0, 9), (2, 0, 41)]],
             [[(1, 0, 2), (2, 0, 1), (0, 0, 300)], [(0, 300, 30), (2, 1, 3), (1, 2, 7)], [(2, 4, 37)]],
             [[(0, 0, 1)], [(0, 1, 2)], [(0, 3, 7), (2, 0, 2)], [(2, 2, 39), (0, 10, 320)]]]
    plans.append([[(i, t, 1) for i in range(3) if t < lens[i]] for t in range(41)])
    for steps in plans:
        state = torch.zeros((5, taps - 1, channels), device="cuda")
        state[4] = 7.0
        for entries in steps:
            st = Step([(i + 1, s, n) for i, s, n in entries], pad_tokens=2, pad_requests=1)
            rows = np.concatenate([xs[i][s:s + n] for i, s, n in entries] + [np.full((2, channels), 9.0)])
            wide = dev(np.concatenate([rows, np.full((len(rows), 8), 55.0)], axis=1), TD[dtype])
            single = all(n == 1 for _, _, n in entries)
            out = host(ops.conv_act(wide, channels, dev(w), dev(b), "silu", state, st.positions, st.seq, st.q_start, st.slots,
                                    move_state=single))
            if taps > 1 and not single:
                ops.conv_state_update(wide, channels, state, st.positions, st.q_start, st.slots, st.n_seqs)
            at = 0
            for i, s, n in entries:
                err = np.abs(out[at:at + n] - refs[i][s:s + n]).max(axis=1)
                assert err.max() < tol, (entries, i, s + int(np.argmax(err)))
                at += n
        assert taps == 1 or (float(state[0].abs().max()) == 0.0 and torch.all(state[4] == 7.0))


class ScanCase:
    def __init__(self, C, N, R, lens, seed, dtype, slow=0.0):
        rng = np.random.default_rng(seed)
        self.C, self.N, self.R, self.lens, self.dtype = C, N, R, list(lens), dtype
        self.R8 = (R + 7) // 8 * 8
        self.u = [bf16_round(rng.normal(size=(n, C))) for n in lens]
        self.z = [bf16_round(rng.normal(size=(n, C))) for n in lens]
        f32 = lambda a: np.asarray(a, dtype=np.float32).astype(np.float64)
        self.r = [bf16_round(rng.normal(size=(n, R))) for n in lens]
        self.b, self.g = [f32(rng.normal(size=(n, N))) for n in lens], [f32(rng.normal(size=(n, N))) for n in lens]
        self.w_dt = bf16_round(rng.normal(size=(C, R)) * 0.4)
        self.bias, self.D = f32(rng.normal(size=C) * 0.5 - 1.0), f32(rng.normal(size=C))
        self.a_log = f32(rng.normal(size=(C, N)) * 0.7 - slow)

    def reference(self, i):
        dt = pn.softplus(self.r[i] @ self.w_dt.T + self.bias)
        y, S = pn.selective_scan(self.u[i], dt, self.a_log, self.b[i], self.g[i], self.D)
        return y * pn.silu(self.z[i]), S

    def run(self, steps, chunk=None, n_slots=6):
        """Steps of (request, start, n) entries; request i lives in slot i + 1.  -> (outputs per request, states)."""
        from swifttransformer_b200 import ops
        from swifttransformer_b200.parts.mamba import TokenChunkPlan
        T, C, N, R8 = TD[self.dtype], self.C, self.N, self.R8
        state = torch.zeros((n_slots, C, N), device="cuda")
        state[n_slots - 1] = 7.0
        A = dev(-np.exp(self.a_log))
        w_dt = torch.zeros((C, R8), dtype=T, device="cuda")
        w_dt[:, :self.R] = dev(self.w_dt, T)
        outs = [np.zeros((n, C)) for n in self.lens]
        for entries in steps:
            st = Step([(i + 1, s, n) for i, s, n in entries], pad_tokens=2, pad_requests=1)
            cat = lambda rows, fill: np.concatenate([rows[i][s:s + n] for i, s, n in entries] + [np.full((2, rows[0].shape[1]), fill)])
            x = dev(cat(self.u, 9.0), T)
            proj = dev(np.concatenate([np.full((st.n_rows, 5), 3.0), cat(self.z, 9.0)], axis=1), T)
            xd = torch.zeros((st.n_rows, R8 + 2 * N), device="cuda")
            xd[:, :self.R], xd[:, R8:R8 + N], xd[:, R8 + N:] = dev(cat(self.r, 9.0)), dev(cat(self.b, 9.0)), dev(cat(self.g, 9.0))
            out = torch.full((st.n_rows, C), 77.0, dtype=T, device="cuda")
            tail = (A, dev(self.D), dev(self.bias), state, out, st.positions)
            if all(n == 1 for _, _, n in entries) and chunk is None:
                ops.mamba_single(x, xd, R8, R8 + N, w_dt, proj, 5, *tail, st.seq, st.slots)
            else:
                dt = dev(cat(self.r, 9.0) @ self.w_dt.T)
                plan = TokenChunkPlan(chunk or ops.MAMBA_CHUNK)
                words = np.zeros(plan.words(st.n_rows, st.n_seqs), dtype=np.int32)
                key = plan.fill(st.lens, None, None, words, st.n_rows, st.n_seqs)
                if key[0]:
                    key = plan.shape_key(st.lens, None, st.n_rows, st.n_seqs)      # as a recorded step has it: padded
                v = plan.view(ints(words), key, st.n_rows, st.n_seqs)
                scratch = torch.full((ops.mamba_scan_scratch(v.n_chunks, C, N),), 1e30, device="cuda") if v.n_chunks else None
                ops.mamba_scan(x, dt, xd, R8, R8 + N, proj, 5, *tail, st.q_start, st.slots, st.n_seqs, chunks=v.chunks,
                               chunk_first=v.first, n_chunks=v.n_chunks, chunk=v.chunk, scratch=scratch)
            o, at = host(out), 0
            assert np.all(o[st.n:] == 77.0)
            for i, s, n in entries:
                outs[i][s:s + n] = o[at:at + n]
                at += n
        assert torch.all(state[n_slots - 1] == 7.0) and float(state[0].abs().max()) == 0.0
        return outs, host(state)


SCANS = [(20, 4, 3, 4), (33, 7, 8, 16), (130, 16, 12, 64), (64, 20, 5, 32), (24, 33, 16, 8), (12, 70, 1, 64), (6, 130, 9, 16),
         (5, 1, 2, 8), (256, 8, 24, 64)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("C,N,R,chunk", SCANS)
def test_scan_in_chunks_portions_and_token_by_token(C, N, R, chunk, dtype):
    c = ScanCase(C, N, R, (137, 1, 64, 18), seed=C + N, dtype=dtype)
    refs = [c.reference(i) for i in range(4)]
    tol = (3e-5 if dtype == "float32" else 1.5e-2)
    whole = [[(i, 0, n) for i, n in enumerate(c.lens)]]
    cut = [[(0, s, n)] for s, n in portions(137, (70, 2, 1, 33, 1, 2, 5))] + [[(3, 0, 2), (2, 0, 40)], [(1, 0, 1), (2, 40, 24), (3, 2, 16)]]
    single = [[(i, t, 1) for i in range(4) if t < c.lens[i]] for t in range(137)]
    for steps, ch in ((whole, chunk), (whole, 1000), (cut, chunk), (cut, 1000), (single, None), (single[:30] + [[(0, 30, 107)]], chunk)):
        outs, state = c.run(steps, ch)
        for i, (ref, S) in enumerate(refs):
            upto = max(s + n for st in steps for j, s, n in st if j == i)
            err = np.abs(outs[i][:upto] - ref[:upto]).max(axis=1)
            assert err.max() < tol * np.abs(ref).max(), (ch, len(steps), i, int(np.argmax(err)), float(err.max()))
            if upto == c.lens[i]:
                assert np.abs(state[i + 1] - S).max() < max(tol, 2e-3 if dtype == "bfloat16" else 0) * np.abs(S).max()


def test_scan_remembers_a_far_token():
    """Slow decays and one loud token near the start: 500 tokens later the read-out is still made of it; a state that is
    lost at a chunk's, a portion's or a step's edge would be empty."""
    c = ScanCase(16, 8, 4, (520,), seed=3, dtype="float32", slow=7.0)
    c.u[0][1:] *= 0.01
    c.u[0][0] *= 5.0
    c.D[:] = 0.0
    ref, _ = c.reference(0)
    c2 = ScanCase(16, 8, 4, (520,), seed=3, dtype="float32", slow=7.0)
    c2.u[0][1:] *= 0.01
    c2.u[0][0] = 0.0
    c2.D[:] = 0.0
    blank, _ = c2.reference(0)
    assert np.abs(ref[-1] - blank[-1]).max() > 0.3 * np.abs(ref[-1]).max()
    for steps, ch in (([[(0, 0, 520)]], 64), ([[(0, s, n)] for s, n in portions(520, (130, 1, 64, 65, 2))], 64),
                      ([[(0, t, 1)] for t in range(520)], None)):
        outs, _ = c.run(steps, ch)
        assert np.abs(outs[0][-1] - ref[-1]).max() < 1e-4 * np.abs(ref).max(), ch


# ------------------------------------------------------------------------------------------ residual arrangement
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [20, 64, 33, 2048, 2056, 4100, 8192, 9001])
def test_gate_norm_and_residual_sum_in_one_kernel(width, dtype):
    """x + N(sigmoid(g + b) y; w) and what reads x next; with and without gate, with the next norm, a copy or nothing;
    results in float and in the activation type; padding rows are left alone."""
    from swifttransformer_b200 import ops
    rng = np.random.default_rng(width)
    T, eps, eps2 = 7, 1e-3, 1e-2
    x, y = rng.normal(size=(T, width)), bf16_round(rng.normal(size=(T, width)) * 0.01)
    g, b = bf16_round(rng.normal(size=(T, width)) * 2), rng.normal(size=width)
    w, w2 = 1 + 0.2 * rng.normal(size=width), 1 + 0.2 * rng.normal(size=width)
    pos = ints(list(range(T - 1)) + [-1])
    for gated in (True, False):
        new = x + pn.rms_unit(y * pn.sigmoid(g + b) if gated else y, eps) * w
        for nxt in ("norm", "copy", "none"):
            for y_dtype in {torch.float32, TD[dtype]}:
                wide = torch.zeros((T, width + 8), dtype=TD[dtype], device="cuda")
                wide[:, :width] = dev(g, TD[dtype])
                gate = wide[:, :width] if gated else None
                xd = dev(x)
                act = torch.full((T, width), 5.0, dtype=TD[dtype], device="cuda") if nxt != "none" else None
                if act is None and not gated and y_dtype != torch.float32 and dtype == "float32":
                    continue
                ops.gated_norm_add(xd, dev(y, y_dtype), gate, dev(b) if gated else None, dev(w), eps, pos,
                                   dev(w2) if nxt == "norm" else None, eps2, act)
                got = host(xd)
                assert np.abs(got[:-1] - new[:-1]).max() < 2e-5 * np.abs(new).max() and np.abs(got[-1] - x[-1]).max() < 1e-6
                if act is not None:
                    ref = pn.rms_unit(new, eps2) * w2 if nxt == "norm" else new
                    tol = 2e-5 if dtype == "float32" else 5e-3
                    assert np.abs(host(act)[:-1] - ref[:-1]).max() < tol * np.abs(ref).max() and np.all(host(act)[-1] == 5.0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("layers,dim", [(3, 5), (1, 16), (4, 64)])
def test_input_by_token(layers, dim, dtype):
    from swifttransformer_b200 import ops
    rng = np.random.default_rng(layers * dim)
    T, V = 21, 13
    table, s, ids = bf16_round(rng.normal(size=(V, layers * dim))), rng.normal(size=(T, dim)) * 2, rng.integers(0, V, T)
    for i in range(layers):
        got = host(ops.side_input(dev(s), dev(table, TD[dtype]), i * dim, ints(ids)))
        ref = pn.gelu_tanh(s) * table[ids][:, i * dim:(i + 1) * dim]
        assert np.abs(got - ref).max() < (1e-5 if dtype == "float32" else 1e-2) * np.abs(ref).max()
    x = rng.normal(size=(T, 11))
    assert np.abs(host(ops.slice_rows(dev(x), 3, 6, TD[dtype])) - x[:, 3:9]).max() < (1e-6 if dtype == "float32" else 2e-2)


# ------------------------------------------------------------------------------------------ routing and experts
ROUTERS = [  # experts, top, groups (count, keep), scale
    (12, 3, (4, 2), 2.5), (6, 6, None, 1.0), (16, 2, (16, 5), 1.0), (9, 1, (3, 1), 0.5), (64, 8, (8, 3), 3.0), (10, 4, (2, 1), 1.5),
    (1, 1, None, 2.0), (70, 5, (35, 20), 1.0)]


@pytest.mark.parametrize("E,top,groups,scale", ROUTERS)
def test_group_limited_choice(E, top, groups, scale):
    """The choice from a product's logits, and from the hidden rows themselves, against the plain router."""
    from swifttransformer_b200 import ops
    rng = np.random.default_rng(E * top)
    T, W = 90, 24
    wr, h = bf16_round(rng.normal(size=(E, W)) * 0.4), bf16_round(rng.normal(size=(T, W)))
    router = dict(experts=E, top=top, scale=scale, **({"groups": dict(count=groups[0], keep=groups[1])} if groups else {}))
    chosen, weights = pn.route(h, wr, router)
    pos = ints(list(range(T - 1)) + [-1])
    rule = dict(renorm=True, scores="sigmoid", groups=groups, scale=scale)
    z = np.concatenate([h @ wr.T, np.full((T, 3), 9.0)], axis=1)
    for experts, got in (ops.moe_choose(dev(z), E, top, pos, **rule),
                         ops.moe_route(dev(h), dev(wr), top, pos, None, **rule)[:2],
                         ops.moe_route(dev(h, torch.bfloat16), dev(wr), top, pos, None, **rule)[:2]):
        e = experts.cpu().numpy()
        assert np.array_equal(e[:-1], chosen[:-1]) and np.all(e[-1] == -1)
        assert np.abs(host(got)[:-1] - weights[:-1]).max() < 1e-5 * max(scale, 1)


def test_group_score_is_the_sum_of_the_two_largest():
    """The group with the single largest score loses to the one whose two largest add up to more, and its best expert
    cannot be chosen; a group of one expert counts that one."""
    from swifttransformer_b200 import ops
    logit = lambda p: float(np.log(p / (1 - p)))
    z = np.array([[logit(p) for p in (0.9, 0.1, 0.1, 0.6, 0.55, 0.05)]])
    experts, w = ops.moe_choose(dev(z), 6, 2, None, renorm=True, scores="sigmoid", groups=(2, 1), scale=1.0)
    assert experts.cpu().tolist() == [[3, 4]] and np.allclose(host(w), [[0.6 / 1.15, 0.55 / 1.15]], atol=1e-6)
    experts, w = ops.moe_choose(dev(z), 6, 2, None, renorm=False, scores="sigmoid", groups=(6, 2), scale=3.0)
    assert experts.cpu().tolist() == [[0, 3]] and np.allclose(host(w), [[2.7, 1.8]], atol=1e-5)


class PartCtx:
    def __init__(self, T):
        self.positions = ints(list(range(T)) + [-1])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T", [5, 70])
@pytest.mark.parametrize("E,top,groups,ff,shared", [(12, 3, (4, 2), 24, 40), (4, 2, None, 20, 0), (8, 1, (2, 1), 64, 24)])
def test_squared_relu_experts_with_a_shared_one(E, top, groups, ff, shared, T, dtype):
    from swifttransformer_b200.parts.base import FEED_FORWARDS
    rng = np.random.default_rng(E * ff + T)
    W = 40
    w = {"router": bf16_round(rng.normal(size=(E, W)))}
    for e in [f"e{i}" for i in range(E)] + (["shared"] if shared else []):
        n = shared if e == "shared" else ff
        w[e + ".up"], w[e + ".down"] = bf16_round(rng.normal(size=(n, W)) * 0.4), bf16_round(rng.normal(size=(W, n)) * 0.3)
    h = bf16_round(rng.normal(size=(T, W)))
    router = dict(experts=E, top=top, scale=1.7, **({"groups": dict(count=groups[0], keep=groups[1])} if groups else {}))
    ref = pn.experts_ff(h, w, "", {"router": router, "expert": {"ff": ff}, "shared": {"ff": shared} if shared else None})
    sh = FEED_FORWARDS.build("dense", hidden=W, inner=shared, activation="relu2", bias=False, fc1_name="shared.up",
                             fc2_name="shared.down", weight_suffix="") if shared else None
    part = FEED_FORWARDS.build("routed_experts", hidden=W, inner=ff, num_experts=E, top=top, activation="relu2", gated=False,
                               expert_names=[{k: f"e{e}.{k}" for k in ("up", "down")} for e in range(E)], router_name="router",
                               shared=sh, renormalise=True, scores="sigmoid", groups=groups, scale=1.7)
    tensors = {k: dev(v, torch.float32 if k == "router" else TD[dtype]) for k, v in w.items()}
    for p in [part] + part.children():
        p.bind(tensors)
    got = host(part.forward(dev(np.concatenate([h, np.zeros((1, W))]), TD[dtype]), PartCtx(T)).value)[:T]
    assert np.abs(got - ref).max() < (2e-5 if dtype == "float32" else 2e-2) * np.abs(ref).max()


# ------------------------------------------------------------------------------------------ whole models
def rot(dims, base, factor=None, original=64, fast=8.0, slow=1.0):
    r = {"dims": dims, "base": base}
    if factor:
        r["scaling"] = {"factor": factor, "original": original, "fast": fast, "slow": slow}
    return r


def lat(heads, dim, rot_dim, vdim, kr, scale, size, r, mlp):
    mx = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kr, scale=scale)
    mx.update({"mask": {"size": size}} if size else {}, **({"rot": r} if r else {}))
    return {"type": "latent_attention", "mixer": mx, "mlp": mlp}


def att(heads, kv, dim, vdim, scale, size, r, mlp):
    mx = dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=scale)
    mx.update({"mask": {"size": size}} if size else {}, **({"rot": r} if r else {}))
    return {"type": "attention", "mixer": mx, "mlp": mlp}


def ssm(inner, state, rank, conv, mlp):
    return {"type": "mamba1", "mixer": dict(inner=inner, state=state, dt_rank=rank, conv=conv), "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, groups=None, scale=1.0, shared=0):
    r = {"experts": experts, "top": top, "scale": scale}
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": r, **({"shared": {"ff": shared}} if shared else {})}


# (``over``: the share of positions that may be further off in bfloat16 because a token went to another expert; in "fast"
# the only layer that chooses between experts is the last one, so that nothing carries a choice on)
CONFIGS = {
    # sizes that are multiples of nothing; the scan first; windows that differ and pass over prompts and decoded
    # tokens; a layer without feed-forward
    "mix": dict(cfg=dict(architecture="Nigilorn", vocab=300, width=44, norm={"eps": 1e-5}, token_side={"dim": 6}, layers=[
        ssm(50, 9, 5, 3, moe(9, 3, 20, (3, 2), 1.5, 28)),
        lat(3, 10, 6, 7, 22, 0.3, 12, rot(6, 100.0, 3.0), dense(40)),
        att(4, 2, 12, 10, 0.4, 9, rot(4, 50.0, 2.0, 40), None),
        ssm(36, 20, 3, 5, dense(30)),
        att(3, 3, 6, 5, 0.6, 33, rot(6, 10.0), moe(4, 1, 12, None, 0.7))]), seed=41, std=0.1, page_size=8, over=0.35),
    # sizes that the tensor-core kernels take; a window longer than a tile of queries
    "fast": dict(cfg=dict(architecture="Nigilorn", vocab=200, width=64, norm={"eps": 3e-6}, token_side={"dim": 24}, layers=[
        lat(8, 16, 8, 24, 64, 0.2, 40, rot(8, 1e4, 4.0, 128), moe(4, 4, 32, (2, 2), 2.5, 48)),
        ssm(96, 16, 8, 4, dense(64)),
        lat(4, 32, 16, 8, 32, 0.2, 150, rot(16, 500.0, 2.0), None),
        att(8, 2, 32, 16, 0.25, 130, rot(16, 3e5, 2.0, 512, 32.0), moe(16, 4, 16, (8, 4), 1.0, 16))]), seed=42, std=0.12,
                 page_size=16, over=0.15),
    # one head, one expert, one tap, a state of one number, no input by token, no mask, no rotation, a window of one
    "lone": dict(cfg=dict(architecture="Nigilorn", vocab=64, width=20, norm={"eps": 1e-4}, layers=[
        att(1, 1, 4, 3, 0.5, 1, rot(2, 3.0), moe(1, 1, 8)),
        ssm(7, 1, 1, 1, None),
        lat(1, 4, 2, 6, 5, 0.5, 0, None, dense(16)),
        lat(2, 3, 0, 4, 9, 0.5, 5, None, moe(3, 2, 8, (3, 2), 3.0, 4)),
        att(3, 1, 6, 6, 0.5, 0, None, moe(2, 2, 4))]), seed=43, std=0.25, page_size=4, over=0.1),
}


def louder(name, t, std):
    """Random weights under which faults show: decays so slow that the state remembers for hundreds of tokens, loud
    routers, gate and step biases as large as their products."""
    f = t.float()
    if name.endswith(".A_log"):
        return f - 3.5
    if name.endswith(".router"):
        return f * 3             # (much louder ones would saturate the sigmoids, and every choice would be a near tie)
    if name.endswith(".D"):
        return 1.0 + f
    if name.endswith(".b") and t.dim() == 1:
        return f * 3
    if name.endswith((".conv", "side.embed")):
        return f / std * 0.5
    return f


def write_model(path, cfg_dict, seed, std):
    from swifttransformer_b200.config import NigilornConfig, save_config
    from swifttransformer_b200.models import build_model_def
    from swifttransformer_b200.weights.random_init import random_tensors
    from swifttransformer_b200.weights.safetensors_io import write_safetensors
    cfg = NigilornConfig.from_dict(cfg_dict)
    save_config(cfg, path)
    tensors = [(s.name, louder(s.name, t, std).to(torch.bfloat16))
               for s, t in random_tensors(build_model_def(cfg).param_specs(), seed, std, "cpu")]
    write_safetensors(os.path.join(path, "model.safetensors"), tensors)
    return path


@pytest.fixture(scope="module")
def model_dirs(tmp_path_factory):
    root = tmp_path_factory.mktemp("nigilorn")
    return {name: write_model(str(root / name), c["cfg"], c["seed"], c["std"]) for name, c in CONFIGS.items()}


_PLAIN = {}


def plain_logits(model_dir, tokens):
    key = (model_dir, tuple(tokens))
    if key not in _PLAIN:
        if model_dir not in _PLAIN:
            _PLAIN[model_dir] = pn.load_model(model_dir)
        cfg, w = _PLAIN[model_dir]
        _PLAIN[key] = pn.forward(cfg, w, tokens)
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


def test_residual_stream_after_every_layer(model_dirs):
    from swifttransformer_b200.engine.replay import TraceSession
    for name in CONFIGS:
        toks = helpers.random_tokens(CONFIGS[name]["cfg"]["vocab"], 29, seed=5)
        s = TraceSession(model_dirs[name], "float32", 64, page_size=CONFIGS[name]["page_size"], max_requests=1)
        s.runner.use_cuda_graphs = False
        got = []
        s.model.after_layer = lambda i, stream: got.append(stream.x.cpu().numpy().copy())
        s.run_step([dict(id="a", tokens=toks, want=[28])], ["a"])
        cfg, w = pn.load_model(model_dirs[name])
        _, ref = pn.forward(cfg, w, toks, return_layers=True)
        assert len(got) == len(ref)
        for i in range(len(ref)):
            assert np.abs(got[i] - ref[i]).max() < 2e-5 * np.abs(ref[i]).max(), (name, i)


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


@pytest.mark.parametrize("name", ["mix", "fast"])
def test_long_decoding_with_pages_and_slots_used_again(model_dirs, name):
    """Three requests after one another through the same single slot and a pool that holds only one of them, each
    decoded token by token for 300 steps after a short prompt: windows pass over decoded tokens, their pages come back,
    and the next request starts from zero states in the slot the last one left."""
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


def test_windows_give_their_pages_back(model_dirs):
    """A model whose every attention has a window holds, however long the request grows, only the window's pages."""
    from swifttransformer_b200.engine.replay import TraceSession
    s = TraceSession(model_dirs["mix"], "float32", 2048, page_size=8, max_requests=1)
    toks = helpers.random_tokens(300, 600, seed=9)
    s.run_step([dict(id=0, tokens=toks[:500], want=[])])
    assert max(g.pool.num_held for g in s.cache.groups) <= 33 // 8 + 2
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
    cfg, w = pn.load_model(model_dirs[name])
    off = 0
    for prompt, out in zip(prompts, outs):
        toks = list(prompt)
        tokens = list(out.output if hasattr(out, "output") else out)
        assert len(tokens) == 12
        for k, tok in enumerate(tokens):
            logits = pn.forward(cfg, w, toks)[-1]
            best = int(np.argmax(logits))
            if tok != best:
                assert dtype == "bfloat16", (name, k, tok, best)
                off += bool(logits[best] - logits[tok] > 0.08 * np.abs(logits).max())      # (another expert was chosen)
            toks.append(tok)
    assert off <= CONFIGS[name]["over"] * 12 * len(prompts), (name, off)


# ------------------------------------------------------------------------------------------ the programs
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def test_run_gpt_takes_a_nigilorn_folder(model_dirs, tmp_path):
    import subprocess
    import sys
    vocab = CONFIGS["mix"]["cfg"]["vocab"]
    prompts = [helpers.random_tokens(vocab, n, 70 + n) for n in (6, 21)]
    inp = tmp_path / "in.txt"
    inp.write_text("\n".join(" ".join(map(str, p)) for p in prompts) + "\n")
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "run_gpt"), model_dirs["mix"], "any", "fp32", str(inp),
                        "--max_decoding_step", "5", "--num_total_blocks", "64"], capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    cfg, w = pn.load_model(model_dirs["mix"])
    lines = [l for l in r.stdout.splitlines() if l.startswith("[")]
    assert len(lines) == 2
    for line, p in zip(lines, prompts):
        got = [int(t) for t in line.split(")")[1].split("(")[0].split()]
        assert got == pn.greedy(cfg, w, p, 5)


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
