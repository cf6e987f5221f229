"""The Nigilorn design's host side on the CPU: configuration, tensor names, cache entries, the plan that cuts portions
into chunks, the stacking of a block's rows onto its sub-layers' products, and the plain implementation's own mechanisms
against closed forms.  (What runs kernels is in test_nigilorn_gpu.py.)"""
from __future__ import annotations

import copy
import json

import numpy as np
import pytest
import torch

import plain_nigilorn as pn
from swifttransformer_b200.cache.manager import CacheManager, PagedCacheView, StateView
from swifttransformer_b200.config import ConfigError, NigilornConfig, load_config
from swifttransformer_b200.models import build_model_def, write_random_model
from swifttransformer_b200.parts.base import POSITION_ENCODINGS, PagedKVSpec, StateSpec, stack_rows
from swifttransformer_b200.parts.mamba import TokenChunkPlan


def raw_config():
    scaling = dict(factor=2.0, original=50, fast=8.0, slow=1.0)
    moe = {"kind": "moe", "expert": {"ff": 10}, "shared": {"ff": 14},
           "router": {"experts": 6, "top": 2, "scale": 1.5, "groups": {"count": 3, "keep": 2}}}
    lat = {"type": "latent_attention", "mlp": {"kind": "dense", "ff": 40},
           "mixer": dict(heads=3, dim=10, rot_dim=6, vdim=7, kv_rank=20, scale=0.25, mask={"size": 9},
                         rot={"dims": 6, "base": 100.0, "scaling": scaling})}
    ssm = {"type": "mamba1", "mlp": moe, "mixer": dict(inner=36, state=5, dt_rank=3, conv=4)}
    att = {"type": "attention", "mlp": None,
           "mixer": dict(heads=4, kv_heads=2, dim=8, vdim=12, scale=0.3, mask={"size": 20}, rot={"dims": 4, "base": 10.0})}
    return dict(architecture="Nigilorn", vocab=50, width=24, norm={"eps": 1e-5}, token_side={"dim": 4},
                layers=[lat, ssm, att, copy.deepcopy(ssm)])


def test_config_round_trip_and_registry(tmp_path):
    cfg = NigilornConfig.from_dict(raw_config())
    assert cfg.norm_eps == 1e-5 and cfg.side_dim == 4 and len(cfg.layers) == 4
    write_random_model(str(tmp_path), cfg, seed=0, std=0.1)
    again = load_config(str(tmp_path))
    assert isinstance(again, NigilornConfig) and again == NigilornConfig.from_dict(json.loads(json.dumps(cfg.to_dict())))
    pcfg, w = pn.load_model(str(tmp_path))
    assert np.isfinite(pn.forward(pcfg, w, [1, 2, 3, 4])).all()


@pytest.mark.parametrize("change,word", [
    (lambda c: c.pop("vocab"), "vocab"),
    (lambda c: c["norm"].update(eps=0), "norm.eps"),
    (lambda c: c["token_side"].update(dim=0), "token_side.dim"),
    (lambda c: c["layers"][0].update(type="window"), "type"),
    (lambda c: c["layers"][0]["mixer"].pop("kv_rank"), "mixer.kv_rank"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "mixer.scale"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=8), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("slow"), "scaling.slow"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(base=1.0), "rot.base"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "mask.size"),
    (lambda c: c["layers"][1]["mixer"].pop("dt_rank"), "mixer.dt_rank"),
    (lambda c: c["layers"][1]["mixer"].update(conv=9), "mixer.conv"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=7), "router.top"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(count=4), "router.groups"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].pop("keep"), "groups.keep"),
    (lambda c: c["layers"][1]["mlp"]["shared"].update(ff=-1), "shared.ff"),
    (lambda c: c["layers"][2]["mixer"].update(kv_heads=3), "kv_heads"),
    (lambda c: c["layers"][0]["mlp"].update(kind="routed"), "mlp.kind"),
])
def test_config_errors_name_the_key(change, word):
    raw = copy.deepcopy(raw_config())
    change(raw)
    with pytest.raises(ConfigError) as e:
        NigilornConfig.from_dict(raw)
    assert word in str(e.value)


def test_optional_groups_switch_their_mechanism_off():
    raw = raw_config()
    raw.pop("token_side")
    raw["layers"][0]["mixer"].pop("mask")
    raw["layers"][0]["mixer"].pop("rot")
    raw["layers"][1]["mlp"].pop("shared")
    raw["layers"][1]["mlp"]["router"].pop("groups")
    raw["layers"][1]["mlp"]["router"].pop("scale")
    mdef = build_model_def(NigilornConfig.from_dict(raw))
    lat, moe = mdef.blocks[0].mixer, mdef.blocks[1].feed_forward
    assert lat.window is None and lat.qk_position is None and mdef.blocks[2].mixer.window == 20
    assert moe.shared is None and moe.rule["groups"] is None and moe.rule["scale"] == 1.0
    names = {s.name for s in mdef.param_specs()}
    assert not any("side" in n or "shared" in n for n in names if n.startswith(("l0", "side", "l1")))


def test_tensor_names_shapes_and_cache_needs():
    mdef = build_model_def(NigilornConfig.from_dict(raw_config()))
    specs = {s.name: tuple(s.shape) for s in mdef.param_specs()}
    assert specs["embed"] == specs["head"] == (50, 24) and specs["final.norm"] == (24,) and specs["side.embed"] == (50, 16)
    for i, two in enumerate((True, True, False, True)):
        want = ["norm1", "norm1b", "rg1", "rg1.b"] + (["norm2", "norm2b", "rg2", "rg2.b"] if two else [])
        assert all(f"l{i}.{n}" in specs for n in want) and (f"l{i}.rg2" in specs) == two
        assert specs[f"l{i}.side.gate"] == (4, 24) and specs[f"l{i}.side.proj"] == (24, 4) and specs[f"l{i}.side.norm"] == (24,)
    assert specs["l0.rg1"] == (24, 24) and specs["l0.rg1.b"] == (24,)
    assert specs["l0.mix.q"] == (48, 24) and specs["l0.mix.dkv"] == (26, 24) and specs["l0.mix.dkv.norm"] == (20,)
    assert specs["l0.mix.uk"] == (30, 20) and specs["l0.mix.uv"] == (21, 20) and specs["l0.mix.o"] == (24, 21)
    assert specs["l1.mix.in"] == (72, 24) and specs["l1.mix.conv"] == (36, 4) and specs["l1.mix.conv.b"] == (36,)
    assert specs["l1.mix.x"] == (13, 36) and specs["l1.mix.dt"] == (36, 3) and specs["l1.mix.dt.b"] == (36,)
    assert specs["l1.mix.A_log"] == (36, 5) and specs["l1.mix.D"] == (36,) and specs["l1.mix.o"] == (24, 36)
    assert specs["l1.mlp.router"] == (6, 24) and specs["l1.mlp.e5.up"] == (10, 24) and specs["l1.mlp.shared.down"] == (24, 14)
    assert "l1.mlp.e0.gate" not in specs and specs["l0.mlp.gate"] == (40, 24)
    assert specs["l2.mix.g"] == (4, 24) and specs["l2.mix.v"] == (24, 24) and "l2.mix.q.b" not in specs
    assert mdef.cache_specs() == [PagedKVSpec(1, 26, 9, value_dim=0), (StateSpec((3, 36)), StateSpec((36, 5))),
                                  PagedKVSpec(2, 8, 20, value_dim=12), (StateSpec((3, 36)), StateSpec((36, 5)))]


def test_cache_entries_and_zeroed_slots():
    mdef = build_model_def(NigilornConfig.from_dict(raw_config()))
    m = CacheManager(mdef.cache_specs(), torch.float32, "cpu", page_size=4, num_pages=16, max_seqs=2, max_seq_len=64)
    lat, (conv, state), att, (conv2, state2) = [e.view() for e in m.entries()]
    assert isinstance(lat, PagedCacheView) and isinstance(att, PagedCacheView) and lat.block_table is not att.block_table
    assert isinstance(state, StateView) and state.state is not state2.state and conv.state.shape == (2, 3, 36)
    s = m.alloc_slot()
    for v in (conv, state, conv2, state2):
        v.state[s].fill_(1.0)
    m.free_slot(s)
    assert m.alloc_slot() == s and all(float(v.state[s].abs().sum()) == 0.0 for v in (conv, state, conv2, state2))


def test_chunks_do_not_cross_requests_and_padding_lies_past_every_request():
    plan = TokenChunkPlan(8)
    lens = np.array([20, 1, 8, 9], dtype=np.int32)
    n_cap, b_cap = 48, 6
    words = np.full(plan.words(n_cap, b_cap), 99, dtype=np.int32)
    assert plan.fill(lens, None, None, words, n_cap, b_cap) == (7,)
    key = plan.shape_key(lens, None, n_cap, b_cap)
    v = plan.view(torch.tensor(words), key, n_cap, b_cap)
    chunks = v.chunks.view(-1, 2).tolist()
    assert key == (12,) and v.n_chunks == 12 and v.chunk == 8
    assert chunks[:7] == [[0, 0], [0, 8], [0, 16], [1, 0], [2, 0], [3, 0], [3, 8]]
    assert all(c == [0, TokenChunkPlan.PAD_OFFSET] for c in chunks[7:])
    assert v.first.tolist() == [0, 3, 4, 5, 7, 7, 7]
    # portions that all fit one chunk: none are made, whatever the step's padding
    short = np.array([8, 1, 2], dtype=np.int32)
    assert plan.shape_key(short, None, 64, 4) == (0,) and plan.fill(short, None, None, words, 48, 6) == (0,)
    assert plan.view(torch.tensor(words), (0,), 48, 6).chunks is None
    # a recording's first run holds no request at all: nothing but padding
    words[:] = 99
    plan.fill(np.zeros(0, dtype=np.int32), None, None, words, n_cap, b_cap)
    v = plan.view(torch.tensor(words), key, n_cap, b_cap)
    assert all(c == [0, TokenChunkPlan.PAD_OFFSET] for c in v.chunks.view(-1, 2).tolist()) and v.first.tolist() == [0] * 7


def test_a_blocks_rows_ride_in_its_sublayers_products():
    a, b = torch.arange(15.0).view(5, 3), torch.ones(8, 3)
    w, off = stack_rows([a, b, a])
    assert w.shape == (24, 3) and off == [0, 8, 16] and torch.equal(w[:5], a) and torch.all(w[5:8] == 0) and torch.equal(w[16:21], a)
    mdef = build_model_def(NigilornConfig.from_dict(raw_config()))
    tensors = {s.name: torch.randn(s.made_shape()) for s in mdef.param_specs()}
    rg = {i: tensors[f"l{i}.rg1"] for i in range(4)}
    rg2 = tensors["l1.rg2"]
    for p in mdef.all_parts():
        p.bind(tensors)
    for i, blk in enumerate(mdef.blocks):
        m = blk.mixer
        assert blk.gate_w[0] is None and m.extra_n == 24 and m.extra_off % 8 == 0 and m.extra_rows is None
        assert torch.equal(m.w_in[m.extra_off:m.extra_off + 24], rg[i])
    assert mdef.blocks[0].gate_w[1] is None and mdef.blocks[0].feed_forward.extra_n == 24
    assert torch.equal(mdef.blocks[1].gate_w[1], rg2)          # a mixture leaves the product to the block


# ------------------------------------------------------------------------------------------ the oracle's own mechanisms
def test_plain_rotation_pairs_window_and_stretching():
    seen = pn.seen_window(12, 4)
    assert seen[11].tolist() == [False] * 8 + [True] * 4 and seen[2].tolist() == [True] * 3 + [False] * 9
    e0 = np.zeros((1, 1, 6))
    e0[..., 2] = 1.0
    r = pn.rotate_neighbours(e0, [1], dict(dims=4, base=100.0))[0, 0]
    assert np.allclose(r, [0, 0, np.cos(0.1), np.sin(0.1), 0, 0])
    # without a ramp between them the pairs before the border keep their frequency, those behind turn `factor` slower
    sc = dict(factor=4.0, original=1000.0, fast=20.0, slow=20.0)
    freq, amp = pn.rotation_frequencies(dict(dims=16, base=1000.0, scaling=sc))
    plain, one = pn.rotation_frequencies(dict(dims=16, base=1000.0))
    assert one == 1.0 and np.isclose(amp, 1 + 0.1 * np.log(4.0))
    border = 16 * np.log(1000 / (2 * np.pi * 20)) / (2 * np.log(1000))
    assert np.allclose(freq[:int(np.floor(border)) + 1], plain[:int(np.floor(border)) + 1]) and np.allclose(freq[-3:], plain[-3:] / 4)
    enc = POSITION_ENCODINGS.build("rotary_pairs", dims=16, base=1000.0, scaling=sc)
    assert np.allclose(enc.frequencies(), freq) and enc.neighbours
    assert not POSITION_ENCODINGS.build("rotary_halves", dims=4, base=10.0).neighbours


def test_plain_scan_convolution_and_activations():
    # one channel, one state number: S <- exp(-d e^a) S + d x b
    y, S = pn.selective_scan(np.array([[2.0], [0.0]]), np.array([[1.0], [0.5]]), np.array([[0.0]]), np.array([[3.0], [9.0]]),
                             np.array([[1.0], [2.0]]), np.array([10.0]))
    assert np.allclose(y[:, 0], [6.0 + 20.0, 2 * 6.0 * np.exp(-0.5)]) and np.allclose(S, 6.0 * np.exp(-0.5))
    u = np.array([[1.0, 10.0], [2.0, 20.0], [3.0, 30.0]])
    assert np.allclose(pn.causal_conv(u, np.array([[0.0, 1.0], [2.0, 3.0]]), np.array([0.5, 0.0])), [[1.5, 30], [2.5, 80], [3.5, 130]])
    assert pn.relu2(np.array([-2.0, 3.0])).tolist() == [0.0, 9.0] and np.isclose(pn.gelu_tanh(np.array(1.0)), 0.841192, atol=1e-6)


def test_plain_routing_by_groups():
    logit = lambda p: np.log(p / (1 - p))
    w = np.array([[logit(p)] for p in (0.9, 0.1, 0.6, 0.55)])
    chosen, weights = pn.route(np.array([[1.0]]), w, dict(top=2, scale=3.0, groups=dict(count=2, keep=1)))
    assert chosen.tolist() == [[2, 3]] and np.allclose(weights, [[3 * 0.6 / 1.15, 3 * 0.55 / 1.15]])
    chosen, weights = pn.route(np.array([[1.0]]), w, dict(top=2))
    assert chosen.tolist() == [[0, 2]] and np.allclose(weights.sum(), 1.0)


def test_plain_sublayer_gate_and_norms():
    w = {"n": np.ones(4), "g": np.zeros((4, 4)), "g.b": np.array([0.0, 50.0, 0.0, 50.0]), "m": np.full(4, 2.0)}
    x = np.array([[1.0, -1.0, 1.0, -1.0]])
    out = pn.sublayer(x, lambda h: h * 3.0, w, "n", "g", "m", 0.0)
    u = np.array([1.5, -3.0, 1.5, -3.0])
    assert np.allclose(out, x + 2.0 * u / np.sqrt(np.mean(u * u)))
