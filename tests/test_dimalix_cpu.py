"""The Dimalix design's host side on the CPU: configuration, tensor names, the order of layer runs, cache entries and the
pages a chunk gives back, rotations stretched by wavelength, and the plain implementation's own mechanisms against closed
forms.  (What runs kernels is in test_dimalix_gpu.py.)"""
from __future__ import annotations

import copy
import json
import math

import numpy as np
import pytest
import torch

import plain_dimalix as pd
from swifttransformer_b200.cache.manager import CacheManager
from swifttransformer_b200.config import ConfigError, DimalixConfig, load_config
from swifttransformer_b200.models import build_model_def, write_random_model
from swifttransformer_b200.parts.base import BLOCKS, FEED_FORWARDS, MIXERS, NORMS, POSITION_ENCODINGS, PagedKVSpec


def raw_config():
    scaling = dict(factor=3.0, original=60, low=1.0, high=3.0)
    moe = {"kind": "moe", "expert": {"ff": 10},
           "router": {"experts": 7, "top": 2, "identity": 2, "groups": {"count": 3, "keep": 2}}}
    lat = {"type": "latent_attention", "mlp": {"kind": "dense", "ff": 40},
           "mixer": dict(heads=3, dim=10, rot_dim=6, vdim=7, kv_rank=20, scale=0.25, mask={"size": 9},
                         rot={"dims": 6, "base": 100.0})}
    att = {"type": "attention", "mlp": moe,
           "mixer": dict(heads=4, kv_heads=2, dim=8, vdim=8, scale=0.3, mask={"size": 20},
                         rot={"dims": 4, "base": 10.0, "scaling": scaling})}
    bare = {"type": "attention", "mlp": None, "mixer": dict(heads=2, kv_heads=2, dim=6, scale=0.3)}
    return dict(architecture="Dimalix", vocab=50, width=24, norm={"eps": 1e-5}, embedding={"scale": 2.5},
                loop={"start": 1, "stop": 3, "times": 3}, layers=[lat, att, bare, copy.deepcopy(lat)])


def test_config_round_trip_and_registry(tmp_path):
    cfg = DimalixConfig.from_dict(raw_config())
    assert cfg.norm_eps == 1e-5 and cfg.embedding_scale == 2.5 and cfg.loop == (1, 3, 3) and len(cfg.layers) == 4
    write_random_model(str(tmp_path), cfg, seed=0, std=0.1)
    again = load_config(str(tmp_path))
    assert isinstance(again, DimalixConfig) and again == DimalixConfig.from_dict(json.loads(json.dumps(cfg.to_dict())))
    pcfg, w = pd.load_model(str(tmp_path))
    assert np.isfinite(pd.forward(pcfg, w, [1, 2, 3, 4])).all()


@pytest.mark.parametrize("change,word", [
    (lambda c: c.pop("vocab"), "vocab"),
    (lambda c: c["norm"].update(eps=0), "norm.eps"),
    (lambda c: c["embedding"].pop("scale"), "embedding.scale"),
    (lambda c: c["loop"].pop("times"), "loop.times"),
    (lambda c: c["loop"].update(stop=5), "loop"),
    (lambda c: c["loop"].update(times=0), "loop"),
    (lambda c: c["layers"][0].update(type="window"), "type"),
    (lambda c: c["layers"][0]["mixer"].pop("kv_rank"), "mixer.kv_rank"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "mixer.scale"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=8), "rot.dims"),
    (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), "mask.size"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("low"), "scaling.low"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].update(high=0.5), "scaling.high"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "kv_heads"),
    (lambda c: c["layers"][1]["mixer"].update(vdim=12), "mixer.vdim"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=10), "router.top"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(identity=-1), "router.identity"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(identity=3), "router.groups"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].pop("keep"), "groups.keep"),
    (lambda c: c["layers"][1]["mlp"]["expert"].update(ff=-1), "expert.ff"),
    (lambda c: c["layers"][0]["mlp"].update(kind="routed"), "mlp.kind"),
])
def test_config_errors_name_the_key(change, word):
    raw = copy.deepcopy(raw_config())
    change(raw)
    with pytest.raises(ConfigError) as e:
        DimalixConfig.from_dict(raw)
    assert word in str(e.value)


def test_optional_groups_switch_their_mechanism_off():
    raw = raw_config()
    for key in ("loop", "embedding"):
        raw.pop(key)
    for key in ("mask", "rot"):
        raw["layers"][0]["mixer"].pop(key)
    raw["layers"][1]["mixer"]["rot"].pop("scaling")
    for key in ("groups", "identity"):
        raw["layers"][1]["mlp"]["router"].pop(key)
    mdef = build_model_def(DimalixConfig.from_dict(raw))
    lat, att, moe = mdef.blocks[0].mixer, mdef.blocks[1].mixer, mdef.blocks[1].feed_forward
    assert lat.window is None and lat.qk_position is None and att.chunk == 20 and att.qk_position.scaling is None
    assert moe.rule["groups"] is None and moe.n_identity == 0 and moe.n_outputs == 7 and mdef.embedding.scale == 1.0
    assert [s.block for s in mdef.layer_order] == [0, 1, 2, 3] and mdef.blocks[2].mixer.chunk is None


def test_tensor_names_shapes_and_cache_needs():
    mdef = build_model_def(DimalixConfig.from_dict(raw_config()))
    specs = {s.name: tuple(s.shape) for s in mdef.param_specs()}
    assert specs["embed"] == specs["head"] == (50, 24) and specs["final.norm"] == (24,)
    for i, two in enumerate((True, True, False, True)):
        assert specs[f"l{i}.norm1"] == specs[f"l{i}.ls1"] == (24,)
        assert (f"l{i}.norm2" in specs) == (f"l{i}.ls2" in specs) == two
    assert specs["l0.mix.q"] == (48, 24) and specs["l0.mix.dkv"] == (26, 24) and specs["l0.mix.dkv.norm"] == (20,)
    assert specs["l0.mix.uk"] == (30, 20) and specs["l0.mix.uv"] == (21, 20) and specs["l0.mix.o"] == (24, 21)
    assert specs["l0.mlp.up"] == (40, 24) and specs["l0.mlp.down"] == (24, 40) and "l0.mlp.gate" not in specs
    assert specs["l1.mix.q"] == (32, 24) and specs["l1.mix.q.b"] == specs["l1.mix.q.norm"] == (32,)
    assert specs["l1.mix.k"] == (16, 24) and specs["l1.mix.k.b"] == specs["l1.mix.k.norm"] == (16,) and "l1.mix.v" not in specs
    assert specs["l1.mix.o"] == (24, 32) and specs["l1.mlp.router"] == (9, 24) and specs["l1.mlp.correction"] == (9,)
    assert specs["l1.mlp.e6.gate"] == (10, 24) and "l1.mlp.e7.gate" not in specs
    # every run of a layer has an entry of its own
    lat, att, bare = PagedKVSpec(1, 26, 9, value_dim=0), PagedKVSpec(2, 8, value_dim=8, block=20), PagedKVSpec(2, 6, value_dim=6)
    assert mdef.cache_specs() == [lat] + [att, bare] * 3 + [lat]


def test_order_of_runs_and_where_passes_open():
    cfg = DimalixConfig.from_dict(raw_config())
    assert cfg.layer_runs() == [(0, False), (1, False), (2, False), (1, True), (2, False), (1, True), (2, False), (3, False)]
    assert pd.layer_runs(raw_config()) == cfg.layer_runs()
    mdef = build_model_def(cfg)
    again = len(mdef.blocks) - 1
    assert [s.block for s in mdef.layer_order] == [0, 1, 2, again, 1, 2, again, 1, 2, 3]
    assert [s.cache for s in mdef.layer_order] == [0, 1, 2, -1, 3, 4, -1, 5, 6, 7]


def test_unused_tensors_of_a_layer_without_feed_forward_are_passed_over():
    mdef = build_model_def(DimalixConfig.from_dict(raw_config()))
    assert mdef.canonical_name("l2.norm2") is None and mdef.canonical_name("l2.ls2") is None
    assert mdef.canonical_name("l1.norm2") == "l1.norm2"


def test_a_chunk_gives_its_pages_back():
    mdef = build_model_def(DimalixConfig.from_dict(raw_config()))
    m = CacheManager(mdef.cache_specs(), torch.float32, "cpu", page_size=8, num_pages=16, max_seqs=2, max_seq_len=96)
    s = m.alloc_slot()
    group = next(g for g in m.groups if g.spec.block == 20)
    for length, first in ((19, 0), (20, 2), (39, 2), (40, 5), (41, 5)):
        assert m.reserve(s, m.lengths[s], length)
        m.commit(s, length)
        # the next query's chunk begins at 20 * (length // 20): pages before that one's are gone
        assert min(group.pages[s], default=first) == first, length
    m.free_slot(s)
    m.check()


def test_parts_refuse_what_does_not_fit():
    mix = dict(hidden=8, num_heads=2, num_kv_heads=1, dim=4, scale=1.0, names={"q": "q", "k": "k", "o": "o"})
    with pytest.raises(ValueError):
        MIXERS.build("grouped_attention", vdim=6, values_are_keys=True, **mix)
    with pytest.raises(ValueError):
        MIXERS.build("grouped_attention", vdim=4, qk_norm_names=("a", "b"), **mix)
    with pytest.raises(ValueError):
        MIXERS.build("grouped_attention", vdim=4, chunk=0, **mix)
    names = [{k: f"e{e}.{k}" for k in ("gate", "up", "down")} for e in range(4)]
    ff = dict(hidden=8, inner=4, num_experts=4, activation="silu", expert_names=names, router_name="r")
    with pytest.raises(ValueError):
        FEED_FORWARDS.build("routed_experts", top=6, identity=1, **ff)
    with pytest.raises(ValueError):
        FEED_FORWARDS.build("routed_experts", top=2, identity=1, groups=(2, 1), **ff)
    assert FEED_FORWARDS.build("routed_experts", top=2, identity=2, groups=(2, 1), **ff).n_outputs == 6
    one = NORMS.build("rmsnorm", width=8, name="n")
    with pytest.raises(ValueError):
        BLOCKS.build("parallel_scaled", mixer=None, feed_forward=None, norm1=one, norm2=one, width=8, scale_names=("a", "b"))


# ------------------------------------------------------------------------------------------ rotations, the oracle
@pytest.mark.parametrize("dims,base,scaling", [(16, 100.0, None), (10, 5e5, dict(factor=8.0, original=500, low=1.0, high=4.0)),
                                               (40, 1e4, dict(factor=2.5, original=2048, low=2.0, high=6.0)),
                                               (12, 30.0, dict(factor=1.0, original=50, low=1.0, high=4.0)),
                                               (8, 1000.0, dict(factor=4.0, original=100, low=3.0, high=3.0))])
def test_frequencies_stretched_by_wavelength(dims, base, scaling):
    rot = dict(dims=dims, base=base, scaling=scaling)
    enc = POSITION_ENCODINGS.build("rotary_pairs", **rot)
    assert np.allclose(enc.frequencies(), pd.rotation_frequencies(rot), rtol=1e-12) and enc.amplitude == 1.0
    plain = pd.rotation_frequencies(dict(dims=dims, base=base))
    if scaling:
        got = np.asarray(enc.frequencies())
        wave = 2 * math.pi / plain
        fast, slow = wave < scaling["original"] / scaling["high"], wave > scaling["original"] / scaling["low"]
        assert np.array_equal(got[fast], plain[fast]) and np.allclose(got[slow], plain[slow] / scaling["factor"])
        between = ~(fast | slow)
        assert np.all(got[between] <= plain[between]) and np.all(got[between] >= plain[between] / scaling["factor"] - 1e-18)


def test_plain_frequency_in_the_middle():
    # one pair of frequency 1: wavelength 2 pi; original = 4 pi: two turns, half way between low 1 and high 3
    f = pd.rotation_frequencies(dict(dims=2, base=7.0, scaling=dict(factor=5.0, original=4 * math.pi, low=1.0, high=3.0)))
    assert np.allclose(f, 0.5 / 5.0 + 0.5)


def test_plain_masks():
    c = pd.seen_chunk(7, 3)
    assert c[2].tolist() == [True] * 3 + [False] * 4 and c[3].tolist() == [False] * 3 + [True] + [False] * 3
    assert c[6].tolist() == [False] * 6 + [True]
    assert pd.seen_window(6, 2)[4].tolist() == [False] * 3 + [True, True, False]
    assert pd.seen_chunk(3, None).tolist() == np.tril(np.ones((3, 3), bool)).tolist()


def test_plain_values_are_keys_before_norm_and_rotation():
    rng = np.random.default_rng(0)
    mx = dict(heads=2, kv_heads=1, dim=4, rot=dict(dims=2, base=10.0))
    w = {"q": rng.normal(size=(8, 5)), "q.b": rng.normal(size=8), "k": rng.normal(size=(4, 5)), "k.b": rng.normal(size=4),
         "q.norm": rng.normal(size=8), "k.norm": rng.normal(size=4)}
    h = rng.normal(size=(3, 5))
    q, k, v = pd.grouped_qkv(h, w, "", mx, 1e-5, [0, 1, 2])
    raw = h @ w["k"].T + w["k.b"]
    assert np.allclose(v[:, 0], raw)
    want = raw[0] / np.sqrt(np.mean(raw[0] ** 2) + 1e-5) * w["k.norm"]
    assert np.allclose(k[0, 0], want)                                  # position 0 is not turned
    qr = (h @ w["q"].T + w["q.b"])[0]
    assert np.allclose(q[0].reshape(-1), qr / np.sqrt(np.mean(qr ** 2) + 1e-5) * w["q.norm"])


def test_plain_routing_with_corrections():
    z = np.log(np.array([[0.4, 0.1, 0.2, 0.3]]))
    # choice scores 0.4 - 0.9, 0.1 - 0.05, 0.2 - 0.5, 0.3 - 0.45: all but one negative
    b = np.array([-0.9, -0.05, -0.5, -0.45])
    chosen, w = pd.route(z, b, dict(top=2))
    assert chosen.tolist() == [[1, 3]] and np.allclose(w, [[0.25, 0.75]])
    # groups by their largest choice score: {-0.5, 0.05} before {-0.3, -0.15}; a left-out group never counts as 0
    chosen, w = pd.route(z, b, dict(top=2, groups=dict(count=2, keep=1)))
    assert chosen.tolist() == [[1, 0]] and np.allclose(w, [[0.2, 0.8]])


def test_plain_identity_experts_and_layer_scale():
    rng = np.random.default_rng(1)
    W = 4
    w = {"e0.gate": rng.normal(size=(3, W)), "e0.up": rng.normal(size=(3, W)), "e0.down": rng.normal(size=(W, 3)),
         "router": np.zeros((2, W)), "correction": np.zeros(2)}
    h = rng.normal(size=(2, W))
    out = pd.experts_ff(h, w, "", dict(router=dict(experts=1, identity=1, top=2)))
    assert np.allclose(out, 0.5 * pd.expert(h, w, "e0.") + 0.5 * h)
    w["correction"] = np.array([0.0, 5.0])
    assert np.allclose(pd.experts_ff(h, w, "", dict(router=dict(experts=1, identity=1, top=1))), h)
    assert np.isclose(pd.gelu_tanh(np.array(1.0)), 0.841192, atol=1e-6)
