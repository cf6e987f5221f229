"""Dimalix put together from the parts.

A decoder-only model whose layers are listed in the configuration:

  embedding     x = embed[token] * embedding.scale
  layer i       x <- x + (ls1 * mixer(N(x; norm1)) + ls2 * ff(N(x; norm2)))             (block ``parallel_scaled``)
  mixers        'latent_attention': queries straight from the input, keys and values from one normed latent per token,
                a rotated key part shared by the heads, a window          (``latent_attention`` with q_rank 0, window)
                'attention': grouped attention whose values are its keys as projected, q and k normed over the whole
                projection before the rotation, chunks                    (``grouped_attention`` with values_are_keys,
                                                                           qk_norm_names, chunk)
                rotations turn neighbouring pairs, with contexts stretched by wavelength (``rotary_pairs``)
  feed-forward  'dense': down(gelu_tanh(up h))                            (``dense``)
                'moe':   SiLU-gated experts, identity outputs among them, chosen by softmax score + correction inside the
                groups with the largest best choice, weighted by their renormalised scores (``routed_experts``)
  loop          the layers start..stop-1 run ``times`` times with the same weights, every pass with cache entries of
                its own; before every pass but the first x <- x + the embedding's rows   (block ``reentry_add``)
  output        N(x; final.norm), then the product with 'head'

Tensor names are those of the design's checkpoints.  The model has no position table and no context limit of its own.
"""
from __future__ import annotations

from ..config.dimalix import DimalixConfig
from ..parts.base import BLOCKS, FEED_FORWARDS, MIXERS, NORMS, POSITION_ENCODINGS
from ..parts.embedding import Embedding, OutputHead
from .base import LayerStep, ModelDef
from .registry import register_model


def _mixer(W, m, kind, mx, eps):
    rot, mask = mx.get("rot"), mx.get("mask")
    turn = None
    if rot and rot["dims"]:
        turn = POSITION_ENCODINGS.build("rotary_pairs", dims=rot["dims"], base=rot["base"], scaling=rot.get("scaling"))
    size = mask["size"] if mask else None
    if kind == "latent_attention":
        names = {k: m + k for k in ("q", "dkv", "uk", "uv", "o")}
        return MIXERS.build("latent_attention", hidden=W, num_heads=mx["heads"], dim=mx["dim"], rot=mx["rot_dim"],
                            vdim=mx["vdim"], kv_rank=mx["kv_rank"], q_rank=0, scale=mx["scale"], eps=eps,
                            names=dict(names, kv_norm=m + "dkv.norm"), qk_position=turn, window=size, float_out=True)
    return MIXERS.build("grouped_attention", hidden=W, num_heads=mx["heads"], num_kv_heads=mx["kv_heads"], dim=mx["dim"],
                        vdim=mx["dim"], scale=mx["scale"], names={k: m + k for k in ("q", "k", "o")}, qk_position=turn,
                        chunk=size, values_are_keys=True, qk_norm_names=(m + "q.norm", m + "k.norm"), qk_norm_eps=eps,
                        float_out=True)


def _feed_forward(W, p, mlp):
    if mlp is None:
        return None
    if mlp["kind"] == "dense":
        return FEED_FORWARDS.build("dense", hidden=W, inner=mlp["ff"], activation="gelu_tanh", fc1_name=p + "up",
                                   fc2_name=p + "down", bias=False, weight_suffix="", float_out=True)
    r = mlp["router"]
    groups = (r["groups"]["count"], r["groups"]["keep"]) if r.get("groups") else None
    return FEED_FORWARDS.build(
        "routed_experts", hidden=W, inner=mlp["expert"]["ff"], num_experts=r["experts"], top=r["top"], activation="silu",
        expert_names=[{k: f"{p}e{e}.{k}" for k in ("gate", "up", "down")} for e in range(r["experts"])],
        router_name=p + "router", correction_name=p + "correction", identity=r.get("identity") or 0, renormalise=True,
        groups=groups, group_score="max")


@register_model(DimalixConfig.ARCHITECTURE)
def build_dimalix(cfg: DimalixConfig) -> ModelDef:
    W, eps = cfg.width, cfg.norm_eps
    norm = lambda name: NORMS.build("rmsnorm", width=W, eps=eps, name=name)
    blocks, unused = [], set()
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        ffn = _feed_forward(W, p + "mlp.", layer.get("mlp"))
        if ffn is None:
            unused |= {p + "norm2", p + "ls2"}          # a checkpoint may hold them all the same
        blocks.append(BLOCKS.build(
            "parallel_scaled", mixer=_mixer(W, p + "mix.", layer["type"], layer["mixer"], eps), feed_forward=ffn,
            norm1=norm(p + "norm1"), norm2=norm(p + "norm2") if ffn is not None else None, width=W,
            scale_names=(p + "ls1", p + "ls2")))
    again = len(blocks)
    if cfg.loop and cfg.loop[2] > 1:
        blocks.append(BLOCKS.build("reentry_add"))
    order, entry = [], 0
    for i, opens in cfg.layer_runs():
        if opens:
            order.append(LayerStep(block=again, cache=-1))
        order.append(LayerStep(block=i, cache=entry))       # every run of a layer has a cache entry of its own
        entry += 1
    return ModelDef(cfg, Embedding(cfg.vocab, W, W, "embed", scale=cfg.embedding_scale), POSITION_ENCODINGS.build("none"),
                    blocks, order, norm("final.norm"), OutputHead(cfg.vocab, W, W, "head"),
                    canonical_name=lambda name: None if name in unused else name)
