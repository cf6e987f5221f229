"""Nigilorn put together from the parts.

A decoder-only model whose layers are listed in the configuration:

  embedding     x = embed[token]
  layer i       for the mixer and then the feed-forward (which may be absent):
                h = N(x; norm1);  x <- x + N(sigmoid(rg1 h + rg1.b) * mixer(h); norm1b)      (block ``gated_sandwich``)
                and an input of the layer's own by token:
                x <- x + N(side.proj (gelu_tanh(side.gate x) * e); side.norm)                (``TokenSide``)
  mixers        'latent_attention': queries straight from the input, keys and values from one normed latent per token,
                a rotated key part shared by the heads, a window         (``latent_attention`` with q_rank 0, window)
                'attention': grouped attention without biases, rotation on part of each head, q and k divided by their
                root mean square, a window, one sigmoid gate per head    (``grouped_attention`` with gate="head")
                'mamba1': the selective scan                             (``mamba``)
                rotations turn neighbouring pairs, with stretched contexts (``rotary_pairs`` with scaling)
  feed-forward  'dense': down(silu(gate h) * (up h))                     (``gated``)
                'moe':   experts down(relu(up h)^2) chosen by sigmoid scores inside the best groups, renormalised and
                scaled, plus a shared expert of that form                (``routed_experts`` with gated=False)
  output        N(x; final.norm), then the product with 'head'

Tensor names are those of the design's checkpoints.  The model has no position table and no context limit of its own.
"""
from __future__ import annotations

from ..config.nigilorn import NigilornConfig
from ..parts.base import BLOCKS, FEED_FORWARDS, MIXERS, NORMS, POSITION_ENCODINGS
from ..parts.embedding import Embedding, OutputHead, TokenSide
from .base import LayerStep, ModelDef
from .registry import register_model


def _rotation(mx):
    rot = mx.get("rot")
    if not rot or not rot["dims"]:
        return None
    return POSITION_ENCODINGS.build("rotary_pairs", dims=rot["dims"], base=rot["base"], scaling=rot.get("scaling"))


def _window(mx):
    return mx["mask"]["size"] if mx.get("mask") else None


def _mixer(W, m, kind, mx, eps):
    if kind == "latent_attention":
        names = {k: m + k for k in ("q", "dkv", "uk", "uv", "o")}
        return MIXERS.build("latent_attention", hidden=W, num_heads=mx["heads"], dim=mx["dim"], rot=mx["rot_dim"],
                            vdim=mx["vdim"], kv_rank=mx["kv_rank"], q_rank=0, scale=mx["scale"], eps=eps,
                            names=dict(names, kv_norm=m + "dkv.norm"), qk_position=_rotation(mx), window=_window(mx),
                            float_out=True)
    if kind == "attention":
        return MIXERS.build("grouped_attention", hidden=W, num_heads=mx["heads"], num_kv_heads=mx["kv_heads"],
                            dim=mx["dim"], vdim=mx["vdim"], scale=mx["scale"],
                            names={k: m + k for k in ("q", "k", "v", "o", "g")}, qkv_bias=False, o_bias=False,
                            window=_window(mx), qk_position=_rotation(mx), gate="head", qk_norm_eps=eps, float_out=True)
    names = {"in": "in", "x": "x", "dt": "dt", "o": "o", "conv": "conv", "conv_bias": "conv.b", "dt_bias": "dt.b",
             "A_log": "A_log", "D": "D"}
    return MIXERS.build("mamba", hidden=W, inner=mx["inner"], state=mx["state"], dt_rank=mx["dt_rank"],
                        conv_taps=mx["conv"], names={k: m + v for k, v in names.items()}, float_out=True)


def _feed_forward(W, p, mlp):
    if mlp is None:
        return None
    if mlp["kind"] == "dense":
        return FEED_FORWARDS.build("gated", hidden=W, inner=mlp["ff"], activation="silu", gate_name=p + "gate",
                                   up_name=p + "up", down_name=p + "down", float_out=True)
    r, shared = mlp["router"], None
    if mlp.get("shared") is not None:
        shared = FEED_FORWARDS.build("dense", hidden=W, inner=mlp["shared"]["ff"], activation="relu2", bias=False,
                                     fc1_name=p + "shared.up", fc2_name=p + "shared.down", weight_suffix="")
    groups = (r["groups"]["count"], r["groups"]["keep"]) if r.get("groups") else None
    return FEED_FORWARDS.build(
        "routed_experts", hidden=W, inner=mlp["expert"]["ff"], num_experts=r["experts"], top=r["top"], activation="relu2",
        expert_names=[{k: f"{p}e{e}.{k}" for k in ("up", "down")} for e in range(r["experts"])],
        router_name=p + "router", shared=shared, renormalise=True, scores="sigmoid", groups=groups,
        scale=1.0 if r.get("scale") is None else r["scale"], gated=False)


@register_model(NigilornConfig.ARCHITECTURE)
def build_nigilorn(cfg: NigilornConfig) -> ModelDef:
    W, eps = cfg.width, cfg.norm_eps
    norm = lambda name: NORMS.build("rmsnorm", width=W, eps=eps, name=name)
    side = TokenSide(cfg.vocab, len(cfg.layers), cfg.side_dim, "side.embed") if cfg.side_dim else None
    blocks = []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        ffn = _feed_forward(W, p + "mlp.", layer.get("mlp"))
        blocks.append(BLOCKS.build(
            "gated_sandwich", mixer=_mixer(W, p + "mix.", layer["type"], layer["mixer"], eps), feed_forward=ffn,
            norm1=norm(p + "norm1"), norm1b=norm(p + "norm1b"), norm2=norm(p + "norm2") if ffn is not None else None,
            norm2b=norm(p + "norm2b") if ffn is not None else None, width=W, gate_names=(p + "rg1", p + "rg2"), side=side,
            side_names={k: f"{p}side.{k}" for k in ("gate", "proj", "norm")} if side is not None else None, layer=i, eps=eps))
    order = [LayerStep(block=i, cache=i) for i in range(len(blocks))]
    return ModelDef(cfg, Embedding(cfg.vocab, W, W, "embed"), POSITION_ENCODINGS.build("none"), blocks, order,
                    NORMS.build("rmsnorm", width=W, eps=eps, name="final.norm"), OutputHead(cfg.vocab, W, W, "head"),
                    shared_parts=[side] if side is not None else [])
