"""Configuration of the Dimalix design: parallel sub-layers with a norm and a scale each, latent attention in a window and
grouped attention in chunks, mixtures with identity experts, a looped stretch of layers.

``config.json`` is nested: ``layers`` is a list of objects, each with ``type`` ("latent_attention" or "attention"),
``mixer`` (its sizes and constants) and ``mlp`` (or null for none):

  latent_attention  ``heads``, ``dim``, ``rot_dim``, ``vdim``, ``kv_rank``, ``scale``, ``mask.size`` (a window), ``rot``
  attention         ``heads``, ``kv_heads``, ``dim``, ``vdim`` (= ``dim``: the values are the keys), ``scale``,
                    ``mask.size`` (chunks), ``rot``
  rot               ``dims``, ``base`` and optionally ``scaling`` (``factor``, ``original``, ``low``, ``high``)
  mlp               ``kind`` "dense" with ``ff``; or "moe" with ``expert.ff``, ``router.experts``, ``router.top`` and
                    optionally ``router.identity`` (outputs that stand for the identity) and ``router.groups``
                    (``count``, ``keep``; over experts and identity outputs together)

Model-wide keys: ``vocab``, ``width``, ``norm.eps`` and optionally ``embedding.scale`` and ``loop`` (``start``, ``stop``,
``times``: the layers start..stop-1 run ``times`` times in a row with the same weights).  The file names the design with
the single string ``architecture``.  Every size and constant is read from the file; an optional group the file does not
mention switches its mechanism off (no ``mask``: every earlier key is seen; no ``rot``: nothing is rotated; no
``scaling``: plain frequencies; no ``groups``: all outputs can be chosen; no ``loop``: every layer runs once).
"""
from __future__ import annotations

import copy
import dataclasses
from typing import Any, ClassVar, Dict, Optional, Tuple

from .base import ConfigError, ModelConfig, register_config


def _need(obj: Any, key: str, where: str, kinds=(int, float)) -> Any:
    if not isinstance(obj, dict) or key not in obj:
        raise ConfigError(f"Dimalix: config.json lacks '{where}{key}'")
    v = obj[key]
    if isinstance(v, bool) or not isinstance(v, kinds):
        raise ConfigError(f"Dimalix: '{where}{key}' has the wrong type ({v!r})")
    return v


def _positive_int(obj: Any, key: str, where: str) -> int:
    v = _need(obj, key, where, int)
    if v <= 0:
        raise ConfigError(f"Dimalix: '{where}{key}' must be a positive integer")
    return v


def _rot(rot: Any, limit: int, what: str, where: str) -> None:
    dims = _need(rot, "dims", where, int)
    if dims < 0 or dims % 2 or dims > limit:
        raise ConfigError(f"Dimalix: '{where}dims' must be even and at most '{what}'")
    if _need(rot, "base", where) <= 0:
        raise ConfigError(f"Dimalix: '{where}base' must be positive")
    sc = rot.get("scaling")
    if sc is not None:
        for key in ("factor", "original", "low", "high"):
            if _need(sc, key, where + "scaling.") <= 0:
                raise ConfigError(f"Dimalix: '{where}scaling.{key}' must be positive")
        if sc["high"] < sc["low"]:
            raise ConfigError(f"Dimalix: '{where}scaling.high' must not be below 'low'")


def _mlp(mlp: Any, where: str) -> None:
    if mlp is None:
        return
    if mlp.get("kind") == "dense":
        _positive_int(mlp, "ff", where)
        return
    if mlp.get("kind") != "moe":
        raise ConfigError(f"Dimalix: '{where}kind' = {mlp.get('kind')!r} is not known (dense, moe)")
    _positive_int(mlp.get("expert"), "ff", where + "expert.")
    r, at = mlp.get("router"), where + "router."
    outputs, top = _positive_int(r, "experts", at), _positive_int(r, "top", at)
    if r.get("identity") is not None:
        if _need(r, "identity", at, int) < 0:
            raise ConfigError(f"Dimalix: '{at}identity' must not be negative")
        outputs += r["identity"]
    if top > outputs:
        raise ConfigError(f"Dimalix: '{at}top' exceeds the number of router outputs")
    if r.get("groups") is not None:
        count = _positive_int(r["groups"], "count", at + "groups.")
        keep = _positive_int(r["groups"], "keep", at + "groups.")
        if outputs % count or keep > count or keep * (outputs // count) < top:
            raise ConfigError(f"Dimalix: '{at}groups' must cut the router outputs into equal groups and keep enough of them "
                              f"for 'top' choices")


@register_config
@dataclasses.dataclass(frozen=True)
class DimalixConfig(ModelConfig):
    ARCHITECTURE: ClassVar[str] = "Dimalix"

    vocab: int
    width: int
    layers: Tuple[Dict[str, Any], ...]
    norm_eps: float
    embedding_scale: float = 1.0
    loop: Optional[Tuple[int, int, int]] = None     # (start, stop, times)

    @classmethod
    def from_dict(cls, raw: Dict[str, Any]) -> "DimalixConfig":
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("Dimalix: config.json lacks 'layers' (a list with one object per layer)")
        loop = None
        if raw.get("loop") is not None:
            loop = tuple(_need(raw["loop"], key, "loop.", int) for key in ("start", "stop", "times"))
        cfg = cls(vocab=_need(raw, "vocab", "", int), width=_need(raw, "width", "", int),
                  layers=tuple(copy.deepcopy(layers)), norm_eps=float(_need(raw.get("norm"), "eps", "norm.")),
                  embedding_scale=float(_need(raw["embedding"], "scale", "embedding.")) if raw.get("embedding") is not None else 1.0,
                  loop=loop)
        cfg.validate()
        return cfg

    def to_dict(self) -> Dict[str, Any]:
        out: Dict[str, Any] = {"architecture": self.ARCHITECTURE, "vocab": self.vocab, "width": self.width,
                               "layers": copy.deepcopy(list(self.layers)), "norm": {"eps": self.norm_eps},
                               "embedding": {"scale": self.embedding_scale}}
        if self.loop:
            out["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        return out

    def layer_runs(self):
        """The order in which layers run: [(layer index, whether a later pass over the stretch opens here)]."""
        n = len(self.layers)
        start, stop, times = self.loop or (0, n, 1)
        runs = [(i, False) for i in range(start)]
        for t in range(times):
            runs += [(i, t > 0 and i == start) for i in range(start, stop)]
        return runs + [(i, False) for i in range(stop, n)]

    def validate(self) -> None:
        if self.vocab <= 0 or self.width <= 0:
            raise ConfigError("Dimalix: 'vocab' and 'width' must be positive")
        if self.norm_eps <= 0:
            raise ConfigError("Dimalix: 'norm.eps' must be positive")
        if self.loop is not None:
            start, stop, times = self.loop
            if not (0 <= start < stop <= len(self.layers)) or times < 1:
                raise ConfigError("Dimalix: 'loop' needs 0 <= start < stop <= number of layers and times >= 1")
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]."
            kind = layer.get("type") if isinstance(layer, dict) else None
            mx = layer.get("mixer") if isinstance(layer, dict) else None
            w = where + "mixer."
            if kind == "latent_attention":
                for key in ("heads", "dim", "vdim", "kv_rank"):
                    _positive_int(mx, key, w)
                if _need(mx, "rot_dim", w, int) < 0:
                    raise ConfigError(f"Dimalix: '{w}rot_dim' must not be negative")
                limit, what = mx["rot_dim"], "rot_dim"
            elif kind == "attention":
                for key in ("heads", "kv_heads", "dim"):
                    _positive_int(mx, key, w)
                if mx["heads"] % mx["kv_heads"]:
                    raise ConfigError(f"Dimalix: '{w}heads' must be a multiple of '{w}kv_heads'")
                if mx.get("vdim", mx["dim"]) != mx["dim"]:
                    raise ConfigError(f"Dimalix: '{w}vdim' must be '{w}dim' (the values are the keys)")
                limit, what = mx["dim"], "dim"
            else:
                raise ConfigError(f"Dimalix: '{where}type' = {kind!r} is not a known layer type (latent_attention, attention)")
            _need(mx, "scale", w)
            if mx.get("mask") is not None:
                _positive_int(mx["mask"], "size", w + "mask.")
            if mx.get("rot") is not None:
                _rot(mx["rot"], limit, what, w + "rot.")
            _mlp(layer.get("mlp"), where + "mlp.")
