"""Configuration of the Nigilorn design: layers of latent attention, gated grouped attention or selective scans inside
gated norm sandwiches, dense and group-routed feed-forwards, and a per-layer input looked up by token.

``config.json`` is nested: ``layers`` is a list of objects, each with ``type`` ("latent_attention", "attention" or
"mamba1"), ``mixer`` (its sizes and constants) and ``mlp`` (or null for none):

  latent_attention  ``heads``, ``dim``, ``rot_dim``, ``vdim``, ``kv_rank``, ``scale``, ``mask.size``, ``rot``
  attention         ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, ``mask.size``, ``rot``
  mamba1            ``inner``, ``state``, ``dt_rank``, ``conv``
  rot               ``dims``, ``base`` and optionally ``scaling`` (``factor``, ``original``, ``fast``, ``slow``)
  mlp               ``kind`` "dense" with ``ff``; or "moe" with ``expert.ff``, ``router.experts``, ``router.top``,
                    ``router.scale``, optionally ``router.groups`` (``count``, ``keep``) and ``shared.ff``

Model-wide keys: ``vocab``, ``width``, ``norm.eps`` and optionally ``token_side.dim``.  The file names the design with the
single string ``architecture``.  Every size and constant is read from the file; an optional group the file does not
mention switches its mechanism off (no ``mask``: every earlier key is seen; no ``rot``: nothing is rotated; no
``scaling``: plain frequencies; no ``groups``: all experts can be chosen; no ``scale`` of a router: 1; no ``shared``: no
shared expert; no ``token_side``: no input by token).
"""
from __future__ import annotations

import copy
import dataclasses
from typing import Any, ClassVar, Dict, Tuple

from .base import ConfigError, ModelConfig, register_config


def _need(obj: Any, key: str, where: str, kinds=(int, float)) -> Any:
    if not isinstance(obj, dict) or key not in obj:
        raise ConfigError(f"Nigilorn: config.json lacks '{where}{key}'")
    v = obj[key]
    if isinstance(v, bool) or not isinstance(v, kinds):
        raise ConfigError(f"Nigilorn: '{where}{key}' has the wrong type ({v!r})")
    return v


def _positive_int(obj: Any, key: str, where: str) -> int:
    v = _need(obj, key, where, int)
    if v <= 0:
        raise ConfigError(f"Nigilorn: '{where}{key}' must be a positive integer")
    return v


def _rot(rot: Any, limit: int, what: str, where: str) -> None:
    dims = _need(rot, "dims", where, int)
    base = _need(rot, "base", where)
    if dims < 0 or dims % 2 or dims > limit:
        raise ConfigError(f"Nigilorn: '{where}dims' must be even and at most '{what}'")
    if rot.get("scaling") is not None:
        for key in ("factor", "original", "fast", "slow"):
            if _need(rot["scaling"], key, where + "scaling.") <= 0:
                raise ConfigError(f"Nigilorn: '{where}scaling.{key}' must be positive")
    if base <= 0 or (rot.get("scaling") is not None and base <= 1):
        raise ConfigError(f"Nigilorn: '{where}base' must be positive (above 1 with scaling)")


def _attention(mx: Any, where: str) -> None:
    _need(mx, "scale", where)
    if mx.get("mask") is not None:
        _positive_int(mx["mask"], "size", where + "mask.")


@register_config
@dataclasses.dataclass(frozen=True)
class NigilornConfig(ModelConfig):
    ARCHITECTURE: ClassVar[str] = "Nigilorn"

    vocab: int
    width: int
    layers: Tuple[Dict[str, Any], ...]
    norm_eps: float
    side_dim: int = 0                                # 0: no input by token

    @classmethod
    def from_dict(cls, raw: Dict[str, Any]) -> "NigilornConfig":
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("Nigilorn: config.json lacks 'layers' (a list with one object per layer)")
        side = raw.get("token_side")
        cfg = cls(vocab=_need(raw, "vocab", "", int), width=_need(raw, "width", "", int),
                  layers=tuple(copy.deepcopy(layers)), norm_eps=float(_need(raw.get("norm"), "eps", "norm.")),
                  side_dim=_positive_int(side, "dim", "token_side.") if side is not None else 0)
        cfg.validate()
        return cfg

    def to_dict(self) -> Dict[str, Any]:
        out: Dict[str, Any] = {"architecture": self.ARCHITECTURE, "vocab": self.vocab, "width": self.width,
                               "layers": copy.deepcopy(list(self.layers)), "norm": {"eps": self.norm_eps}}
        if self.side_dim:
            out["token_side"] = {"dim": self.side_dim}
        return out

    def validate(self) -> None:
        if self.vocab <= 0 or self.width <= 0:
            raise ConfigError("Nigilorn: 'vocab' and 'width' must be positive")
        if self.norm_eps <= 0:
            raise ConfigError("Nigilorn: 'norm.eps' must be positive")
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]."
            kind = layer.get("type") if isinstance(layer, dict) else None
            mx = layer.get("mixer") if isinstance(layer, dict) else None
            w = where + "mixer."
            if kind == "latent_attention":
                for key in ("heads", "dim", "vdim", "kv_rank"):
                    _positive_int(mx, key, w)
                if _need(mx, "rot_dim", w, int) < 0:
                    raise ConfigError(f"Nigilorn: '{w}rot_dim' must not be negative")
                _attention(mx, w)
                if mx.get("rot") is not None:
                    _rot(mx["rot"], mx["rot_dim"], "rot_dim", w + "rot.")
            elif kind == "attention":
                for key in ("heads", "kv_heads", "dim", "vdim"):
                    _positive_int(mx, key, w)
                if mx["heads"] % mx["kv_heads"]:
                    raise ConfigError(f"Nigilorn: '{w}heads' must be a multiple of '{w}kv_heads'")
                _attention(mx, w)
                if mx.get("rot") is not None:
                    _rot(mx["rot"], mx["dim"], "dim", w + "rot.")
            elif kind == "mamba1":
                for key in ("inner", "state", "dt_rank", "conv"):
                    _positive_int(mx, key, w)
                if mx["conv"] > 8 or mx["state"] > 1024:
                    raise ConfigError(f"Nigilorn: '{w}conv' goes up to 8 taps and '{w}state' up to 1024")
            else:
                raise ConfigError(f"Nigilorn: '{where}type' = {kind!r} is not a known layer type (latent_attention, "
                                  f"attention, mamba1)")
            mlp = layer.get("mlp")
            if mlp is None:
                continue
            if mlp.get("kind") == "dense":
                _positive_int(mlp, "ff", where + "mlp.")
            elif mlp.get("kind") == "moe":
                _positive_int(mlp.get("expert"), "ff", where + "mlp.expert.")
                r, at = mlp.get("router"), where + "mlp.router."
                n, top = _positive_int(r, "experts", at), _positive_int(r, "top", at)
                if top > n:
                    raise ConfigError(f"Nigilorn: '{at}top' exceeds the number of experts")
                if r.get("scale") is not None:
                    _need(r, "scale", at)
                if r.get("groups") is not None:
                    count = _positive_int(r["groups"], "count", at + "groups.")
                    keep = _positive_int(r["groups"], "keep", at + "groups.")
                    if n % count or keep > count or keep * (n // count) < top:
                        raise ConfigError(f"Nigilorn: '{at}groups' must cut the experts into equal groups and keep enough "
                                          f"of them for 'top' experts")
                if mlp.get("shared") is not None:
                    _positive_int(mlp["shared"], "ff", where + "mlp.shared.")
            else:
                raise ConfigError(f"Nigilorn: '{where}mlp.kind' = {mlp.get('kind')!r} is not known (dense, moe)")
