"""Typed Rudutar configuration, read from the design's own config.json.

Keys: ``architecture`` ("Rudutar"), ``vocab``, ``width``, ``norm.eps`` and ``layers``, a list whose entries give ``type``
("attention" or "attention_2"), the mixer's sizes ``mixer`` and the feed-forward ``mlp``: null for none; ``kind`` "dense"
with ``ff``; or ``kind`` "moe" with ``expert.ff``, ``router`` (``experts``, ``top``, ``scale``, and ``groups.count`` and
``groups.keep``) and ``shared.ff`` (absent or null: no shared expert).

    attention     heads, kv_heads, dim, vdim, conv, scale, mask.size, q_temp.coef, q_temp.every, and optionally kv_from:
                  the index of an earlier such layer whose keys and values this one reads
    attention_2   heads, kv_heads, dim, vdim (equal to dim), scale, mask.size, rot.dims, rot.base

No size has a default (``q_temp`` may be left out for none, ``rot`` for a mixer that does not rotate, ``router.groups`` for
one group, ``router.scale`` for 1); a key this reader does not know is refused, so that a variant it cannot compute never
runs as something else.
"""
from __future__ import annotations

import json
from dataclasses import dataclass
from pathlib import Path
from typing import Any, Mapping

from .koronex import _need, _only
from .qwen2 import ConfigError


@dataclass(frozen=True)
class SlopedMixer:
    """"attention"."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int
    scale: float
    window: int
    q_temp: tuple[float, float] | None
    kv_from: int | None


@dataclass(frozen=True)
class KeyValueMixer:
    """"attention_2"."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int
    rot_dims: int
    rot_base: float


@dataclass(frozen=True)
class DenseFF:
    ff: int


@dataclass(frozen=True)
class RoutedFF:
    experts: int
    top: int
    scale: float
    group_count: int
    group_keep: int
    expert_ff: int
    shared_ff: int | None


@dataclass(frozen=True)
class RudutarLayer:
    type: str
    mixer: SlopedMixer | KeyValueMixer
    mlp: DenseFF | RoutedFF | None


def _mlp(raw, where: str):
    if raw is None:
        return None
    kind = _need(raw, "kind", where)
    if kind == "dense":
        _only(raw, ("kind", "ff"), where[:-1])
        ff = int(_need(raw, "ff", where))
        if ff < 1:
            raise ConfigError(f"{where}ff must be positive")
        return DenseFF(ff)
    if kind != "moe":
        raise ConfigError(f"{where}kind {kind!r} is not a feed-forward of this design")
    _only(raw, ("kind", "expert", "router", "shared"), where[:-1])
    expert, router = _need(raw, "expert", where), _need(raw, "router", where)
    _only(expert, ("ff",), where + "expert")
    _only(router, ("experts", "top", "groups", "scale"), where + "router")
    groups, shared, scale = router.get("groups"), raw.get("shared"), router.get("scale")
    count = keep = 1
    if groups is not None:
        _only(groups, ("count", "keep"), where + "router.groups")
        count, keep = int(_need(groups, "count", where + "router.groups.")), int(_need(groups, "keep", where + "router.groups."))
    if shared is not None:
        _only(shared, ("ff",), where + "shared")
    out = RoutedFF(int(_need(router, "experts", where + "router.")), int(_need(router, "top", where + "router.")),
                   1.0 if scale is None else float(scale), count, keep, int(_need(expert, "ff", where + "expert.")),
                   None if shared is None else int(_need(shared, "ff", where + "shared.")))
    if out.experts < 1 or out.expert_ff < 1 or (out.shared_ff is not None and out.shared_ff < 1):
        raise ConfigError(f"{where}: experts, expert.ff and shared.ff must be positive")
    if count < 1 or out.experts % count or not 1 <= keep <= count:
        raise ConfigError(f"{where}router.groups: {out.experts} experts do not form {count} equal groups of which {keep} are kept")
    if not 1 <= out.top <= out.experts // count * keep:
        raise ConfigError(f"{where}router.top {out.top} is more than the kept groups hold")
    return out


def _mixer(kind: str, m, where: str):
    common = ("heads", "kv_heads", "dim", "vdim", "scale", "mask")
    _only(m, common + (("conv", "q_temp", "kv_from") if kind == "attention" else ("rot",)), where + "mixer")
    at = where + "mixer."
    mask = _need(m, "mask", at)
    _only(mask, ("size",), at + "mask")
    sizes = {k: int(_need(m, k, at)) for k in ("heads", "kv_heads", "dim", "vdim")}
    sizes.update(scale=float(_need(m, "scale", at)), window=int(_need(mask, "size", at + "mask.")))
    if kind == "attention":
        temp = m.get("q_temp")
        if temp is not None:
            _only(temp, ("coef", "every"), at + "q_temp")
            temp = (float(_need(temp, "coef", at + "q_temp.")), float(_need(temp, "every", at + "q_temp.")))
            if not temp[1] > 0:
                raise ConfigError(f"{at}q_temp.every must be positive")
        out = SlopedMixer(**sizes, conv=int(_need(m, "conv", at)), q_temp=temp,
                          kv_from=None if m.get("kv_from") is None else int(m["kv_from"]))
        if not 1 <= out.conv <= 16:
            raise ConfigError(f"{at}conv: 1 to 16 taps")
    else:
        rot, dims, base = m.get("rot"), 0, 1.0
        if rot is not None:
            _only(rot, ("dims", "base"), at + "rot")
            dims = int(_need(rot, "dims", at + "rot."))
            base = float(_need(rot, "base", at + "rot.")) if dims else 1.0
        out = KeyValueMixer(**sizes, rot_dims=dims, rot_base=base)
        if out.vdim != out.dim:
            raise ConfigError(f"{at}vdim must equal dim: the values are the keys")
        if dims < 0 or dims % 2 or dims > out.dim or not base > 0:
            raise ConfigError(f"{at}rot: dims must be even and at most dim, base positive")
    if min(out.heads, out.kv_heads, out.dim, out.vdim, out.window) < 1 or out.heads % out.kv_heads:
        raise ConfigError(f"{where}mixer: heads, kv_heads (a divisor of heads), dim, vdim and mask.size must be positive")
    return out


@dataclass(frozen=True)
class RudutarConfig:
    vocab: int
    width: int
    eps: float
    layers: tuple[RudutarLayer, ...]
    architecture: str = "Rudutar"

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "RudutarConfig":
        _only(d, ("architecture", "architectures", "vocab", "width", "norm", "layers"), "the top level")
        norm = _need(d, "norm", "")
        _only(norm, ("eps",), "norm")
        layers = []
        for i, raw in enumerate(_need(d, "layers", "")):
            where = f"layers[{i}]."
            _only(raw, ("type", "mixer", "mlp"), where[:-1])
            kind = _need(raw, "type", where)
            if kind not in ("attention", "attention_2"):
                raise ConfigError(f"{where}type {kind!r} is not a mixer of this design")
            layers.append(RudutarLayer(kind, _mixer(kind, _need(raw, "mixer", where), where), _mlp(raw.get("mlp"), where + "mlp.")))
        if not layers:
            raise ConfigError("config.json: no layers")
        for i, layer in enumerate(layers):
            j = getattr(layer.mixer, "kv_from", None)
            if j is None:
                continue
            if not 0 <= j < i or layers[j].type != "attention" or layers[j].mixer.kv_from is not None:
                raise ConfigError(f"layers[{i}].mixer.kv_from {j} must name an earlier attention layer with keys of its own")
            a, b = layer.mixer, layers[j].mixer
            if (a.kv_heads, a.dim, a.vdim) != (b.kv_heads, b.dim, b.vdim):
                raise ConfigError(f"layers[{i}] reads the keys of layer {j}, whose kv_heads, dim or vdim differ")
        cfg = cls(vocab=int(_need(d, "vocab", "")), width=int(_need(d, "width", "")),
                  eps=float(_need(norm, "eps", "norm.")), layers=tuple(layers))
        if cfg.vocab < 1 or cfg.width < 1 or not cfg.eps > 0:
            raise ConfigError("vocab and width must be positive and norm.eps above zero")
        return cfg

    @classmethod
    def from_json(cls, path) -> "RudutarConfig":
        path = Path(path)
        if path.is_dir():
            path = path / "config.json"
        return cls.from_dict(json.loads(path.read_text()))
