"""Typed Zetenex configuration, read from the design's own config.json.

Keys: ``architecture`` ("Zetenex"), ``vocab``, ``width``, ``norm.eps``, ``canon.taps`` (the input convolutions),
``embedding.scale``, ``layers`` and optionally ``loop`` (``start``, ``stop``, ``times``: layers start .. stop - 1 run
``times`` times in a row; null or left out: every layer runs once).  A layer gives ``type``, the mixer's sizes ``mixer``
and the feed-forward ``mlp`` (null for none; else ``kind`` "dense" with ``ff``):

    mingru     width
    parallel   left_scale, right_scale,
               left: heads, kv_heads, dim, vdim, scale, and optionally q_temp (coef, every)
               right: inner, state, dt_rank, conv

No size has a default; a key this reader does not know is refused, so that a variant it cannot compute never runs as
something else.
"""
from __future__ import annotations

import json
from dataclasses import dataclass
from pathlib import Path
from typing import Any, Mapping

from .koronex import _need, _only
from .qwen2 import ConfigError


@dataclass(frozen=True)
class MinGRUMixer:
    width: int


@dataclass(frozen=True)
class LeftMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    q_temp: tuple[float, float] | None = None


@dataclass(frozen=True)
class RightMixer:
    inner: int
    state: int
    dt_rank: int
    conv: int


@dataclass(frozen=True)
class ParallelMixer:
    left: LeftMixer
    right: RightMixer
    left_scale: float
    right_scale: float


@dataclass(frozen=True)
class ZetenexLayer:
    type: str
    mixer: MinGRUMixer | ParallelMixer
    ff: int | None


@dataclass(frozen=True)
class Loop:
    start: int
    stop: int
    times: int


def _parallel(m, where: str) -> ParallelMixer:
    _only(m, ("left", "right", "left_scale", "right_scale"), where[:-1])
    a, b = _need(m, "left", where), _need(m, "right", where)
    la, lb = where + "left.", where + "right."
    _only(a, ("heads", "kv_heads", "dim", "vdim", "scale", "q_temp"), la[:-1])
    _only(b, ("inner", "state", "dt_rank", "conv"), lb[:-1])
    temp = a.get("q_temp")
    if temp is not None:
        _only(temp, ("coef", "every"), la + "q_temp")
        temp = (float(_need(temp, "coef", la + "q_temp.")), float(_need(temp, "every", la + "q_temp.")))
        if not temp[1] > 0:
            raise ConfigError(f"{la}q_temp.every must be positive")
    left = LeftMixer(*(int(_need(a, k, la)) for k in ("heads", "kv_heads", "dim", "vdim")), float(_need(a, "scale", la)), temp)
    right = RightMixer(*(int(_need(b, k, lb)) for k in ("inner", "state", "dt_rank", "conv")))
    if min(left.heads, left.kv_heads, left.dim, left.vdim) < 1 or left.heads % left.kv_heads:
        raise ConfigError(f"{la[:-1]}: heads, kv_heads (a divisor of heads), dim and vdim must be positive")
    if min(right.inner, right.state, right.dt_rank, right.conv) < 1:
        raise ConfigError(f"{lb[:-1]}: inner, state, dt_rank and conv must be positive")
    return ParallelMixer(left, right, float(_need(m, "left_scale", where)), float(_need(m, "right_scale", where)))


def _mlp(raw, where: str) -> int | None:
    if raw is None:
        return None
    kind = _need(raw, "kind", where)
    if kind != "dense":
        raise ConfigError(f"{where}kind {kind!r} is not a feed-forward of this design")
    _only(raw, ("kind", "ff"), where[:-1])
    ff = int(_need(raw, "ff", where))
    if ff < 1:
        raise ConfigError(f"{where}ff must be positive")
    return ff


def _loop(raw, layers: int) -> Loop | None:
    if raw is None:
        return None
    _only(raw, ("start", "stop", "times"), "loop")
    loop = Loop(*(int(_need(raw, k, "loop.")) for k in ("start", "stop", "times")))
    if not 0 <= loop.start < loop.stop <= layers or loop.times < 1:
        raise ConfigError(f"loop: layers {loop.start} to {loop.stop} of {layers}, {loop.times} times, make no sense")
    return loop


@dataclass(frozen=True)
class ZetenexConfig:
    vocab: int
    width: int
    eps: float
    taps: int
    embedding_scale: float
    layers: tuple[ZetenexLayer, ...]
    loop: Loop | None = None
    architecture: str = "Zetenex"

    @classmethod
    def from_dict(cls, d: Mapping[str, Any]) -> "ZetenexConfig":
        _only(d, ("architecture", "architectures", "vocab", "width", "norm", "canon", "embedding", "layers", "loop"),
              "the top level")
        norm, canon, emb = _need(d, "norm", ""), _need(d, "canon", ""), _need(d, "embedding", "")
        _only(norm, ("eps",), "norm")
        _only(canon, ("taps",), "canon")
        _only(emb, ("scale",), "embedding")
        layers = []
        for i, raw in enumerate(_need(d, "layers", "")):
            where = f"layers[{i}]."
            _only(raw, ("type", "mixer", "mlp"), where[:-1])
            kind, m = _need(raw, "type", where), _need(raw, "mixer", where)
            if kind == "mingru":
                _only(m, ("width",), where + "mixer")
                mixer = MinGRUMixer(int(_need(m, "width", where + "mixer.")))
                if mixer.width < 1:
                    raise ConfigError(f"{where}mixer.width must be positive")
            elif kind == "parallel":
                mixer = _parallel(m, where + "mixer.")
            else:
                raise ConfigError(f"{where}type {kind!r} is not a mixer of this design")
            layers.append(ZetenexLayer(kind, mixer, _mlp(raw.get("mlp"), where + "mlp.")))
        if not layers:
            raise ConfigError("config.json: no layers")
        cfg = cls(vocab=int(_need(d, "vocab", "")), width=int(_need(d, "width", "")), eps=float(_need(norm, "eps", "norm.")),
                  taps=int(_need(canon, "taps", "canon.")), embedding_scale=float(_need(emb, "scale", "embedding.")),
                  layers=tuple(layers), loop=_loop(d.get("loop"), len(layers)))
        if cfg.vocab < 1 or cfg.width < 1 or cfg.taps < 1 or not cfg.eps > 0:
            raise ConfigError("vocab, width and canon.taps must be positive and norm.eps above zero")
        return cfg

    @classmethod
    def from_json(cls, path) -> "ZetenexConfig":
        path = Path(path)
        if path.is_dir():
            path = path / "config.json"
        return cls.from_dict(json.loads(path.read_text()))
