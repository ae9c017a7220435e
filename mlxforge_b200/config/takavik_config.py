"""Typed configuration of the Takavik decoder, read from its own ``config.json`` keys.

    {"architecture": "Takavik", "vocab": V, "width": H, "streams": S, "norm": {"eps": e},
     "layers": [{"type": "parallel" | "mamba2" | "gla", "mixer": {...},
                 "mlp": {"kind": "dense", "ff": F} | null}, ...]}

Mixer keys.  ``parallel``: ``left`` (attention: ``heads, kv_heads, dim, vdim, scale``, ``q_temp.{coef, every}``) and
``right`` (selective scan: ``inner, state, dt_rank, conv``).  ``mamba2``: ``heads, vdim, state, groups, norm_groups,
conv``.  ``gla``: ``heads, dim, vdim, tau``.  What a file may leave out: ``streams`` (one ordinary residual stream
without connections), ``kv_heads`` (``heads``), ``vdim`` of an attention or gla mixer (``dim``), ``scale`` (``dim^-1/2``),
``q_temp`` (none), ``groups`` and ``norm_groups`` (1).  The low rank of a ``gla`` layer's decay is not in config.json: it
is the first extent of the tensor ``l<i>.mix.a1`` (``with_tensor_shapes``); a configuration that is to be written with
random weights names it as ``mixer.decay_rank``.
"""
from __future__ import annotations

import copy
import math
from dataclasses import dataclass, field, replace
from typing import Any, Dict, Tuple

from .ledinex_config import _finite
from .model_config import ConfigError, ModelConfig, _optional, _require, architecture_name
from .notirax_config import _obj, _opt, _positive, _req

LAYER_TYPES = ("parallel", "mamba2", "gla")


def _multiple(a: int, b: int, where: str, what: str, of: str) -> None:
    if a % b:
        raise ConfigError(f"config.json: {where}{what} ({a}) must be a multiple of {where}{of} ({b})")


def _parse_attention(m: Dict[str, Any], where: str) -> Dict[str, Any]:
    out = {"heads": _positive(_req(m, "heads", int, where), where + "heads"),
           "dim": _positive(_req(m, "dim", int, where), where + "dim")}
    out["kv_heads"] = _positive(_opt(m, "kv_heads", int, out["heads"], where), where + "kv_heads")
    out["vdim"] = _positive(_opt(m, "vdim", int, out["dim"], where), where + "vdim")
    _multiple(out["heads"], out["kv_heads"], where, "heads", "kv_heads")
    out["scale"] = _finite(_opt(m, "scale", float, float(out["dim"]) ** -0.5, where), where + "scale")
    out["q_temp"] = None
    t, w = _obj(m, "q_temp", where, required=False), where + "q_temp."
    if t:
        out["q_temp"] = {"coef": _finite(_req(t, "coef", float, w), w + "coef"),
                         "every": _positive(_finite(_req(t, "every", float, w), w + "every"), w + "every")}
    return out


def _parse_scan(m: Dict[str, Any], where: str) -> Dict[str, Any]:
    return {k: _positive(_req(m, k, int, where), where + k) for k in ("inner", "state", "dt_rank", "conv")}


def _parse_mamba2(m: Dict[str, Any], where: str) -> Dict[str, Any]:
    out = {k: _positive(_req(m, k, int, where), where + k) for k in ("heads", "vdim", "state", "conv")}
    for k in ("groups", "norm_groups"):
        out[k] = _positive(_opt(m, k, int, 1, where), where + k)
    _multiple(out["heads"], out["groups"], where, "heads", "groups")
    _multiple(out["heads"] * out["vdim"], out["norm_groups"], where, "heads * vdim", "norm_groups")
    return out


def _parse_gla(m: Dict[str, Any], where: str) -> Dict[str, Any]:
    out = {k: _positive(_req(m, k, int, where), where + k) for k in ("heads", "dim")}
    out["vdim"] = _positive(_opt(m, "vdim", int, out["dim"], where), where + "vdim")
    out["tau"] = _positive(_finite(_req(m, "tau", float, where), where + "tau"), where + "tau")
    out["decay_rank"] = _opt(m, "decay_rank", int, 0, where)
    return out


def _parse_mixer(kind: str, m: Dict[str, Any], where: str) -> Dict[str, Any]:
    if kind == "mamba2":
        return _parse_mamba2(m, where)
    if kind == "gla":
        return _parse_gla(m, where)
    return {"left": _parse_attention(_obj(m, "left", where), where + "left."),
            "right": _parse_scan(_obj(m, "right", where), where + "right.")}


def _parse_mlp(m: Dict[str, Any], where: str) -> Dict[str, Any]:
    kind = _req(m, "kind", str, where)
    if kind != "dense":
        raise ConfigError(f"config.json: {where}kind '{kind}' is not supported (supported: dense)")
    return {"kind": kind, "ff": _positive(_req(m, "ff", int, where), where + "ff")}


@dataclass(frozen=True)
class TakavikConfig(ModelConfig):
    vocab: int = 0
    width: int = 0
    streams: int = 0                 # 0: config.json names none (one ordinary residual stream)
    norm_eps: float = 0.0
    # per layer: {"type", "mixer": {...}, "mlp": {...} | None}, parsed and checked
    layers: Tuple[Dict[str, Any], ...] = field(default=(), compare=False)

    @classmethod
    def from_json(cls, j: Dict[str, Any]) -> "TakavikConfig":
        if not isinstance(j, dict):
            raise ConfigError("config.json: top level must be an object")
        arch = architecture_name(j)
        vocab = _positive(_require(j, "vocab", int), "vocab")
        width = _positive(_require(j, "width", int), "width")
        streams = _optional(j, "streams", int, 0)
        if streams < 0 or streams > 8:
            raise ConfigError(f"config.json: field 'streams' must be between 1 and 8, got {streams}")
        eps = _req(_obj(j, "norm", ""), "eps", float, "norm.")
        if not (eps >= 0.0 and math.isfinite(eps)):
            raise ConfigError(f"config.json: field 'norm.eps' must be non-negative, got {eps}")
        raw_layers = j.get("layers")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError("config.json: missing required field 'layers' (a list of layers)")
        layers = []
        for i, layer in enumerate(raw_layers):
            where = f"layers[{i}]."
            if not isinstance(layer, dict):
                raise ConfigError(f"config.json: field 'layers[{i}]' has wrong type: expected object")
            kind = _req(layer, "type", str, where)
            if kind not in LAYER_TYPES:
                raise ConfigError(f"config.json: {where}type '{kind}' is not supported (supported: "
                                  f"{', '.join(LAYER_TYPES)})")
            mixer = _parse_mixer(kind, _obj(layer, "mixer", where), where + "mixer.")
            mlp = layer.get("mlp")
            if mlp is not None and not isinstance(mlp, dict):
                raise ConfigError(f"config.json: field '{where}mlp' has wrong type: expected object or null")
            layers.append({"type": kind, "mixer": mixer,
                           "mlp": None if mlp is None else _parse_mlp(mlp, where + "mlp.")})
        return cls(architecture=arch, raw=dict(j), vocab=vocab, width=width, streams=streams, norm_eps=eps,
                   layers=tuple(layers))

    def with_tensor_shapes(self, shapes: Dict[str, tuple]) -> "TakavikConfig":
        layers = copy.deepcopy(list(self.layers))
        for i, layer in enumerate(layers):
            name = f"l{i}.mix.a1"
            if layer["type"] == "gla" and name in shapes and len(shapes[name]) == 2:
                layer["mixer"]["decay_rank"] = int(shapes[name][0])
        return replace(self, layers=tuple(layers))

    def to_json(self) -> Dict[str, Any]:
        """The config.json this configuration would be read back from."""
        out: Dict[str, Any] = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
                               "norm": {"eps": self.norm_eps}, "layers": []}
        if self.streams:
            out["streams"] = self.streams
        for layer in self.layers:
            m = copy.deepcopy(layer["mixer"])
            if layer["type"] == "parallel" and m["left"]["q_temp"] is None:
                del m["left"]["q_temp"]
            out["layers"].append({"type": layer["type"], "mixer": m, "mlp": copy.deepcopy(layer["mlp"])})
        return out
