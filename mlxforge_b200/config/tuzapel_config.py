"""Typed configuration of the Tuzapel decoder, read from its own ``config.json`` keys.

    {"architecture": "Tuzapel", "vocab": V, "width": H, "norm": {"eps": e}, "logit_softcap": c,
     "layers": [{"type": "latent_attention" | "attention", "mixer": {...},
                 "mlp": {"kind": "dense", "ff": F, "limit": l}
                      | {"kind": "moe", "expert": {"ff": F, "limit": l}, "router": {"experts": E, "top": k}}
                      | null}, ...]}

Mixer keys.  ``attention``: ``heads, kv_heads, dim, vdim, scale, conv`` (taps), ``mask.size``, ``rot.{base, dims,
scaling}`` with ``scaling.{factor, low, high, original}``, and ``kv_from`` (the layer whose keys and values this
one reads; it has none of its own).  ``latent_attention``: ``heads, dim, rot_dim, vdim, q_rank, kv_rank, scale,
rot.{base, dims}``.  What a file may leave out: ``logit_softcap`` (none), ``kv_heads`` (``heads``), ``vdim``
(``dim``), ``scale`` (the inverse root of the query size), ``conv`` (no convolution and no ``*.conv`` tensors),
``mask`` (causal), ``rot`` of an attention (no rotation), ``rot.dims`` (all of ``dim`` or ``rot_dim``),
``rot.scaling`` (plain frequencies), ``limit`` (no clamp).
"""
from __future__ import annotations

import math
from dataclasses import dataclass, field
from typing import Any, Dict, Optional, Tuple

from .model_config import ConfigError, ModelConfig, _require, architecture_name
from .notirax_config import _obj, _opt, _positive, _req

LAYER_TYPES = ("latent_attention", "attention")
MLP_KINDS = ("dense", "moe")


def _finite(v: float, name: str) -> float:
    if not math.isfinite(v):
        raise ConfigError(f"config.json: field '{name}' must be finite")
    return v


def _parse_rot(m: Dict[str, Any], dim: int, where: str, required: bool, scaled: bool) -> Optional[Dict[str, Any]]:
    rot = _obj(m, "rot", where, required=required)
    if not rot:
        return None
    w = where + "rot."
    out: Dict[str, Any] = {"base": _req(rot, "base", float, w), "dims": _opt(rot, "dims", int, dim, w), "scaling": None}
    if not (out["base"] > 0 and math.isfinite(out["base"])):
        raise ConfigError(f"config.json: field '{w}base' must be positive, got {out['base']}")
    if out["dims"] < 0 or out["dims"] % 2 or out["dims"] > dim:
        raise ConfigError(f"config.json: field '{w}dims' must be even and between 0 and {dim}, got {out['dims']}")
    sc = _obj(rot, "scaling", w, required=False)
    if sc:
        if not scaled:
            raise ConfigError(f"config.json: field '{w}scaling' is not supported in this mixer")
        out["scaling"] = {k: _positive(_req(sc, k, float, w + "scaling."), w + "scaling." + k)
                          for k in ("factor", "low", "high", "original")}
        if out["scaling"]["high"] < out["scaling"]["low"]:
            raise ConfigError(f"config.json: field '{w}scaling.high' must not be below '{w}scaling.low'")
    return out


def _parse_attention(m: Dict[str, Any], where: str) -> Dict[str, Any]:
    out = {"heads": _positive(_req(m, "heads", int, where), where + "heads"),
           "dim": _positive(_req(m, "dim", int, where), where + "dim")}
    out["kv_heads"] = _positive(_opt(m, "kv_heads", int, out["heads"], where), where + "kv_heads")
    out["vdim"] = _positive(_opt(m, "vdim", int, out["dim"], where), where + "vdim")
    if out["heads"] % out["kv_heads"]:
        raise ConfigError(f"config.json: {where}heads ({out['heads']}) must be a multiple of {where}kv_heads "
                          f"({out['kv_heads']})")
    out["scale"] = _finite(_opt(m, "scale", float, float(out["dim"]) ** -0.5, where), where + "scale")
    out["conv"] = _opt(m, "conv", int, 0, where)
    out["window"] = _opt(_obj(m, "mask", where, required=False), "size", int, 0, where + "mask.")
    for key, v in (("conv", out["conv"]), ("mask.size", out["window"])):
        if v < 0:
            raise ConfigError(f"config.json: field '{where}{key}' must not be negative, got {v}")
    out["rot"] = _parse_rot(m, out["dim"], where, False, True)
    out["kv_from"] = None if m.get("kv_from") is None else _req(m, "kv_from", int, where)
    return out


def _parse_latent(m: Dict[str, Any], where: str) -> Dict[str, Any]:
    out = {k: _positive(_req(m, k, int, where), where + k) for k in ("heads", "dim", "q_rank", "kv_rank")}
    out["rot_dim"] = _req(m, "rot_dim", int, where)
    if out["rot_dim"] < 0 or out["rot_dim"] % 2:
        raise ConfigError(f"config.json: field '{where}rot_dim' must be even and not negative, got {out['rot_dim']}")
    out["vdim"] = _positive(_opt(m, "vdim", int, out["dim"], where), where + "vdim")
    out["scale"] = _finite(_opt(m, "scale", float, float(out["dim"] + out["rot_dim"]) ** -0.5, where), where + "scale")
    out["rot"] = _parse_rot(m, out["rot_dim"], where, out["rot_dim"] > 0, False)
    return out


def _limit(m: Dict[str, Any], where: str) -> Optional[float]:
    v = m.get("limit")
    return None if v is None else _positive(_req(m, "limit", float, where), where + "limit")


def _parse_mlp(m: Dict[str, Any], where: str) -> Dict[str, Any]:
    kind = _req(m, "kind", str, where)
    if kind not in MLP_KINDS:
        raise ConfigError(f"config.json: {where}kind '{kind}' is not supported (supported: {', '.join(MLP_KINDS)})")
    if kind == "dense":
        return {"kind": kind, "ff": _positive(_req(m, "ff", int, where), where + "ff"), "limit": _limit(m, where)}
    expert, router = _obj(m, "expert", where), _obj(m, "router", where)
    out = {"kind": kind, "ff": _positive(_req(expert, "ff", int, where + "expert."), where + "expert.ff"),
           "limit": _limit(expert, where + "expert."),
           "experts": _positive(_req(router, "experts", int, where + "router."), where + "router.experts"),
           "top": _positive(_req(router, "top", int, where + "router."), where + "router.top")}
    if out["top"] > out["experts"]:
        raise ConfigError(f"config.json: {where}router: {out['experts']} experts cannot give a token {out['top']}")
    return out


def _check_sources(layers) -> None:
    """A layer may read the keys and values of an earlier attention layer of its own geometry that has some."""
    for i, layer in enumerate(layers):
        m = layer["mixer"]
        j = m.get("kv_from")
        if j is None:
            continue
        where = f"layers[{i}].mixer."
        if not (0 <= j < i) or layers[j]["type"] != "attention" or layers[j]["mixer"]["kv_from"] is not None:
            raise ConfigError(f"config.json: field '{where}kv_from' must name an earlier attention layer with keys and "
                              f"values of its own, got {j}")
        src = layers[j]["mixer"]
        for k in ("kv_heads", "dim", "vdim"):
            if m[k] != src[k]:
                raise ConfigError(f"config.json: {where}{k} ({m[k]}) differs from layer {j}'s ({src[k]}), whose keys and "
                                  f"values it reads")


@dataclass(frozen=True)
class TuzapelConfig(ModelConfig):
    vocab: int = 0
    width: int = 0
    norm_eps: float = 0.0
    logit_softcap: float = 0.0      # 0: logits as they are
    # per layer: {"type", "mixer": {...}, "mlp": {...} | None}, parsed and checked
    layers: Tuple[Dict[str, Any], ...] = field(default=(), compare=False)

    @classmethod
    def from_json(cls, j: Dict[str, Any]) -> "TuzapelConfig":
        if not isinstance(j, dict):
            raise ConfigError("config.json: top level must be an object")
        arch = architecture_name(j)
        vocab = _positive(_require(j, "vocab", int), "vocab")
        width = _positive(_require(j, "width", int), "width")
        eps = _req(_obj(j, "norm", ""), "eps", float, "norm.")
        if not (eps >= 0.0 and math.isfinite(eps)):
            raise ConfigError(f"config.json: field 'norm.eps' must be non-negative, got {eps}")
        cap = _opt(j, "logit_softcap", float, 0.0, "")
        if not (cap >= 0.0 and math.isfinite(cap)):
            raise ConfigError(f"config.json: field 'logit_softcap' must not be negative, got {cap}")
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
            m = _obj(layer, "mixer", where)
            mixer = _parse_attention(m, where + "mixer.") if kind == "attention" else _parse_latent(m, where + "mixer.")
            mlp = layer.get("mlp")
            if mlp is not None and not isinstance(mlp, dict):
                raise ConfigError(f"config.json: field '{where}mlp' has wrong type: expected object or null")
            layers.append({"type": kind, "mixer": mixer,
                           "mlp": None if mlp is None else _parse_mlp(mlp, where + "mlp.")})
        _check_sources(layers)
        return cls(architecture=arch, raw=dict(j), vocab=vocab, width=width, norm_eps=eps, logit_softcap=cap,
                   layers=tuple(layers))

    def to_json(self) -> Dict[str, Any]:
        """The config.json this configuration would be read back from."""
        out: Dict[str, Any] = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
                               "norm": {"eps": self.norm_eps}, "layers": []}
        if self.logit_softcap:
            out["logit_softcap"] = self.logit_softcap
        for layer in self.layers:
            m = layer["mixer"]
            keys = (("heads", "kv_heads", "dim", "vdim", "scale") if layer["type"] == "attention"
                    else ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank", "scale"))
            mixer: Dict[str, Any] = {k: m[k] for k in keys}
            if m["rot"]:
                mixer["rot"] = {"base": m["rot"]["base"], "dims": m["rot"]["dims"]}
                if m["rot"]["scaling"]:
                    mixer["rot"]["scaling"] = dict(m["rot"]["scaling"])
            if m.get("conv"):
                mixer["conv"] = m["conv"]
            if m.get("window"):
                mixer["mask"] = {"size": m["window"]}
            if m.get("kv_from") is not None:
                mixer["kv_from"] = m["kv_from"]
            mlp, j = layer["mlp"], None
            if mlp is not None:
                limit = {} if mlp["limit"] is None else {"limit": mlp["limit"]}
                j = (dict({"kind": "dense", "ff": mlp["ff"]}, **limit) if mlp["kind"] == "dense" else
                     {"kind": "moe", "expert": dict({"ff": mlp["ff"]}, **limit),
                      "router": {"experts": mlp["experts"], "top": mlp["top"]}})
            out["layers"].append({"type": layer["type"], "mixer": mixer, "mlp": j})
        return out
