"""Typed configuration of the Lanirax architecture.

config.json names the design with ``"architecture": "Lanirax"`` and describes the model layer by layer:

* ``vocab``, ``width``: vocabulary and residual width; ``norm`` = ``{"eps"}``: the epsilon of every RMS norm;
* ``postln_alpha``: the weight of the residual in the sum that a layer's norms are taken of;
* ``layers``: a list of ``{"type", "mixer", "mlp"}`` and optionally ``"weights_of": j`` (the layer has no tensors of its own
  and runs layer j's, with a cache of its own; sizes and constants are then layer j's).  ``type`` is
  ``"attention"`` (``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, and optionally ``q_temp`` = ``{"coef", "every"}``, the
  growth of the query's temperature with its position) or
  ``"parallel"`` (two mixers side by side: ``left`` = attention whose values are the projected keys, with ``heads``,
  ``kv_heads``, ``dim``, ``vdim`` (= ``dim``), ``scale``, ``mask`` = ``{"size"}``, a sliding window of that many tokens, ``rot`` =
  ``{"dims", "base", "scaling"}``, the scaling (optional) with ``factor``, ``original``, ``fast``, ``slow``; ``right`` = the gated
  delta rule with one decay per head, with ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``conv`` taps);
  ``mlp`` is null or ``{"kind": "moe", "expert": {"ff"}, "router": {"experts", "top"}}``.

``kv_heads`` left out means as many as ``heads``.  ``max_position_embeddings`` and ``eos_token_id`` are optional additions of
this engine.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Dict, Tuple

from .base import ConfigError, ModelConfig, token_id_list

ATTENTION, PARALLEL = "attention", "parallel"
DEFAULT_MAX_POSITIONS = 32768


def _int(d: Dict[str, Any], key: str, where: str, minimum: int = 1) -> int:
    v = d.get(key)
    if isinstance(v, bool) or not isinstance(v, int) or v < minimum:
        raise ConfigError(f"config.json: {where}'{key}' must be an integer >= {minimum}, got {v!r}")
    return v


def _float(d: Dict[str, Any], key: str, where: str, positive: bool = False) -> float:
    v = d.get(key)
    if isinstance(v, bool) or not isinstance(v, (int, float)):
        raise ConfigError(f"config.json: {where}'{key}' must be a number, got {v!r}")
    if positive and v <= 0.0:
        raise ConfigError(f"config.json: {where}'{key}' must be positive, got {v!r}")
    return float(v)


def _object(d: Dict[str, Any], key: str, where: str, content: str) -> Dict[str, Any]:
    v = d.get(key)
    if not isinstance(v, dict):
        raise ConfigError(f"config.json: {where}'{key}' must be an object with {content}")
    return v


def _heads(m: Dict[str, Any], where: str) -> None:
    m.setdefault("kv_heads", m.get("heads"))
    heads, kv = _int(m, "heads", where), _int(m, "kv_heads", where)
    if heads % kv:
        raise ConfigError(f"config.json: {where}{heads} heads are not a multiple of {kv} kv_heads")
    _int(m, "dim", where)


def _check_rot(m: Dict[str, Any], where: str) -> None:
    if m.get("rot") is None:
        return
    rot = _object(m, "rot", where, "'dims' and 'base'")
    where += "rot: "
    dims = _int(rot, "dims", where, 2)
    if dims % 2 or dims > m["dim"]:
        raise ConfigError(f"config.json: {where}dims={dims} must be even and at most dim={m['dim']}")
    _float(rot, "base", where, positive=True)
    if rot.get("scaling") is not None:
        scaling = _object(rot, "scaling", where, "'factor', 'original', 'fast' and 'slow'")
        for key in ("factor", "original", "fast", "slow"):
            _float(scaling, key, where + "scaling: ", positive=True)
        if rot["base"] == 1:
            raise ConfigError(f"config.json: {where}a scaled rotation needs a base other than 1")


def _check_mixer(kind: Any, m: Dict[str, Any], where: str) -> None:
    if kind == ATTENTION:
        _heads(m, where)
        m.setdefault("vdim", m["dim"])
        _int(m, "vdim", where); _float(m, "scale", where)
        if m.get("q_temp") is not None:
            temp = _object(m, "q_temp", where, "'coef' and 'every'")
            _float(temp, "coef", where + "q_temp: "); _float(temp, "every", where + "q_temp: ", positive=True)
    elif kind == PARALLEL:
        left, right = _object(m, "left", where, "an attention's sizes"), _object(m, "right", where, "a delta rule's sizes")
        at = where + "left: "
        _heads(left, at)
        left.setdefault("vdim", left["dim"])
        if _int(left, "vdim", at) != left["dim"]:
            raise ConfigError(f"config.json: {at}the values are the projected keys, so vdim must equal dim={left['dim']}")
        _float(left, "scale", at, positive=True)
        _check_rot(left, at)
        if left.get("mask") is not None:
            _int(_object(left, "mask", at, "'size'"), "size", at + "mask: ")
        at = where + "right: "
        _heads(right, at)
        _int(right, "vdim", at); _int(right, "conv", at)
    else:
        raise ConfigError(f"config.json: {where}unknown layer type {kind!r} ({ATTENTION}, {PARALLEL})")


def _check_mlp(mlp: Any, where: str) -> None:
    if mlp is None:
        return
    if not isinstance(mlp, dict) or mlp.get("kind") != "moe":
        raise ConfigError(f"config.json: {where}mlp must be null or of kind 'moe', got {mlp!r}")
    where += "mlp."
    _int(_object(mlp, "expert", where, "'ff'"), "ff", where + "expert: ")
    router = _object(mlp, "router", where, "'experts' and 'top'")
    experts, top = _int(router, "experts", where + "router: "), _int(router, "top", where + "router: ")
    if top > experts:
        raise ConfigError(f"config.json: {where}router: top={top} of {experts} experts")


def weight_owner(layers, i: int) -> int:
    """The layer whose tensors layer ``i`` runs (itself, unless it names another with ``weights_of``)."""
    seen = set()
    while layers[i].get("weights_of") is not None:
        if i in seen:
            raise ConfigError(f"config.json: layers[{i}]: 'weights_of' goes in a circle")
        seen.add(i)
        i = layers[i]["weights_of"]
    return i


@dataclass(frozen=True)
class LaniraxConfig(ModelConfig):
    width: int = 0
    layers: Tuple[Dict[str, Any], ...] = ()
    norm_eps: float = 1e-6
    alpha: float = 1.0

    @classmethod
    def from_dict(cls, raw: Dict[str, Any]) -> "LaniraxConfig":
        vocab, width = _int(raw, "vocab", ""), _int(raw, "width", "")
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: 'layers' must be a list with at least one layer")
        checked = []
        for i, layer in enumerate(layers):
            where = f"layers[{i}]: "
            if not isinstance(layer, dict) or not isinstance(layer.get("mixer"), dict):
                raise ConfigError(f"config.json: {where}an object with 'type', 'mixer' and 'mlp' is expected")
            layer = copy.deepcopy(layer)
            _check_mixer(layer.get("type"), layer["mixer"], where)
            _check_mlp(layer.get("mlp"), where)
            out = {"type": layer["type"], "mixer": layer["mixer"], "mlp": layer.get("mlp")}
            if layer.get("weights_of") is not None:
                out["weights_of"] = _int(layer, "weights_of", where, 0)
            checked.append(out)
        for i, layer in enumerate(checked):
            j = layer.get("weights_of")
            if j is None:
                continue
            if j >= len(checked) or j == i:
                raise ConfigError(f"config.json: layers[{i}]: 'weights_of' must name another layer, got {j}")
            weight_owner(checked, i)           # refuses a circle
        eps = _float(_object(raw, "norm", "", "'eps'"), "eps", "norm: ", positive=True)
        alpha = _float(raw, "postln_alpha", "")
        max_pos = raw.get("max_position_embeddings")
        max_pos = DEFAULT_MAX_POSITIONS if max_pos is None else _int(raw, "max_position_embeddings", "")
        eos = token_id_list(raw.get("eos_token_id"))
        for t in raw.get("_generation_eos_token_ids", []):
            if t not in eos:
                eos.append(t)
        return cls(architecture="Lanirax", vocab_size=vocab, max_position_embeddings=max_pos, eos_token_ids=tuple(eos),
                   width=width, layers=tuple(checked), norm_eps=eps, alpha=alpha)

    def to_json_dict(self) -> Dict[str, Any]:
        out: Dict[str, Any] = {"architecture": "Lanirax", "vocab": self.vocab_size, "width": self.width,
                               "layers": copy.deepcopy(list(self.layers)), "norm": {"eps": self.norm_eps}, "postln_alpha": self.alpha}
        if self.max_position_embeddings != DEFAULT_MAX_POSITIONS:
            out["max_position_embeddings"] = self.max_position_embeddings
        if self.eos_token_ids:
            out["eos_token_id"] = list(self.eos_token_ids) if len(self.eos_token_ids) > 1 else self.eos_token_ids[0]
        return out


def sketch_config(vocab: int, width: int, n_layers: int, heads: int, kv_heads: int, head_dim: int, ff: int, window: int = 256,
                  experts: int = 16, top: int = 4, alpha: float = 1.5, taps: int = 4, max_positions: int = DEFAULT_MAX_POSITIONS,
                  eps: float = 1e-5, rope_base: float = 10000.0, shared_from: int = 0) -> LaniraxConfig:
    """A configuration of the usual proportions from a few sizes, for random-weight models (the command line's
    ``tiny-model``, measurements): layers go parallel, attention and again; attention heads of ``head_dim``, rotated over half
    of it; state heads of ``head_dim`` filling the width; ``ff`` is the width all of a token's experts have together.
    ``shared_from`` > 0: the layers from that index on run the weights of the layer that many places before them."""
    n = max(1, width // head_dim)
    expert = {"kind": "moe", "expert": {"ff": max(8, ff // top // 8 * 8)}, "router": {"experts": experts, "top": top}}
    layers = []
    for i in range(n_layers):
        if i % 2 == 0:
            kind, m = PARALLEL, {
                "left": {"heads": heads, "kv_heads": kv_heads, "dim": head_dim, "vdim": head_dim, "scale": head_dim ** -0.5,
                         "mask": {"size": window},
                         "rot": {"dims": max(2, head_dim // 4 * 2), "base": rope_base,
                                 "scaling": {"factor": 4.0, "original": 2048, "fast": 32.0, "slow": 1.0}}},
                "right": {"heads": n, "kv_heads": n // 2 if n % 2 == 0 else n, "dim": head_dim, "vdim": head_dim, "conv": taps}}
        else:
            kind, m = ATTENTION, {"heads": heads, "kv_heads": kv_heads, "dim": head_dim, "vdim": head_dim, "scale": head_dim ** -0.5,
                                  "q_temp": {"coef": 0.1, "every": 1024}}
        layer = {"type": kind, "mixer": m, "mlp": copy.deepcopy(expert)}
        if shared_from > 0 and i >= shared_from:
            layer["weights_of"] = i - shared_from
        layers.append(layer)
    return LaniraxConfig.from_dict({"architecture": "Lanirax", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps},
                                    "postln_alpha": alpha, "max_position_embeddings": max_positions})
