"""Typed configuration of the Rapovik architecture.

config.json names the design with ``"architecture": "Rapovik"`` and describes the model layer by layer:

* ``vocab``, ``width``: vocabulary and residual width;
* ``norm`` = ``{"eps"}``: the epsilon of every RMS norm;
* ``layers``: a list of ``{"type", "mixer", "mlp"}``.  ``type`` is
  ``"latent_attention"`` (``heads``, ``dim`` = unrotated query/key size per head, ``rot_dim`` = rotated size, ``vdim``, ``kv_rank``,
  ``scale``, ``rot`` = ``{"dims", "base"}`` and optionally ``mask`` = ``{"size"}``, a sliding window of that many tokens),
  ``"mamba2"`` (``heads``, ``vdim``, ``state``, ``groups``, ``conv`` taps, ``norm_groups``) or
  ``"mlstm"`` (``heads``, ``dim``, ``vdim``, ``gate_cap``);
  ``mlp`` is null, ``{"kind": "dense", "ff", "limit"}`` or ``{"kind": "moe", "expert": {"ff", "limit"}, "router": {"experts",
  "top", "groups": {"count", "keep"}}, "shared": {"ff", "limit"}}`` (``groups`` and ``shared`` optional);
* ``loop`` = ``{"start", "stop", "times"}`` (optional): layers start..stop-1 run ``times`` times in a row with the same weights,
  every run with a cache or state of its own.

``max_position_embeddings`` and ``eos_token_id`` are optional additions of this engine.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple

from .base import ConfigError, ModelConfig, token_id_list

LATENT_ATTENTION, MAMBA2, MLSTM = "latent_attention", "mamba2", "mlstm"
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


def _check_mixer(kind: Any, m: Dict[str, Any], where: str) -> None:
    if kind == LATENT_ATTENTION:
        for key in ("heads", "dim", "rot_dim", "vdim", "kv_rank"):
            _int(m, key, where)
        _float(m, "scale", where)
        rot = _object(m, "rot", where, "'dims' and 'base'")
        dims = _int(rot, "dims", where + "rot: ", 2)
        if dims % 2 or dims > m["rot_dim"]:
            raise ConfigError(f"config.json: {where}rot.dims={dims} must be even and at most rot_dim={m['rot_dim']}")
        _float(rot, "base", where + "rot: ", positive=True)
        if m.get("mask") is not None:
            _int(_object(m, "mask", where, "'size'"), "size", where + "mask: ")
    elif kind == MAMBA2:
        for key in ("heads", "vdim", "state", "groups", "conv", "norm_groups"):
            _int(m, key, where)
        if m["heads"] % m["groups"]:
            raise ConfigError(f"config.json: {where}{m['heads']} heads are not a multiple of {m['groups']} groups")
        if (m["heads"] * m["vdim"]) % m["norm_groups"]:
            raise ConfigError(f"config.json: {where}{m['heads'] * m['vdim']} values cannot be normalised in norm_groups={m['norm_groups']} equal parts")
    elif kind == MLSTM:
        for key in ("heads", "dim", "vdim"):
            _int(m, key, where)
        _float(m, "gate_cap", where, positive=True)
    else:
        raise ConfigError(f"config.json: {where}unknown layer type {kind!r} ({LATENT_ATTENTION}, {MAMBA2}, {MLSTM})")


def _check_mlp(mlp: Any, where: str) -> None:
    if mlp is None:
        return
    if not isinstance(mlp, dict) or mlp.get("kind") not in ("dense", "moe"):
        raise ConfigError(f"config.json: {where}mlp must be null or of kind 'dense' or 'moe', got {mlp!r}")
    where += "mlp"
    if mlp["kind"] == "dense":
        _int(mlp, "ff", where + ": "); _float(mlp, "limit", where + ": ", positive=True)
        return
    for key in ("expert", "shared"):
        if key == "expert" or mlp.get("shared") is not None:
            part = _object(mlp, key, where + ": ", "'ff' and 'limit'")
            _int(part, "ff", f"{where}.{key}: "); _float(part, "limit", f"{where}.{key}: ", positive=True)
    r = _object(mlp, "router", where + ": ", "'experts' and 'top'")
    where += ".router: "
    experts, top = _int(r, "experts", where), _int(r, "top", where)
    if top > experts:
        raise ConfigError(f"config.json: {where}top={top} of {experts} experts")
    if r.get("groups") is not None:
        groups = _object(r, "groups", where, "'count' and 'keep'")
        count, keep = _int(groups, "count", where + "groups: "), _int(groups, "keep", where + "groups: ")
        if experts % count or keep > count or keep * (experts // count) < top:
            raise ConfigError(f"config.json: {where}{experts} experts in {count} groups of which {keep} are kept cannot give {top}")


@dataclass(frozen=True)
class RapovikConfig(ModelConfig):
    width: int = 0
    layers: Tuple[Dict[str, Any], ...] = ()
    loop: Optional[Tuple[int, int, int]] = None      # (start, stop, times)
    norm_eps: float = 1e-6

    @classmethod
    def from_dict(cls, raw: Dict[str, Any]) -> "RapovikConfig":
        vocab, width = _int(raw, "vocab", ""), _int(raw, "width", "")
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: 'layers' must be a list with at least one layer")
        checked = []
        for i, layer in enumerate(layers):
            where = f"layers[{i}]: "
            if not isinstance(layer, dict) or not isinstance(layer.get("mixer"), dict):
                raise ConfigError(f"config.json: {where}an object with 'type', 'mixer' and 'mlp' is expected")
            _check_mixer(layer.get("type"), layer["mixer"], where)
            _check_mlp(layer.get("mlp"), where)
            checked.append({"type": layer["type"], "mixer": copy.deepcopy(layer["mixer"]), "mlp": copy.deepcopy(layer.get("mlp"))})
        loop = None
        if raw.get("loop") is not None:
            lp = _object(raw, "loop", "", "'start', 'stop' and 'times'")
            start, stop, times = _int(lp, "start", "loop: ", 0), _int(lp, "stop", "loop: ", 0), _int(lp, "times", "loop: ")
            if not start <= stop <= len(checked):
                raise ConfigError(f"config.json: loop {start}..{stop} does not lie within the {len(checked)} layers")
            loop = (start, stop, times)
        eps = _float(_object(raw, "norm", "", "'eps'"), "eps", "norm: ", positive=True)
        max_pos = raw.get("max_position_embeddings")
        max_pos = DEFAULT_MAX_POSITIONS if max_pos is None else _int(raw, "max_position_embeddings", "")
        eos = token_id_list(raw.get("eos_token_id"))
        for t in raw.get("_generation_eos_token_ids", []):
            if t not in eos:
                eos.append(t)
        return cls(architecture="Rapovik", vocab_size=vocab, max_position_embeddings=max_pos, eos_token_ids=tuple(eos),
                   width=width, layers=tuple(checked), loop=loop, norm_eps=eps)

    def layer_runs(self) -> Tuple[int, ...]:
        """The layers' indices in the order they run."""
        n = len(self.layers)
        if self.loop is None:
            return tuple(range(n))
        start, stop, times = self.loop
        return tuple(range(start)) + tuple(range(start, stop)) * times + tuple(range(stop, n))

    def to_json_dict(self) -> Dict[str, Any]:
        out: Dict[str, Any] = {"architecture": "Rapovik", "vocab": self.vocab_size, "width": self.width,
                               "layers": copy.deepcopy(list(self.layers)), "norm": {"eps": self.norm_eps}}
        if self.loop is not None:
            out["loop"] = {"start": self.loop[0], "stop": self.loop[1], "times": self.loop[2]}
        if self.max_position_embeddings != DEFAULT_MAX_POSITIONS:
            out["max_position_embeddings"] = self.max_position_embeddings
        if self.eos_token_ids:
            out["eos_token_id"] = list(self.eos_token_ids) if len(self.eos_token_ids) > 1 else self.eos_token_ids[0]
        return out


def sketch_config(vocab: int, width: int, n_layers: int, heads: int, head_dim: int, ff: int, kv_rank: Optional[int] = None,
                  window: int = 0, experts: int = 16, top: int = 4, groups: Tuple[int, int] = (4, 2),
                  loop: Optional[Tuple[int, int, int]] = None, max_positions: int = DEFAULT_MAX_POSITIONS, eps: float = 1e-5,
                  rope_base: float = 10000.0) -> RapovikConfig:
    """A configuration of the usual proportions from a few sizes, for random-weight models (the command line's ``tiny-model``,
    measurements): layers go state space, matrix memory, latent attention and again, the first with a dense feed-forward and the
    others with mixtures of experts; state heads of ``head_dim`` filling the width, attention heads of ``head_dim`` unrotated and
    half as many rotated elements, a latent of ``kv_rank`` (default: a quarter of the width)."""
    rot = max(2, head_dim // 4 * 2)
    r = kv_rank or max(8, width // 32 * 8)
    eff = max(8, ff // top // 8 * 8)
    n = max(1, width // head_dim)
    g = 2 if n % 2 == 0 else 1
    kinds = (MAMBA2, MLSTM, LATENT_ATTENTION)
    layers = []
    for i in range(n_layers):
        kind = kinds[i % 3]
        if kind == MAMBA2:
            m: Dict[str, Any] = {"heads": n, "vdim": head_dim, "state": head_dim, "groups": g, "conv": 4, "norm_groups": g}
        elif kind == MLSTM:
            m = {"heads": n, "dim": head_dim, "vdim": head_dim, "gate_cap": 15.0}
        else:
            m = {"heads": heads, "dim": head_dim, "rot_dim": rot, "vdim": head_dim, "kv_rank": r, "scale": (head_dim + rot) ** -0.5,
                 "rot": {"dims": rot, "base": rope_base}}
            if window > 0:
                m["mask"] = {"size": window}
        mlp: Dict[str, Any] = {"kind": "dense", "ff": ff, "limit": 7.0}
        if i > 0:
            mlp = {"kind": "moe", "expert": {"ff": eff, "limit": 7.0}, "shared": {"ff": eff * 2, "limit": 7.0},
                   "router": {"experts": experts, "top": top, "groups": {"count": groups[0], "keep": groups[1]}}}
        layers.append({"type": kind, "mixer": m, "mlp": mlp})
    raw: Dict[str, Any] = {"architecture": "Rapovik", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps},
                           "max_position_embeddings": max_positions}
    if loop is not None:
        raw["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return RapovikConfig.from_dict(raw)
