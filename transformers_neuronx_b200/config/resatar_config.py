"""Typed configuration of the Resatar decoder, read from the keys of its own config.json.

    {"architecture": "Resatar", "vocab": V, "width": W, "norm": {"eps": e},
     "layers": [{"type": ..., "mixer": {...}, "mlp": {...} | null}, ...]}

A layer's `type` names its mixer:
  'attention'  heads, kv_heads, dim, vdim, scale, optionally rot {dims, base, optionally scaling {factor, low, high,
               original}} and v_mix (true: the layer mixes its values with those of the first such layer)
  'mamba1'     inner, dt_rank, state, conv (taps)
  'parallel'   left {heads, kv_heads, dim, vdim, scale, optionally mask {size, keep_first}}, right {heads, dim, vdim,
               decay: one number a head}, left_scale, right_scale
A layer's `mlp` is {"kind": "dense", "ff": F}, or {"kind": "moe", "expert": {"ff": F}, "router": {"experts": E, "top": k},
optionally "shared": {"ff": S}}, or null.  Every layer carries its own sizes, so layers of one model may differ.  Nothing
has a default but `init_std` (the spread of random weights, used only when a folder is written from a seed) and
`max_positions` (the longest request the engine admits; the design itself has no limit); a mechanism whose key is absent
is not there (`rot`, `scaling`, `mask`, `shared`: none; `v_mix`: false; `keep_first`: 0; `kv_heads`: as many as heads).
"""
from __future__ import annotations

import copy
import json
import os
from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple

from .model_config import ConfigError

LAYER_TYPES = ("attention", "mamba1", "parallel")


def _pos_int(d, key, where):
    v = d.get(key)
    if not isinstance(v, int) or isinstance(v, bool) or v <= 0:
        raise ConfigError(f"{where}: key {key!r} must be a positive integer, got {v!r}")
    return v


def _number(d, key, where):
    v = d.get(key)
    if not isinstance(v, (int, float)) or isinstance(v, bool):
        raise ConfigError(f"{where}: key {key!r} must be a number, got {v!r}")
    return float(v)


def _positive(d, key, where):
    v = _number(d, key, where)
    if not (v > 0):
        raise ConfigError(f"{where}: key {key!r} must be positive, got {v!r}")
    return v


def _section(d, key, where, what):
    v = d.get(key)
    if not isinstance(v, dict):
        raise ConfigError(f"{where}: key {key!r} must hold {what}")
    return v


def _check_heads(m, where):
    if isinstance(m.get("heads"), int):
        m.setdefault("kv_heads", m["heads"])
    for k in ("heads", "kv_heads", "dim", "vdim"):
        _pos_int(m, k, where)
    if m["heads"] % m["kv_heads"]:
        raise ConfigError(f"{where}: {m['heads']} heads cannot share {m['kv_heads']} key/value heads")
    _positive(m, "scale", where)


def _check_attention(m, where):
    _check_heads(m, where)
    if not isinstance(m.setdefault("v_mix", False), bool):
        raise ConfigError(f"{where}: key 'v_mix' must be true or false, got {m['v_mix']!r}")
    if m.get("rot") is None:
        return
    rot, rw = _section(m, "rot", where, "'dims' and 'base'"), where + ".rot"
    if _pos_int(rot, "dims", rw) > m["dim"] or rot["dims"] % 2:
        raise ConfigError(f"{rw}: {rot['dims']} rotated dims do not fit heads of {m['dim']}")
    _positive(rot, "base", rw)
    if rot.get("scaling") is None:
        return
    sc, sw = _section(rot, "scaling", rw, "'factor', 'low', 'high' and 'original'"), rw + ".scaling"
    for k in ("factor", "low", "high", "original"):
        _positive(sc, k, sw)
    if sc["high"] <= sc["low"]:
        raise ConfigError(f"{sw}: 'high' ({sc['high']}) must exceed 'low' ({sc['low']})")


def _check_mamba(m, where):
    for k in ("inner", "dt_rank", "state", "conv"):
        _pos_int(m, k, where)


def _check_parallel(m, where):
    left, lw = _section(m, "left", where, "the attention's sizes"), where + ".left"
    _check_heads(left, lw)
    if left.get("mask") is not None:
        mask = _section(left, "mask", lw, "'size' and 'keep_first'")
        _pos_int(mask, "size", lw + ".mask")
        keep = mask.setdefault("keep_first", 0)
        if not isinstance(keep, int) or isinstance(keep, bool) or keep < 0:
            raise ConfigError(f"{lw}.mask: key 'keep_first' must be a number of positions, got {keep!r}")
    right, rw = _section(m, "right", where, "the recurrence's sizes"), where + ".right"
    for k in ("heads", "dim", "vdim"):
        _pos_int(right, k, rw)
    decay = right.get("decay")
    if not isinstance(decay, list) or len(decay) != right["heads"]:
        raise ConfigError(f"{rw}: key 'decay' must list one number for each of the {right['heads']} heads")
    for i, d in enumerate(decay):
        if not isinstance(d, (int, float)) or isinstance(d, bool):
            raise ConfigError(f"{rw}: decay[{i}] must be a number, got {d!r}")
    _number(m, "left_scale", where)
    _number(m, "right_scale", where)


def _check_mlp(mlp, where):
    if mlp is None:
        return
    if not isinstance(mlp, dict) or mlp.get("kind") not in ("dense", "moe"):
        raise ConfigError(f"{where}: kind must be 'dense' or 'moe' (or the layer's mlp null), got {mlp!r}")
    if mlp["kind"] == "dense":
        _pos_int(mlp, "ff", where)
        return
    _pos_int(_section(mlp, "expert", where, "'ff'"), "ff", where + ".expert")
    r, rw = _section(mlp, "router", where, "'experts' and 'top'"), where + ".router"
    E, top = _pos_int(r, "experts", rw), _pos_int(r, "top", rw)
    if top > E:
        raise ConfigError(f"{rw}: {top} of {E} experts is not a choice")
    if mlp.get("shared") is not None:
        _pos_int(_section(mlp, "shared", where, "'ff'"), "ff", where + ".shared")


def _check_layer(i: int, layer: Dict[str, Any]) -> None:
    where = f"layers[{i}]"
    if not isinstance(layer, dict) or layer.get("type") not in LAYER_TYPES:
        t = layer.get("type") if isinstance(layer, dict) else layer
        raise ConfigError(f"{where}: unknown layer type {t!r}; known: {', '.join(LAYER_TYPES)}")
    m = _section(layer, "mixer", where, "the mixer's sizes")
    {"attention": _check_attention, "mamba1": _check_mamba, "parallel": _check_parallel}[layer["type"]](m, where + ".mixer")
    _check_mlp(layer.get("mlp"), where + ".mlp")


@dataclass(frozen=True, eq=False)
class ResatarConfig:
    vocab: int
    width: int
    layers: Tuple[Dict[str, Any], ...]
    norm_eps: float
    init_std: float = 0.05
    max_positions: int = 1 << 20
    architecture: str = "Resatar"

    def __post_init__(self):
        for name in ("vocab", "width", "max_positions"):
            v = getattr(self, name)
            if not isinstance(v, int) or isinstance(v, bool) or v <= 0:
                raise ConfigError(f"config key {name!r} must be a positive integer, got {v!r}")
        if not (self.norm_eps > 0):
            raise ConfigError(f"norm.eps must be positive, got {self.norm_eps!r}")
        if not self.layers:
            raise ConfigError("config key 'layers' must list at least one layer")
        for i, layer in enumerate(self.layers):
            _check_layer(i, layer)
        first = self.first_mixing_layer
        for i, layer in enumerate(self.layers):
            if layer["type"] == "attention" and layer["mixer"]["v_mix"]:
                for k in ("kv_heads", "vdim"):
                    if layer["mixer"][k] != self.layers[first]["mixer"][k]:
                        raise ConfigError(f"layers[{i}].mixer: {k} differs from that of layer {first}, whose values it mixes in")

    def __eq__(self, other):
        return isinstance(other, ResatarConfig) and self.to_dict() == other.to_dict()

    @property
    def first_mixing_layer(self) -> Optional[int]:
        """The layer whose values the later layers with v_mix mix into theirs."""
        return next((i for i, l in enumerate(self.layers) if l["type"] == "attention" and l["mixer"]["v_mix"]), None)

    # what the engine's front door asks of any configuration
    @property
    def vocab_size(self) -> int:
        return self.vocab

    torch_dtype = "bfloat16"                 # the type the design's checkpoints are stored in

    @property
    def max_position_embeddings(self) -> int:
        return self.max_positions

    eos_token_id: Optional[int] = None
    bos_token_id: Optional[int] = None
    pad_token_id: Optional[int] = None

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "ResatarConfig":
        missing = [k for k in ("vocab", "width", "layers", "norm") if k not in d]
        if missing:
            raise ConfigError("config.json lacks required key(s): " + ", ".join(missing))
        if not isinstance(d["norm"], dict) or "eps" not in d["norm"]:
            raise ConfigError("config key 'norm' must hold 'eps'")
        if not isinstance(d["layers"], list):
            raise ConfigError("config key 'layers' must be a list")
        kw = dict(vocab=d["vocab"], width=d["width"], layers=tuple(copy.deepcopy(l) for l in d["layers"]),
                  norm_eps=_number(d["norm"], "eps", "norm"))
        for k in ("init_std", "max_positions"):
            if k in d:
                kw[k] = d[k]
        return cls(**kw)

    @classmethod
    def from_json(cls, path: str) -> "ResatarConfig":
        with open(path) as fp:
            return cls.from_dict(json.load(fp))

    @classmethod
    def from_pretrained(cls, folder: str) -> "ResatarConfig":
        return cls.from_json(os.path.join(folder, "config.json"))

    def to_dict(self) -> Dict[str, Any]:
        return {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
                "norm": {"eps": self.norm_eps}, "layers": [copy.deepcopy(l) for l in self.layers],
                "init_std": self.init_std, "max_positions": self.max_positions}

    def save(self, folder: str) -> None:
        os.makedirs(folder, exist_ok=True)
        with open(os.path.join(folder, "config.json"), "w") as fp:
            json.dump(self.to_dict(), fp, indent=1)
