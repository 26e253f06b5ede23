"""Typed configuration of the Taborax decoder, read from the keys of its own config.json.

    {"architecture": "Taborax", "vocab": V, "width": W, "norm": {"eps": e}, "loop": {"start": a, "stop": b, "times": n},
     "layers": [{"type": ..., "mixer": {...}, "mlp": {...} | null}, ...]}

A layer's `type` names its mixer:
  'latent_attention'  heads, dim, vdim, q_rank, kv_rank, scale
  'attention'         heads, kv_heads, dim, vdim (= dim: the values are the keys), scale, rot {dims, base}
A layer's `mlp` is {"kind": "dense", "ff": F}, or {"kind": "moe", "expert": {"ff": F}, "router": {"experts": E, "top": k,
"groups": {"count": g, "keep": n}, "identity": i}, "shared": {"ff": S}}, or null.  The router has E + i outputs, the last i
of which are identity experts.  `loop`: the layers from `start` up to (not with) `stop` are walked `times` times.  Every
layer carries its own sizes, so layers of one model may differ.  Nothing has a default but `init_std` (the spread of random
weights, used only when a folder is written from a seed) and `max_positions` (the longest request the engine admits; the
design itself has no limit); a mechanism whose key is absent or null is not there (`loop`, `rot`, `groups`, `identity`,
`shared`, `mlp`).
"""
from __future__ import annotations

import copy
import json
import os
from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple

from .model_config import ConfigError

LAYER_TYPES = ("latent_attention", "attention")


def _pos_int(d, key, where):
    v = d.get(key)
    if not isinstance(v, int) or isinstance(v, bool) or v <= 0:
        raise ConfigError(f"{where}: key {key!r} must be a positive integer, got {v!r}")
    return v


def _count(d, key, where):
    """A whole number that may be 0 or absent (then 0)."""
    v = d.get(key)
    v = 0 if v is None else v
    if not isinstance(v, int) or isinstance(v, bool) or v < 0:
        raise ConfigError(f"{where}: key {key!r} must be a whole number, got {v!r}")
    return v


def _positive(d, key, where):
    v = d.get(key)
    if not isinstance(v, (int, float)) or isinstance(v, bool) or not (v > 0):
        raise ConfigError(f"{where}: key {key!r} must be a positive number, got {v!r}")
    return float(v)


def _section(d, key, where, what):
    v = d.get(key)
    if not isinstance(v, dict):
        raise ConfigError(f"{where}: key {key!r} must hold {what}")
    return v


def _check_mixer(kind, m, where):
    for k in ("heads", "dim", "vdim"):
        _pos_int(m, k, where)
    _positive(m, "scale", where)
    if kind == "latent_attention":
        _pos_int(m, "q_rank", where)
        _pos_int(m, "kv_rank", where)
        return
    if m["heads"] % _pos_int(m, "kv_heads", where):
        raise ConfigError(f"{where}: {m['heads']} heads cannot share {m['kv_heads']} key/value heads")
    if m["vdim"] != m["dim"]:
        raise ConfigError(f"{where}: the values are the keys, so vdim must equal dim ({m['vdim']} and {m['dim']})")
    if m.get("rot") is None:
        return
    rot, rw = _section(m, "rot", where, "'dims' and 'base'"), where + ".rot"
    dims = _count(rot, "dims", rw)
    if dims % 2 or dims > m["dim"]:
        raise ConfigError(f"{rw}: {dims} rotated dims do not fit heads of {m['dim']}")
    _positive(rot, "base", rw)


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
    outputs = _pos_int(r, "experts", rw) + _count(r, "identity", rw)
    open_to = outputs
    if r.get("groups") is not None:
        g, gw = _section(r, "groups", rw, "'count' and 'keep'"), rw + ".groups"
        count, keep = _pos_int(g, "count", gw), _pos_int(g, "keep", gw)
        if outputs % count or keep > count:
            raise ConfigError(f"{gw}: {keep} of {count} equal groups of {outputs} experts is not a choice")
        open_to = keep * (outputs // count)
    if _pos_int(r, "top", rw) > open_to:
        raise ConfigError(f"{rw}: {r['top']} of {open_to} experts is not a choice")
    if mlp.get("shared") is not None:
        _pos_int(_section(mlp, "shared", where, "'ff'"), "ff", where + ".shared")


def _check_layer(i: int, layer: Dict[str, Any]) -> None:
    where = f"layers[{i}]"
    if not isinstance(layer, dict) or layer.get("type") not in LAYER_TYPES:
        t = layer.get("type") if isinstance(layer, dict) else layer
        raise ConfigError(f"{where}: unknown layer type {t!r}; known: {', '.join(LAYER_TYPES)}")
    _check_mixer(layer["type"], _section(layer, "mixer", where, "the mixer's sizes"), where + ".mixer")
    _check_mlp(layer.get("mlp"), where + ".mlp")


@dataclass(frozen=True, eq=False)
class TaboraxConfig:
    vocab: int
    width: int
    layers: Tuple[Dict[str, Any], ...]
    norm_eps: float
    loop: Optional[Dict[str, int]] = None
    init_std: float = 0.05
    max_positions: int = 1 << 20
    architecture: str = "Taborax"

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
        if self.loop is not None:
            if not isinstance(self.loop, dict):
                raise ConfigError("config key 'loop' must hold start, stop and times")
            a = _count(self.loop, "start", "loop")
            b, _ = _pos_int(self.loop, "stop", "loop"), _pos_int(self.loop, "times", "loop")
            if not (a < b <= len(self.layers)):
                raise ConfigError(f"loop: layers {a} .. {b} - 1 are not a run of the model's {len(self.layers)} layers")

    def __eq__(self, other):
        return isinstance(other, TaboraxConfig) and self.to_dict() == other.to_dict()

    def layer_runs(self):
        """[(layer, whether a pass of the loop begins with it)] in the order they run."""
        n = len(self.layers)
        if self.loop is None:
            return [(i, False) for i in range(n)]
        a, b, times = self.loop.get("start") or 0, self.loop["stop"], self.loop["times"]
        one_pass = [(i, i == a) for i in range(a, b)]
        return [(i, False) for i in range(a)] + one_pass * times + [(i, False) for i in range(b, n)]

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
    def from_dict(cls, d: Dict[str, Any]) -> "TaboraxConfig":
        missing = [k for k in ("vocab", "width", "layers", "norm") if k not in d]
        if missing:
            raise ConfigError("config.json lacks required key(s): " + ", ".join(missing))
        if not isinstance(d["layers"], list):
            raise ConfigError("config key 'layers' must be a list")
        kw = dict(vocab=d["vocab"], width=d["width"], layers=tuple(copy.deepcopy(l) for l in d["layers"]),
                  norm_eps=_positive(_section(d, "norm", "config", "'eps'"), "eps", "norm"),
                  loop=copy.deepcopy(d.get("loop")))
        for k in ("init_std", "max_positions"):
            if k in d:
                kw[k] = d[k]
        return cls(**kw)

    @classmethod
    def from_json(cls, path: str) -> "TaboraxConfig":
        with open(path) as fp:
            return cls.from_dict(json.load(fp))

    @classmethod
    def from_pretrained(cls, folder: str) -> "TaboraxConfig":
        return cls.from_json(os.path.join(folder, "config.json"))

    def to_dict(self) -> Dict[str, Any]:
        d = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
             "layers": [copy.deepcopy(l) for l in self.layers], "init_std": self.init_std,
             "max_positions": self.max_positions}
        if self.loop is not None:
            d["loop"] = copy.deepcopy(self.loop)
        return d

    def save(self, folder: str) -> None:
        os.makedirs(folder, exist_ok=True)
        with open(os.path.join(folder, "config.json"), "w") as fp:
            json.dump(self.to_dict(), fp, indent=1)
