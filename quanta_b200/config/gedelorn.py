"""Typed configuration of the Gedelorn decoder, from config.json.

The file is nested: ``vocab``, ``width``, ``norm.eps`` and ``layers``, a list in run order whose entries give the layer's
``type``, the mixer's sizes and constants (``mixer``) and its feed-forward (``mlp``; null for a layer with a mixer only).

* ``mlstm``: ``heads``, ``dim``, ``vdim``, ``gate_cap``.
* ``mamba2``: ``heads``, ``vdim``, ``state``, ``groups``, ``conv`` (taps), ``norm_groups``.
* ``parallel``: ``left`` (``heads``, ``kv_heads``, ``dim``, ``scale``, ``softcap``, ``mask.size``, ``rot.dims`` / ``rot.base``; the
  values are the keys, so ``vdim`` equals ``dim``), ``right`` (``heads``, ``dim``, ``vdim``, ``decay``: one number a head),
  ``left_scale``, ``right_scale``.
* ``mlp.kind`` ``dense``: ``ff``; ``moe``: ``expert.ff``, ``router`` (``experts``, ``top``, ``scale``), ``shared.ff``.

Every size and constant the layers use is read here; what the layers cannot run is refused.
"""

from __future__ import annotations

import copy
from dataclasses import dataclass, field

from .minimax_m3 import ConfigError

MAX_HEAD_SIZE = 256
_NEEDS = {
    "mlstm": ("heads", "dim", "vdim", "gate_cap"),
    "mamba2": ("heads", "vdim", "state", "groups", "conv", "norm_groups"),
    "parallel": ("left", "right", "left_scale", "right_scale"),
}
_LEFT = ("heads", "kv_heads", "dim", "scale", "softcap", "mask", "rot")
_RIGHT = ("heads", "dim", "vdim", "decay")


@dataclass(frozen=True)
class GedelornLayer:
    type: str
    mixer: dict
    mlp: dict | None


def _need(where: str, d: dict, keys) -> None:
    missing = [k for k in keys if k not in d]
    if missing:
        raise ConfigError(f"{where} lacks {missing}")


def _positive(where: str, d: dict, keys) -> None:
    for k in keys:
        if int(d[k]) <= 0:
            raise ConfigError(f"{where}.{k} must be positive")


def _key_size(where: str, n: int) -> None:
    if not 0 < n <= MAX_HEAD_SIZE:
        raise ConfigError(f"{where}: head sizes lie between 1 and {MAX_HEAD_SIZE}, got {n}")


def _check_parallel(where: str, m: dict) -> None:
    left, right = m["left"], m["right"]
    _need(f"{where}.left", left, _LEFT)
    _positive(f"{where}.left", left, ("heads", "kv_heads", "dim"))
    if int(left["heads"]) % int(left["kv_heads"]):
        raise ConfigError(f"{where}.left: {left['heads']} heads are not a multiple of {left['kv_heads']} kv heads")
    _key_size(f"{where}.left.dim", int(left["dim"]))
    if int(left.get("vdim", left["dim"])) != int(left["dim"]):
        raise ConfigError(f"{where}.left: the values are the keys, so vdim equals dim")
    if int(left["mask"].get("size", 0)) < 1:
        raise ConfigError(f"{where}.left.mask.size must hold at least the token itself")
    if not float(left["softcap"]) > 0:
        raise ConfigError(f"{where}.left.softcap must be positive")
    dims = int((left["rot"] or {}).get("dims") or 0)
    if dims < 0 or dims % 2 or dims > int(left["dim"]) or (dims and float(left["rot"].get("base", 0)) <= 0):
        raise ConfigError(f"{where}.left.rot: dims must be even and at most {left['dim']}, base positive")
    _need(f"{where}.right", right, _RIGHT)
    _positive(f"{where}.right", right, ("heads", "dim", "vdim"))
    _key_size(f"{where}.right.dim", int(right["dim"]))
    if len(right["decay"]) != int(right["heads"]) or any(not 0.0 <= float(d) <= 1.0 for d in right["decay"]):
        raise ConfigError(f"{where}.right.decay: one number from 0 to 1 for each of {right['heads']} heads")


def _check_mlp(where: str, mlp: dict) -> None:
    kind = mlp.get("kind")
    if kind == "dense":
        if int(mlp.get("ff", 0)) <= 0:
            raise ConfigError(f"{where}.ff must be positive")
        return
    if kind != "moe":
        raise ConfigError(f"{where}.kind {kind!r} is not 'dense' or 'moe'")
    _need(where, mlp, ("expert", "router"))
    _need(f"{where}.router", mlp["router"], ("experts", "top", "scale"))
    if int(mlp["expert"].get("ff", 0)) <= 0 or (mlp.get("shared") is not None and int(mlp["shared"].get("ff", 0)) <= 0):
        raise ConfigError(f"{where}: expert.ff and shared.ff must be positive")
    if not 0 < int(mlp["router"]["top"]) <= int(mlp["router"]["experts"]):
        raise ConfigError(f"{where}.router: top must lie between 1 and the number of experts")


@dataclass(frozen=True)
class GedelornConfig:
    vocab: int
    width: int
    layers: tuple[GedelornLayer, ...]
    norm_eps: float
    eos_token_ids: tuple = ()
    architecture: str = "Gedelorn"
    extra: dict = field(default_factory=dict, compare=False)

    # ---- reading ---------------------------------------------------------------------------------
    @classmethod
    def from_dict(cls, raw: dict, generation: dict | None = None) -> "GedelornConfig":
        for key in ("vocab", "width", "layers", "norm"):
            if key not in raw:
                raise ConfigError(f"config.json lacks {key!r}")
        if "eps" not in raw["norm"]:
            raise ConfigError("config.json lacks norm.eps")
        layers = []
        for i, entry in enumerate(raw["layers"]):
            if "type" not in entry or "mixer" not in entry:
                raise ConfigError(f"layers[{i}] needs 'type' and 'mixer'")
            mlp = entry.get("mlp")
            layers.append(GedelornLayer(str(entry["type"]), copy.deepcopy(dict(entry["mixer"])),
                                        None if mlp is None else copy.deepcopy(dict(mlp))))
        eos = (generation or {}).get("eos_token_id", raw.get("eos_token_id"))
        eos = () if eos is None else tuple(eos) if isinstance(eos, (list, tuple)) else (int(eos),)
        known = {"architecture", "architectures", "model_type", "vocab", "width", "layers", "norm", "eos_token_id"}
        cfg = cls(vocab=int(raw["vocab"]), width=int(raw["width"]), layers=tuple(layers), norm_eps=float(raw["norm"]["eps"]),
                  eos_token_ids=eos, architecture=str(raw.get("architecture") or (raw.get("architectures") or ["Gedelorn"])[0]),
                  extra={k: v for k, v in raw.items() if k not in known})
        cfg.validate()
        return cfg

    def validate(self) -> None:
        if self.vocab <= 0 or self.width <= 0 or not self.layers:
            raise ConfigError("vocab, width and the number of layers must be positive")
        if self.norm_eps < 0:
            raise ConfigError("norm.eps cannot be negative")
        for i, layer in enumerate(self.layers):
            where, m = f"layers[{i}].mixer", layer.mixer
            if layer.type not in _NEEDS:
                raise ConfigError(f"layers[{i}].type {layer.type!r} is not one of {tuple(_NEEDS)}")
            _need(where, m, _NEEDS[layer.type])
            if layer.type == "mlstm":
                _positive(where, m, ("heads", "dim", "vdim"))
                _key_size(f"{where}.dim", int(m["dim"]))
                if not float(m["gate_cap"]) > 0:
                    raise ConfigError(f"{where}.gate_cap must be positive")
            elif layer.type == "mamba2":
                _positive(where, m, ("heads", "vdim", "state", "groups", "conv", "norm_groups"))
                _key_size(f"{where}.state", int(m["state"]))
                if int(m["heads"]) % int(m["groups"]):
                    raise ConfigError(f"{where}: {m['heads']} heads are not a multiple of {m['groups']} groups")
                if (int(m["heads"]) * int(m["vdim"])) % int(m["norm_groups"]):
                    raise ConfigError(f"{where}: {m['norm_groups']} parts do not divide heads * vdim")
            else:
                _check_parallel(where, m)
            if layer.mlp is not None:
                _check_mlp(f"layers[{i}].mlp", layer.mlp)

    def to_dict(self) -> dict:
        d = dict(self.extra)
        d.update({"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
                  "layers": [{"type": l.type, "mixer": copy.deepcopy(l.mixer), "mlp": copy.deepcopy(l.mlp)} for l in self.layers]})
        if self.eos_token_ids:
            d["eos_token_id"] = list(self.eos_token_ids)
        return d
