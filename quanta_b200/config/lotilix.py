"""Typed configuration of the Lotilix decoder, from config.json.

The file is nested: ``vocab``, ``width``, ``norm.eps``, ``token_side.dim`` (numbers per layer of the token's own input)
and ``layers``, a list in run order whose entries give the layer's ``type``, the mixer's sizes and constants (``mixer``)
and its feed-forward (``mlp``; null for a layer with a mixer only).

* ``latent_attention``: ``heads``, ``dim`` / ``rot_dim`` (plain and rotated query/key sizes), ``vdim``, ``q_rank``,
  ``kv_rank``, ``scale``, ``mask.size`` (the window) and ``rot.base``.
* ``channel_delta``: ``heads``, ``kv_heads`` (groups of q/k heads), ``dim``, ``vdim``, ``conv`` (taps).  The inner ranks
  of the decay and of the output gate are the checkpoint's tensor shapes (``with_tensor_shapes``; ``decay_rank`` and
  ``gate_rank`` in ``mixer`` for a model that is drawn at random).
* ``attention``: ``heads``, ``kv_heads``, ``dim``, ``scale``, ``mask.size`` (the chunk), ``rot.dims`` / ``rot.base`` and
  ``rot.scaling`` (``factor``, ``low``, ``high``, ``original``).  The values are the keys, so ``vdim`` equals ``dim``.
* ``mlp.kind`` ``dense``: ``ff``.

Every size and constant the layers use is read here; what the layers cannot run is refused.
"""

from __future__ import annotations

import copy
from dataclasses import dataclass, field, replace

from .minimax_m3 import ConfigError

MAX_HEAD_SIZE = 256
MAX_LATENT = 512
DEFAULT_INNER_RANK = 16        # of decay and gate when no checkpoint says otherwise (random models)
_NEEDS = {
    "latent_attention": ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank", "scale", "mask", "rot"),
    "channel_delta": ("heads", "kv_heads", "dim", "vdim", "conv"),
    "attention": ("heads", "kv_heads", "dim", "scale", "mask"),
}


@dataclass(frozen=True)
class LotilixLayer:
    type: str
    mixer: dict
    mlp: dict | None


def _check_rotation(where: str, rot: dict, most: int) -> None:
    dims = int(rot.get("dims") or 0)
    if dims < 0 or dims % 2 or dims > most or (dims and float(rot.get("base", 0)) <= 0):
        raise ConfigError(f"{where}: dims must be even and at most {most}, base positive")
    sc = rot.get("scaling")
    if sc is not None:
        missing = [k for k in ("factor", "low", "high", "original") if k not in sc]
        if missing:
            raise ConfigError(f"{where}.scaling lacks {missing}")
        if float(sc["factor"]) <= 0 or float(sc["original"]) <= 0 or not 0 < float(sc["low"]) < float(sc["high"]):
            raise ConfigError(f"{where}.scaling: needs factor, original > 0 and 0 < low < high")


@dataclass(frozen=True)
class LotilixConfig:
    vocab: int
    width: int
    layers: tuple[LotilixLayer, ...]
    norm_eps: float
    side_dim: int
    eos_token_ids: tuple = ()
    architecture: str = "Lotilix"
    extra: dict = field(default_factory=dict, compare=False)

    # ---- reading ---------------------------------------------------------------------------------
    @classmethod
    def from_dict(cls, raw: dict, generation: dict | None = None) -> "LotilixConfig":
        for key in ("vocab", "width", "layers", "norm", "token_side"):
            if key not in raw:
                raise ConfigError(f"config.json lacks {key!r}")
        if "eps" not in raw["norm"] or "dim" not in raw["token_side"]:
            raise ConfigError("config.json lacks norm.eps or token_side.dim")
        layers = []
        for i, entry in enumerate(raw["layers"]):
            if "type" not in entry or "mixer" not in entry:
                raise ConfigError(f"layers[{i}] needs 'type' and 'mixer'")
            mlp = entry.get("mlp")
            layers.append(LotilixLayer(str(entry["type"]), copy.deepcopy(dict(entry["mixer"])),
                                       None if mlp is None else copy.deepcopy(dict(mlp))))
        eos = (generation or {}).get("eos_token_id", raw.get("eos_token_id"))
        eos = () if eos is None else tuple(eos) if isinstance(eos, (list, tuple)) else (int(eos),)
        known = {"architecture", "architectures", "model_type", "vocab", "width", "layers", "norm", "token_side",
                 "eos_token_id"}
        cfg = cls(vocab=int(raw["vocab"]), width=int(raw["width"]), layers=tuple(layers),
                  norm_eps=float(raw["norm"]["eps"]), side_dim=int(raw["token_side"]["dim"]), eos_token_ids=eos,
                  architecture=str(raw.get("architecture") or (raw.get("architectures") or ["Lotilix"])[0]),
                  extra={k: v for k, v in raw.items() if k not in known})
        cfg.validate()
        return cfg

    def validate(self) -> None:
        if self.vocab <= 0 or self.width <= 0 or self.side_dim <= 0 or not self.layers:
            raise ConfigError("vocab, width, token_side.dim and the number of layers must be positive")
        if self.norm_eps < 0:
            raise ConfigError("norm.eps cannot be negative")
        for i, layer in enumerate(self.layers):
            where, m = f"layers[{i}].mixer", layer.mixer
            if layer.type not in _NEEDS:
                raise ConfigError(f"layers[{i}].type {layer.type!r} is not one of {tuple(_NEEDS)}")
            missing = [k for k in _NEEDS[layer.type] if k not in m]
            if missing:
                raise ConfigError(f"{where} lacks {missing}")
            if int(m["heads"]) <= 0 or int(m["dim"]) <= 0:
                raise ConfigError(f"{where}: heads and dim must be positive")
            if "mask" in _NEEDS[layer.type] and int(m["mask"].get("size", 0)) < 1:
                raise ConfigError(f"{where}.mask.size must hold at least the token itself")
            if layer.type == "latent_attention":
                if min(int(m["rot_dim"]), int(m["vdim"]), int(m["q_rank"])) <= 0 or int(m["rot_dim"]) % 2:
                    raise ConfigError(f"{where}: rot_dim, vdim and q_rank must be positive, rot_dim even")
                if not 0 < int(m["kv_rank"]) <= MAX_LATENT:
                    raise ConfigError(f"{where}.kv_rank must lie between 1 and {MAX_LATENT}")
                if int(m["rot"].get("dims", m["rot_dim"])) != int(m["rot_dim"]):
                    raise ConfigError(f"{where}.rot.dims is the rotated part, rot_dim")
                _check_rotation(f"{where}.rot", dict(m["rot"], dims=m["rot_dim"]), int(m["rot_dim"]))
            else:
                if int(m["kv_heads"]) <= 0 or int(m["heads"]) % int(m["kv_heads"]):
                    raise ConfigError(f"{where}: {m['heads']} heads are not a positive multiple of {m['kv_heads']} kv heads")
                if not int(m["dim"]) <= MAX_HEAD_SIZE or not 0 < int(m.get("vdim", m["dim"])) <= MAX_HEAD_SIZE:
                    raise ConfigError(f"{where}: dim and vdim must lie between 1 and {MAX_HEAD_SIZE}")
            if layer.type == "channel_delta":
                if int(m["conv"]) < 1:
                    raise ConfigError(f"{where}.conv: the convolution has at least one tap")
                if int(m.get("decay_rank", 1)) < 1 or int(m.get("gate_rank", 1)) < 1:
                    raise ConfigError(f"{where}: the inner ranks must be positive")
            if layer.type == "attention":
                if int(m.get("vdim", m["dim"])) != int(m["dim"]):
                    raise ConfigError(f"{where}: the values are the keys, so vdim equals dim")
                if m.get("rot") is not None:
                    _check_rotation(f"{where}.rot", m["rot"], int(m["dim"]))
            if layer.mlp is not None:
                if layer.mlp.get("kind") != "dense":
                    raise ConfigError(f"layers[{i}].mlp.kind {layer.mlp.get('kind')!r} is not 'dense'")
                if int(layer.mlp.get("ff", 0)) <= 0:
                    raise ConfigError(f"layers[{i}].mlp.ff must be positive")

    def with_tensor_shapes(self, shape_of) -> "LotilixConfig":
        """Fill in the sizes that are the checkpoint's tensor shapes (``shape_of(name)`` -> shape or None)."""
        layers = []
        for i, layer in enumerate(self.layers):
            if layer.type == "channel_delta":
                m = dict(layer.mixer)
                for key, tensor in (("decay_rank", "a1"), ("gate_rank", "g1")):
                    shape = shape_of(f"l{i}.mix.{tensor}")
                    if shape is not None and len(shape) == 2:
                        m[key] = int(shape[0])
                layer = replace(layer, mixer=m)
            layers.append(layer)
        cfg = replace(self, layers=tuple(layers))
        cfg.validate()
        return cfg

    def to_dict(self) -> dict:
        d = dict(self.extra)
        d.update({
            "architecture": self.architecture, "vocab": self.vocab, "width": self.width,
            "norm": {"eps": self.norm_eps}, "token_side": {"dim": self.side_dim},
            "layers": [{"type": l.type, "mixer": copy.deepcopy(l.mixer), "mlp": copy.deepcopy(l.mlp)} for l in self.layers],
        })
        if self.eos_token_ids:
            d["eos_token_id"] = list(self.eos_token_ids)
        return d
