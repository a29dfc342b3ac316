"""Configuration of the Sizudra decoder, read from its own config.json keys.

``vocab``, ``width``, ``norm.eps``, optionally ``embedding.bigram`` (``buckets, mul_prev, mul_cur``: a table of token pairs is
added to the embedded token) and ``layers``: a list of entries with ``type`` (``attention``, or ``attention_2``: the form with a
sink), ``mixer`` (its sizes and constants) and ``mlp`` (``{"kind": "dense", "ff": n}``, ``{"kind": "moe", "router": {"experts",
"top"}, "expert": {"ff"}, "shared": {"ff"}}``, ``shared`` optional, or null).

A mixer: ``heads, kv_heads, dim, vdim, scale``, optionally ``rot`` (``base, dims``), ``mask`` (``size``: the last n keys;
``keep_first``: the sequence's first keys beside them), ``softcap`` (of the scaled scores) and ``v_mix`` (the values are
blended with those of the first layer that says so).
"""
from __future__ import annotations

import copy
from typing import Optional, Tuple

from .model_config import ConfigError

MIXER_TYPES = ("attention", "attention_2")
_MIXER_KEYS = ("heads", "kv_heads", "dim", "vdim", "scale")


def _need(d, keys, where: str) -> None:
    if not isinstance(d, dict):
        raise ConfigError(f"config.json: {where} must be an object")
    missing = [k for k in keys if k not in d]
    if missing:
        raise ConfigError(f"config.json: {where} lacks {missing}")


class SizudraConfig:
    def __init__(self, raw: dict):
        self.raw = copy.deepcopy(raw)
        self.validate()

    @classmethod
    def from_dict(cls, raw: dict) -> "SizudraConfig":
        return cls(raw)

    # ------------------------------------------------------------------ what it holds
    @property
    def vocab(self) -> int:
        return int(self.raw["vocab"])

    vocab_size = vocab

    @property
    def width(self) -> int:
        return int(self.raw["width"])

    @property
    def eps(self) -> float:
        return float(self.raw["norm"]["eps"])

    @property
    def layers(self):
        return self.raw["layers"]

    @property
    def bigram(self) -> Optional[Tuple[int, int, int]]:
        b = (self.raw.get("embedding") or {}).get("bigram")
        return (int(b["buckets"]), int(b["mul_prev"]), int(b["mul_cur"])) if b else None

    def value_source(self) -> Optional[int]:
        """The first layer whose values later layers blend in, or None."""
        return next((i for i, layer in enumerate(self.layers) if layer["mixer"].get("v_mix")), None)

    # ------------------------------------------------------------------ checking
    def validate(self) -> None:
        raw = self.raw
        _need(raw, ("vocab", "width", "norm", "layers"), "the top level")
        _need(raw["norm"], ("eps",), "norm")
        if self.vocab <= 0 or self.width <= 0 or not (self.eps > 0):
            raise ConfigError("vocab, width and norm.eps must be positive")
        b = (raw.get("embedding") or {}).get("bigram")
        if b is not None:
            _need(b, ("buckets", "mul_prev", "mul_cur"), "embedding.bigram")
            if int(b["buckets"]) <= 0 or int(b["mul_prev"]) < 0 or int(b["mul_cur"]) < 0:
                raise ConfigError("embedding.bigram: buckets must be positive, the factors not negative")
        if not isinstance(raw["layers"], list) or not raw["layers"]:
            raise ConfigError("layers must be a list with at least one entry")
        for i, layer in enumerate(raw["layers"]):
            where = f"layers[{i}]"
            _need(layer, ("type", "mixer"), where)
            if layer["type"] not in MIXER_TYPES:
                raise ConfigError(f"{where}.type={layer['type']!r}; known: {list(MIXER_TYPES)}")
            self._check_mixer(layer["mixer"], where + ".mixer")
            self._check_mlp(layer.get("mlp"), where + ".mlp")
        src = self.value_source()
        for i, layer in enumerate(raw["layers"]):
            if layer["mixer"].get("v_mix") and any(int(layer["mixer"][k]) != int(raw["layers"][src]["mixer"][k]) for k in ("kv_heads", "vdim")):
                raise ConfigError(f"layers[{i}].mixer: kv_heads and vdim must equal those of layer {src}, whose values it blends in")

    @staticmethod
    def _check_mixer(m: dict, where: str) -> None:
        _need(m, _MIXER_KEYS, where)
        if min(int(m[k]) for k in ("heads", "kv_heads", "dim", "vdim")) <= 0 or not float(m["scale"]) > 0:
            raise ConfigError(f"{where}: sizes and scale must be positive")
        if int(m["heads"]) % int(m["kv_heads"]):
            raise ConfigError(f"{where}: heads={m['heads']} is not a multiple of kv_heads={m['kv_heads']}")
        rot = m.get("rot")
        if rot is not None:
            _need(rot, ("base", "dims"), where + ".rot")
            if int(rot["dims"]) % 2 or not (0 <= int(rot["dims"]) <= int(m["dim"])) or not float(rot["base"]) > 0:
                raise ConfigError(f"{where}.rot: dims={rot['dims']} must be even and at most dim, base positive")
        mask = m.get("mask")
        if mask is not None:
            _need(mask, ("size",), where + ".mask")
            if int(mask["size"]) <= 0 or int(mask.get("keep_first") or 0) < 0:
                raise ConfigError(f"{where}.mask: size must be positive, keep_first not negative")
        if m.get("softcap") is not None and not float(m["softcap"]) > 0:
            raise ConfigError(f"{where}.softcap must be positive")

    @staticmethod
    def _check_mlp(mlp: Optional[dict], where: str) -> None:
        if mlp is None:
            return
        _need(mlp, ("kind",), where)
        if mlp["kind"] == "dense":
            _need(mlp, ("ff",), where)
            if int(mlp["ff"]) <= 0:
                raise ConfigError(f"{where}.ff must be positive")
        elif mlp["kind"] == "moe":
            _need(mlp, ("router", "expert"), where)
            _need(mlp["router"], ("experts", "top"), where + ".router")
            _need(mlp["expert"], ("ff",), where + ".expert")
            if not (1 <= int(mlp["router"]["top"]) <= int(mlp["router"]["experts"])) or int(mlp["expert"]["ff"]) <= 0:
                raise ConfigError(f"{where}.router: top={mlp['router']['top']} of {mlp['router']['experts']} experts, ff={mlp['expert']['ff']}")
            if mlp.get("shared"):
                _need(mlp["shared"], ("ff",), where + ".shared")
                if int(mlp["shared"]["ff"]) <= 0:
                    raise ConfigError(f"{where}.shared.ff must be positive")
        else:
            raise ConfigError(f"{where}.kind={mlp['kind']!r}; known: dense, moe")

    # ------------------------------------------------------------------ writing
    def to_dict(self) -> dict:
        d = copy.deepcopy(self.raw)
        d.setdefault("architecture", "Sizudra")
        return d
