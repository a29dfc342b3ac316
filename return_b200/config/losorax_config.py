"""Configuration of the Losorax decoder, read from its own config.json keys.

``vocab``, ``width``, ``norm.eps`` and ``layers``: a list of entries with ``type`` (which mixer the layer has: ``attention`` or
``general_delta``), ``mixer`` (its sizes and constants) and ``mlp`` (``{"kind": "dense", "ff": n}``, ``{"kind": "moe", "router":
{"experts", "top"}, "expert": {"ff"}}`` or null).

``attention``: ``heads, kv_heads, dim, vdim, scale, bias_max`` (the reach of the bias by distance), optionally ``conv`` (taps
of the convolution), ``q_temp`` (``coef, every``: the query temperature) and ``kv_from`` (the layer whose keys and values
this one reads; it then has no projections of its own for them).  ``general_delta``: ``heads, dim``.

Two sizes are not config keys but shapes of tensors: the rows of an attention's bias table (``l<i>.mix.rel``) and the rank
of a ``general_delta`` mixer's decay (``l<i>.mix.w1``).  ``from_model_dir`` reads them from the safetensors header and keeps
them in the mixer's entry as ``bias_rows`` and ``decay_rank``, so that the configuration alone says every size from then on
(``to_dict`` writes them, ``from_dict`` takes them back).
"""
from __future__ import annotations

import copy
import json
import os
from typing import Optional

from .model_config import ConfigError

_MIXER_KEYS = {"attention": ("heads", "kv_heads", "dim", "vdim", "scale", "bias_max"), "general_delta": ("heads", "dim")}
MIXER_TYPES = tuple(_MIXER_KEYS)
# what only a tensor's rows give: mixer type -> (key it is kept under, tensor of the mixer)
_FROM_SHAPES = {"attention": ("bias_rows", "rel"), "general_delta": ("decay_rank", "w1")}


def _need(d, keys, where: str) -> None:
    if not isinstance(d, dict):
        raise ConfigError(f"config.json: {where} must be an object")
    missing = [k for k in keys if k not in d]
    if missing:
        raise ConfigError(f"config.json: {where} lacks {missing}")


class LosoraxConfig:
    def __init__(self, raw: dict):
        self.raw = copy.deepcopy(raw)
        self.validate()

    # ------------------------------------------------------------------ reading
    @classmethod
    def from_dict(cls, raw: dict) -> "LosoraxConfig":
        return cls(raw)

    @classmethod
    def from_model_dir(cls, model_dir: str, raw: Optional[dict] = None) -> "LosoraxConfig":
        """config.json plus the sizes that only tensor shapes give."""
        if raw is None:
            with open(os.path.join(model_dir, "config.json")) as f:
                raw = json.load(f)
        raw = copy.deepcopy(raw)
        layers = raw.get("layers") or []
        wanted = [(i, *_FROM_SHAPES[layer["type"]]) for i, layer in enumerate(layers)
                  if isinstance(layer, dict) and layer.get("type") in _FROM_SHAPES and isinstance(layer.get("mixer"), dict)
                  and _FROM_SHAPES[layer["type"]][0] not in layer["mixer"]]
        if wanted:
            from ..weights.safetensors_io import ModelFiles
            files = ModelFiles(model_dir)
            try:
                for i, key, tensor in wanted:
                    name = f"l{i}.mix.{tensor}"
                    if name not in files:
                        raise ConfigError(f"{model_dir}: tensor {name} is missing; its rows give {key}")
                    layers[i]["mixer"][key] = int(files.shape(name)[0])
            finally:
                files.close()
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

    # ------------------------------------------------------------------ checking
    def validate(self) -> None:
        raw = self.raw
        _need(raw, ("vocab", "width", "norm", "layers"), "the top level")
        _need(raw["norm"], ("eps",), "norm")
        if self.vocab <= 0 or self.width <= 0 or not (self.eps > 0):
            raise ConfigError("vocab, width and norm.eps must be positive")
        if not isinstance(raw["layers"], list) or not raw["layers"]:
            raise ConfigError("layers must be a list with at least one entry")
        for i, layer in enumerate(raw["layers"]):
            where = f"layers[{i}]"
            _need(layer, ("type", "mixer"), where)
            kind = layer["type"]
            if kind not in MIXER_TYPES:
                raise ConfigError(f"{where}.type={kind!r}; known: {list(MIXER_TYPES)}")
            m = layer["mixer"]
            _need(m, _MIXER_KEYS[kind], where + ".mixer")
            if min(int(m[k]) for k in ("heads", "kv_heads", "dim", "vdim") if k in _MIXER_KEYS[kind]) <= 0:
                raise ConfigError(f"{where}.mixer: sizes must be positive")
            key = _FROM_SHAPES[kind][0]
            if key in m and int(m[key]) < (2 if kind == "attention" else 1):
                raise ConfigError(f"{where}.mixer.{key}={m[key]} is too small")
            if kind == "attention":
                self._check_attention(i, m, where + ".mixer")
            self._check_mlp(layer.get("mlp"), where + ".mlp")

    def _check_attention(self, i: int, m: dict, where: str) -> None:
        if int(m["heads"]) % int(m["kv_heads"]):
            raise ConfigError(f"{where}: heads={m['heads']} is not a multiple of kv_heads={m['kv_heads']}")
        if not float(m["bias_max"]) > int(m.get("bias_rows", 0)) // 2:
            raise ConfigError(f"{where}.bias_max={m['bias_max']}: beyond half of the bias table's {m.get('bias_rows')} rows")
        if m.get("conv") is not None and not (0 <= int(m["conv"]) <= 33):
            raise ConfigError(f"{where}.conv={m['conv']}: up to 33 taps")
        if m.get("q_temp") is not None:
            _need(m["q_temp"], ("coef", "every"), where + ".q_temp")
            every = m["q_temp"]["every"]
            if float(every) != int(every) or int(every) < 1:
                raise ConfigError(f"{where}.q_temp.every={every} must be a positive whole number")
        src = m.get("kv_from")
        if src is not None:
            src, layers = int(src), self.raw["layers"]
            if not (0 <= src < i) or layers[src]["type"] != "attention" or layers[src]["mixer"].get("kv_from") is not None:
                raise ConfigError(f"{where}.kv_from={src}: an earlier attention layer with keys of its own")
            if any(int(layers[src]["mixer"][k]) != int(m[k]) for k in ("kv_heads", "dim", "vdim")):
                raise ConfigError(f"{where}: kv_heads, dim and vdim must equal those of layer {src}")

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
        else:
            raise ConfigError(f"{where}.kind={mlp['kind']!r}; known: dense, moe")

    # ------------------------------------------------------------------ writing
    def to_dict(self) -> dict:
        d = copy.deepcopy(self.raw)
        d.setdefault("architecture", "Losorax")
        return d
