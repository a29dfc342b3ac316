"""The Losorax decoder as a ``DecoderSpec`` plus the map from its checkpoint tensor names to the parts' parameters.

Layers normed before and after each sublayer by an elementwise squash, tanh(alpha x) * w + b, with a learned scale on each
sublayer's output and a blend of what the mixer reads with the row before.  A layer's mixer is a causal attention (q, k, v
convolved over time, q and k heads normed, a query temperature, a learned bias by distance, one added to the softmax's
denominator; optionally on the keys and values of an earlier layer) or a general delta rule.  Feed-forwards are gated
units or mixtures of experts with logistic scores that weigh the experts' inputs.  An untied head.

Tensor names: ``embed``, ``final.norm``, ``head``; ``l<i>.{norm1, norm1b, norm2, norm2b}``, every norm with ``.alpha`` and ``.b``;
``l<i>.{shift, ls1, ls2}``; ``l<i>.mix.{q, k, v, o, rel, q.conv, k.conv, v.conv}`` (attention; no k, v with ``kv_from``) or
``l<i>.mix.{r, k, v, g, a, a.b, w1, w2, w0, norm, o}``; ``l<i>.mlp.{gate, up, down}`` or ``l<i>.mlp.{router, e<j>.{gate, up,
down}}``.
"""
from __future__ import annotations

import math
from typing import Dict, Optional, Tuple

from ..config.losorax_config import LosoraxConfig
from ..config.model_config import ConfigError
from ..parts.spec import (DecoderSpec, GatedAttentionSpec, GeneralDeltaSpec, MoESpec, SandwichBlockSpec, ScheduleEntry,
                          SwiGLUSpec, TanhNormSpec)
from ..weights.loader import Source

DECAY_SCALE = math.exp(-0.5)      # w = exp(-e^(-1/2) sigmoid(.)) in the general delta rule
UNIT_EPS = 1e-6                   # under the root of its unit keys
SINK_SCORE = 0.0                  # one is added to the softmax's denominator: exp(0)


def _size_from_shape(i: int, m: dict, key: str) -> int:
    if key not in m:
        raise ConfigError(f"layers[{i}].mixer: {key} is not known; it is a shape of the checkpoint: read the configuration with "
                          f"LosoraxConfig.from_model_dir, or give {key} in the mixer's entry")
    return int(m[key])


def _mixer_spec(cfg: LosoraxConfig, i: int):
    layer = cfg.layers[i]
    m, W, eps = layer["mixer"], cfg.width, cfg.eps
    if layer["type"] == "general_delta":
        return GeneralDeltaSpec(hidden_size=W, num_heads=int(m["heads"]), key_dim=int(m["dim"]),
                                decay_rank=_size_from_shape(i, m, "decay_rank"), eps=eps, decay_scale=DECAY_SCALE, unit_eps=UNIT_EPS)
    t = m.get("q_temp")
    return GatedAttentionSpec(hidden_size=W, num_heads=int(m["heads"]), num_kv_heads=int(m["kv_heads"]), key_dim=int(m["dim"]),
                              value_dim=int(m["vdim"]), scale=float(m["scale"]), own_cache=m.get("kv_from") is None,
                              conv_taps=int(m.get("conv") or 0) or None, head_norm_eps=eps,
                              temperature=(float(t["coef"]), int(t["every"])) if t else None,
                              distance_bias=(_size_from_shape(i, m, "bias_rows"), float(m["bias_max"])), fixed_sink=SINK_SCORE)


def _mlp_spec(mlp: Optional[dict], width: int):
    if not mlp:
        return None
    if mlp["kind"] == "dense":
        ff = int(mlp["ff"])
        return SwiGLUSpec(hidden_size=width, intermediate_size=ff, interleave=_interleave(ff))
    r = mlp["router"]
    return MoESpec(hidden_size=width, num_experts=int(r["experts"]), top=int(r["top"]),
                   expert=SwiGLUSpec(hidden_size=width, intermediate_size=int(mlp["expert"]["ff"]), interleave=0),
                   score="sigmoid", renormalize=False, weigh_input=True)


def _interleave(ff: int) -> int:
    return 8 if ff % 8 == 0 else 0


def decoder_spec(cfg: LosoraxConfig, max_positions: Optional[int] = None) -> DecoderSpec:
    norm = TanhNormSpec(size=cfg.width)
    blocks, schedule = [], []
    for i, layer in enumerate(cfg.layers):
        ff = _mlp_spec(layer.get("mlp"), cfg.width)
        blocks.append(SandwichBlockSpec(mixer=_mixer_spec(cfg, i), feed_forward=ff, mixer_norm=norm, mixer_post_norm=norm,
                                        feed_forward_norm=norm if ff is not None else None,
                                        feed_forward_post_norm=norm if ff is not None else None, layer_scale=True, token_shift=True))
        src = layer["mixer"].get("kv_from") if layer["type"] == "attention" else None
        schedule.append(ScheduleEntry(i, cache_of=int(src) if src is not None else None))
    return DecoderSpec(vocab_size=cfg.vocab, hidden_size=cfg.width, layers=tuple(blocks), schedule=tuple(schedule),
                       final_norm=norm, tie_embeddings=False)


def _norm_sources(ours: str, theirs: str) -> Dict[str, Source]:
    return {ours + ".weight": Source((theirs,)), ours + ".bias": Source((theirs + ".b",)), ours + ".alpha": Source((theirs + ".alpha",))}


def weight_sources(cfg: LosoraxConfig) -> Dict[str, Source]:
    m: Dict[str, Source] = {"embed": Source(("embed",)), "lm_head": Source(("head",)), **_norm_sources("final_norm", "final.norm")}
    for i, layer in enumerate(cfg.layers):
        src, dst, mm = f"l{i}.", f"layers.{i}.", layer["mixer"]
        mix, out = src + "mix.", dst + "mixer."
        m.update(_norm_sources(dst + "mixer_norm", src + "norm1"))
        m.update(_norm_sources(dst + "mixer_post_norm", src + "norm1b"))
        m[dst + "shift"] = Source((src + "shift",))
        m[dst + "mixer_scale"] = Source((src + "ls1",))
        if layer["type"] == "attention":
            names = ("q", "k", "v") if mm.get("kv_from") is None else ("q",)
            padded = (max(int(mm["dim"]), int(mm["vdim"])) + 15) // 16 * 16
            m[out + "in"] = Source(tuple(mix + n for n in names))
            if mm.get("conv"):
                m[out + "conv"] = Source(tuple(mix + n + ".conv" for n in names))
            m[out + "rel"] = Source((mix + "rel",))
            m[out + "o"] = Source((mix + "o",), pad_cols=(int(mm["vdim"]), padded))
        else:
            m[out + "in"] = Source(tuple(mix + n for n in ("r", "k", "v", "g", "a", "w1")))
            for ours, theirs in (("decay_up", "w2"), ("decay_bias", "w0"), ("rate_bias", "a.b"), ("norm", "norm"), ("o", "o")):
                m[out + ours] = Source((mix + theirs,))
        mlp = layer.get("mlp")
        if mlp:
            p, ff = src + "mlp.", dst + "feed_forward."
            m.update(_norm_sources(dst + "feed_forward_norm", src + "norm2"))
            m.update(_norm_sources(dst + "feed_forward_post_norm", src + "norm2b"))
            m[dst + "feed_forward_scale"] = Source((src + "ls2",))
            if mlp["kind"] == "dense":
                m[ff + "gate_up"] = Source((p + "gate", p + "up"), interleave=_interleave(int(mlp["ff"])))
                m[ff + "down"] = Source((p + "down",))
            else:
                E = int(mlp["router"]["experts"])
                m[ff + "router"] = Source((p + "router",))
                m[ff + "experts.gate_up"] = Source(tuple(f"{p}e{j}.{n}" for j in range(E) for n in ("gate", "up")))
                m[ff + "experts.down"] = Source(tuple(f"{p}e{j}.down" for j in range(E)))
    return m


def checkpoint_shapes(cfg: LosoraxConfig) -> Dict[str, Tuple[Tuple[int, ...], str]]:
    """Every tensor of a checkpoint: name -> (shape, law of its random values).  Matrices are drawn with a deviation of
    fan_in^-1/2 (three times that for the routers: logistic scores far apart without running into one), the vectors so that
    squashes, gates and decays are neither shut nor saturated."""
    W, V = cfg.width, cfg.vocab
    out: Dict[str, Tuple[Tuple[int, ...], str]] = {"embed": ((V, W), "normal:1.0"), "head": ((V, W), "fan_in")}

    def norm(name: str) -> None:
        out[name] = ((W,), "ones_normal")
        out[name + ".b"] = ((W,), "normal:0.2")
        out[name + ".alpha"] = ((), "half_to_one")

    norm("final.norm")
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}.", layer["mixer"]
        x = p + "mix."
        norm(p + "norm1")
        norm(p + "norm1b")
        out[p + "shift"] = ((W,), "uniform01")
        out[p + "ls1"] = ((W,), "half_to_one")
        if layer["type"] == "attention":
            H, G, D, Vd, K = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), int(m.get("conv") or 0)
            rows = {"q": H * D} if m.get("kv_from") is not None else {"q": H * D, "k": G * D, "v": G * Vd}
            for n, r in rows.items():
                out[x + n] = ((r, W), "fan_in")
                if K:
                    out[x + n + ".conv"] = ((r, K), "normal:0.5")
            out[x + "rel"] = ((_size_from_shape(i, m, "bias_rows"), H), "normal:1.0")
            out[x + "o"] = ((W, H * Vd), "fan_in")
        else:
            HD, R = int(m["heads"]) * int(m["dim"]), _size_from_shape(i, m, "decay_rank")
            for n in ("r", "k", "v", "g", "a"):
                out[x + n] = ((HD, W), "fan_in")
            out[x + "a.b"] = ((HD,), "normal:0.5")
            out[x + "w1"] = ((R, W), "fan_in")
            out[x + "w2"] = ((HD, R), "fan_in")
            out[x + "w0"] = ((HD,), "normal:0.5")
            out[x + "norm"] = ((HD,), "ones_normal")
            out[x + "o"] = ((W, HD), "fan_in")
        mlp = layer.get("mlp")
        if mlp:
            z = p + "mlp."
            norm(p + "norm2")
            norm(p + "norm2b")
            out[p + "ls2"] = ((W,), "half_to_one")
            if mlp["kind"] == "dense":
                ff = int(mlp["ff"])
                out[z + "gate"], out[z + "up"], out[z + "down"] = ((ff, W), "fan_in"), ((ff, W), "fan_in"), ((W, ff), "fan_in")
            else:
                E, F = int(mlp["router"]["experts"]), int(mlp["expert"]["ff"])
                out[z + "router"] = ((E, W), "fan_in:3")
                for j in range(E):
                    out[f"{z}e{j}.gate"], out[f"{z}e{j}.up"] = ((F, W), "fan_in"), ((F, W), "fan_in")
                    out[f"{z}e{j}.down"] = ((W, F), "fan_in")
    return out


def ignorable_tensors(cfg: LosoraxConfig):
    """A layer without a feed-forward never reads the second pair of norms and scale; a file may hold them all the same."""
    return {f"l{i}.{n}" for i, layer in enumerate(cfg.layers) if not layer.get("mlp")
            for n in ("norm2", "norm2.b", "norm2.alpha", "norm2b", "norm2b.b", "norm2b.alpha", "ls2")}
