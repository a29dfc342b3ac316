"""The Sizudra decoder as a ``DecoderSpec`` plus the map from its checkpoint tensor names to the parts' parameters.

An embedding plus a row of a table of token pairs; layers whose sublayers read the residual stream itself and are normed on
their output only; grouped-query attention with normed, partly rotated queries and keys and values that are blended with
those of the first such layer, in two forms: over all earlier keys, or over a window that keeps the sequence's first keys
in sight, with softly capped scores and a sink.  Feed-forwards are units gated by the tanh form of gelu, or mixtures of
experts without a gate (relu squared) beside a shared one behind a gate per token.  A final norm and an untied head.

Tensor names: ``embed``, ``bigram``, ``final.norm``, ``head``; ``l<i>.{norm1, norm2}``; ``l<i>.mix.{q, k, v, o, q.norm, k.norm,
vmix, sink}``; ``l<i>.mlp.{gate, up, down}`` or ``l<i>.mlp.{router, e<j>.{up, down}, shared.{up, down, sg}}``.
"""
from __future__ import annotations

from typing import Dict, Optional, Tuple

from ..config.sizudra_config import SizudraConfig
from ..parts.spec import (AttentionSpec, DecoderSpec, DenseMLPSpec, MoESpec, NormSpec, PostNormBlockSpec, ScaledRopeSpec,
                          SwiGLUSpec)
from ..weights.loader import Source

EXPERT_ACTIVATION = "relu2"
DENSE_ACTIVATION = "gelu_tanh"


def _padded_head(m: dict) -> int:
    return (max(int(m["dim"]), int(m["vdim"])) + 15) // 16 * 16


def _value_mix(cfg: SizudraConfig, i: int) -> Optional[str]:
    if not cfg.layers[i]["mixer"].get("v_mix"):
        return None
    if i != cfg.value_source():
        return "blend"
    return "source" if any(layer["mixer"].get("v_mix") for layer in cfg.layers[i + 1:]) else None


def _mixer_spec(cfg: SizudraConfig, i: int, max_positions: int) -> AttentionSpec:
    layer = cfg.layers[i]
    m, rot, mask, cap = layer["mixer"], layer["mixer"].get("rot"), layer["mixer"].get("mask"), layer["mixer"].get("softcap")
    position = (ScaledRopeSpec(rotary_dim=int(rot["dims"]), theta=float(rot["base"]), max_positions=max_positions)
                if rot and int(rot["dims"]) else None)
    return AttentionSpec(hidden_size=cfg.width, num_heads=int(m["heads"]), num_kv_heads=int(m["kv_heads"]), head_dim=_padded_head(m),
                         scale=float(m["scale"]), window=int(mask["size"]) if mask else None,
                         qk_norm=NormSpec(size=int(m["dim"]), eps=cfg.eps), position=position, key_dim=int(m["dim"]),
                         value_dim=int(m["vdim"]), keep_first=int(mask.get("keep_first") or 0) if mask else 0,
                         softcap=float(cap) if cap else None, sink=layer["type"] == "attention_2", value_mix=_value_mix(cfg, i))


def _mlp_spec(mlp: Optional[dict], width: int):
    if not mlp:
        return None
    if mlp["kind"] == "dense":
        ff = int(mlp["ff"])
        return SwiGLUSpec(hidden_size=width, intermediate_size=ff, interleave=_interleave(ff), activation=DENSE_ACTIVATION)
    r, shared = mlp["router"], mlp.get("shared")

    def unit(sizes):
        return DenseMLPSpec(hidden_size=width, intermediate_size=int(sizes["ff"]), activation=EXPERT_ACTIVATION)
    return MoESpec(hidden_size=width, num_experts=int(r["experts"]), top=int(r["top"]), expert=unit(mlp["expert"]),
                   shared=unit(shared) if shared else None, renorm_tiny=0.0, shared_gate=bool(shared))


def _interleave(ff: int) -> int:
    return 8 if ff % 8 == 0 else 0


def decoder_spec(cfg: SizudraConfig, max_positions: Optional[int] = None) -> DecoderSpec:
    norm = NormSpec(size=cfg.width, eps=cfg.eps)
    blocks = []
    for i, layer in enumerate(cfg.layers):
        ff = _mlp_spec(layer.get("mlp"), cfg.width)
        blocks.append(PostNormBlockSpec(mixer=_mixer_spec(cfg, i, max_positions or 4096), feed_forward=ff, mixer_post_norm=norm,
                                        feed_forward_post_norm=norm if ff is not None else None))
    return DecoderSpec(vocab_size=cfg.vocab, hidden_size=cfg.width, layers=tuple(blocks), schedule=DecoderSpec.in_order(len(blocks)),
                       final_norm=norm, tie_embeddings=False, embedding_pairs=cfg.bigram)


def weight_sources(cfg: SizudraConfig) -> Dict[str, Source]:
    m: Dict[str, Source] = {"embed": Source(("embed",)), "final_norm.weight": Source(("final.norm",)), "lm_head": Source(("head",))}
    if cfg.bigram is not None:
        m["embed_pairs"] = Source(("bigram",))
    for i, layer in enumerate(cfg.layers):
        src, dst, mm = f"l{i}.", f"layers.{i}.", layer["mixer"]
        mix, out = src + "mix.", dst + "mixer."
        D, dim, vdim = _padded_head(mm), int(mm["dim"]), int(mm["vdim"])
        m[dst + "mixer_post_norm.weight"] = Source((src + "norm1",))
        m[out + "qkv"] = Source((mix + "q", mix + "k", mix + "v"), pad_rows=((dim, D), (dim, D), (vdim, D)))
        m[out + "q_norm.weight"] = Source((mix + "q.norm",), pad_rows=((dim, D),))
        m[out + "k_norm.weight"] = Source((mix + "k.norm",), pad_rows=((dim, D),))
        m[out + "o"] = Source((mix + "o",), pad_cols=(vdim, D))
        if layer["type"] == "attention_2":
            m[out + "sink"] = Source((mix + "sink",))
        if _value_mix(cfg, i) == "blend":
            m[out + "value_share"] = Source((mix + "vmix",))
        mlp = layer.get("mlp")
        if not mlp:
            continue
        p, ff = src + "mlp.", dst + "feed_forward."
        m[dst + "feed_forward_post_norm.weight"] = Source((src + "norm2",))
        if mlp["kind"] == "dense":
            m[ff + "gate_up"] = Source((p + "gate", p + "up"), interleave=_interleave(int(mlp["ff"])))
            m[ff + "down"] = Source((p + "down",))
            continue
        E = int(mlp["router"]["experts"])
        m[ff + "router"] = Source((p + "router",) + ((p + "shared.sg",) if mlp.get("shared") else ()))
        m[ff + "experts.up"] = Source(tuple(f"{p}e{j}.up" for j in range(E)))
        m[ff + "experts.down"] = Source(tuple(f"{p}e{j}.down" for j in range(E)))
        if mlp.get("shared"):
            m[ff + "shared.up"] = Source((p + "shared.up",))
            m[ff + "shared.down"] = Source((p + "shared.down",))
    return m


def checkpoint_shapes(cfg: SizudraConfig) -> Dict[str, Tuple[Tuple[int, ...], str]]:
    """Every tensor of a checkpoint: name -> (shape, law of its random values).  Matrices are drawn with a deviation of
    fan_in^-1/2 (twice that for the routers: choices that are not close calls), norm weights around one, the sinks and the
    shares of the blended values so that they matter."""
    W, V = cfg.width, cfg.vocab
    out: Dict[str, Tuple[Tuple[int, ...], str]] = {"embed": ((V, W), "normal:1.0"), "final.norm": ((W,), "ones_normal"),
                                                   "head": ((V, W), "fan_in")}
    if cfg.bigram is not None:
        out["bigram"] = ((cfg.bigram[0] + 1, W), "normal:0.5")
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}.", layer["mixer"]
        x, H, G, D, Vd = p + "mix.", int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
        out[p + "norm1"] = ((W,), "ones_normal")
        out[x + "q"] = ((H * D, W), "fan_in")
        out[x + "k"] = ((G * D, W), "fan_in")
        out[x + "v"] = ((G * Vd, W), "fan_in")
        out[x + "q.norm"] = ((D,), "ones_normal")
        out[x + "k.norm"] = ((D,), "ones_normal")
        out[x + "o"] = ((W, H * Vd), "fan_in")
        if layer["type"] == "attention_2":
            out[x + "sink"] = ((H,), "normal:1.0")
        if _value_mix(cfg, i) == "blend":
            out[x + "vmix"] = ((), "uniform01")
        mlp = layer.get("mlp")
        if not mlp:
            continue
        z = p + "mlp."
        out[p + "norm2"] = ((W,), "ones_normal")
        if mlp["kind"] == "dense":
            ff = int(mlp["ff"])
            out[z + "gate"] = ((ff, W), "fan_in")
            out[z + "up"] = ((ff, W), "fan_in")
            out[z + "down"] = ((W, ff), "fan_in")
            continue
        E, F = int(mlp["router"]["experts"]), int(mlp["expert"]["ff"])
        out[z + "router"] = ((E, W), "fan_in:2")
        for j in range(E):
            out[f"{z}e{j}.up"] = ((F, W), "fan_in")
            out[f"{z}e{j}.down"] = ((W, F), "fan_in")
        if mlp.get("shared"):
            S = int(mlp["shared"]["ff"])
            out[z + "shared.up"] = ((S, W), "fan_in")
            out[z + "shared.down"] = ((W, S), "fan_in")
            out[z + "shared.sg"] = ((1, W), "fan_in")
    return out


def ignorable_tensors(cfg: SizudraConfig):
    """What a file may hold although nothing reads it: the share of a layer that blends no values in (the first of those that
    could), and the second norm of a layer without a feed-forward."""
    return ({f"l{i}.mix.vmix" for i in range(len(cfg.layers)) if _value_mix(cfg, i) != "blend"}
            | {f"l{i}.norm2" for i, layer in enumerate(cfg.layers) if not layer.get("mlp")})
