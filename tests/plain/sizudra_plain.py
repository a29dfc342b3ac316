"""A plain, slow implementation of the Sizudra decoder, written from its equations, one function per mechanism: the oracle
of the tests.  It has no cache, no batches and no portions (a sequence is run whole), and imports nothing from the
``return_b200`` package.  The configuration is config.json as a plain dict, the weights a dict name -> tensor.

Notation.  a: a sublayer's input [T, width].  Linear maps are stored [out, in] and applied as ``a @ W.T``.  Positions start
at 0.
"""
from __future__ import annotations

import json
import math
import os
import struct

import torch

_DT = {"BF16": torch.bfloat16, "F32": torch.float32, "F16": torch.float16, "I32": torch.int32, "F64": torch.float64}


def read_safetensors(path):
    with open(path, "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        meta = json.loads(f.read(n))
        data = f.read()
    out = {}
    for name, m in meta.items():
        if name == "__metadata__":
            continue
        lo, hi = m["data_offsets"]
        out[name] = torch.frombuffer(bytearray(data[lo:hi]), dtype=_DT[m["dtype"]]).reshape(m["shape"]).clone()
    return out


def read_model(model_dir, dtype=torch.float64):
    with open(os.path.join(model_dir, "config.json")) as f:
        c = json.load(f)
    w = {k: (v.to(dtype) if v.is_floating_point() else v)
         for k, v in read_safetensors(os.path.join(model_dir, "model.safetensors")).items()}
    return c, w


# --------------------------------------------------------------------------- small pieces

def rms_norm(x, weight, eps):
    """x over the root of (its mean square plus eps), along the last axis, times a weight per element."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def relu_squared(z):
    return torch.clamp(z, min=0.0) ** 2


def pair_rows(ids, buckets, mul_prev, mul_cur):
    """For every token the row of the pair table: a hash of (previous token, token); the first token has the last row."""
    return [buckets if t == 0 else (ids[t - 1] * mul_prev + ids[t] * mul_cur) % buckets for t in range(len(ids))]


def rotate_halves(x, base, dims, first_position=0):
    """x [T, heads, n]: of every head's first ``dims`` elements, i and i + dims / 2 turn by p * base^(-2i / dims)."""
    T, half = x.shape[0], dims // 2
    f = torch.tensor([float(base) ** (-2.0 * i / dims) for i in range(half)], dtype=torch.float64)
    angle = torch.arange(first_position, first_position + T, dtype=torch.float64)[:, None] * f
    c, s = torch.cos(angle).to(x.dtype)[:, None], torch.sin(angle).to(x.dtype)[:, None]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], -1)


def visible(T, mask):
    """[T, T] bool: which keys j (columns) a query i (rows) sees.  ``mask``: None, or {size, keep_first}: the last ``size``
    keys, its own included, and the sequence's first ``keep_first`` keys."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    ok = j <= i
    if mask:
        ok = ok & ((i - j < mask["size"]) | (j < mask.get("keep_first", 0)))
    return ok


def soft_cap(s, cap):
    return cap * torch.tanh(s / cap)


def softmax_with_sink(s, ok, sink=None):
    """exp(s) over (the sum of exp(s) + exp(sink)) along the last axis, over the allowed columns.  s [H, T, T]; sink [H]
    or None."""
    s = s.masked_fill(~ok, float("-inf"))
    top = s.max(-1, keepdim=True).values
    if sink is not None:
        top = torch.maximum(top, sink[:, None, None])
    e = torch.exp(s - top)
    below = e.sum(-1, keepdim=True)
    if sink is not None:
        below = below + torch.exp(sink[:, None, None] - top)
    return e / below


def blend_values(v, first, share):
    """Values that are part their own and part those of an earlier layer."""
    return (1.0 - share) * v + share * first


# --------------------------------------------------------------------------- the mixer

def attention(w, p, m, a, eps, first_values=None):
    """Causal attention with normed and rotated queries and keys; optionally a window that keeps the first tokens, capped
    scores and a sink.  ``first_values``: the values to blend in (None: the layer takes its own).  Returns (output, values as
    projected)."""
    T = a.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms_norm((a @ w[p + "q"].T).view(T, H, d), w[p + "q.norm"], eps)
    k = rms_norm((a @ w[p + "k"].T).view(T, G, d), w[p + "k.norm"], eps)
    v = own = (a @ w[p + "v"].T).view(T, G, dv)
    rot = m.get("rot")
    if rot and rot["dims"]:
        q, k = rotate_halves(q, rot["base"], rot["dims"]), rotate_halves(k, rot["base"], rot["dims"])
    if first_values is not None:
        v = blend_values(v, first_values, w[p + "vmix"])
    s = torch.einsum("ihd,jhd->hij", q, k.repeat_interleave(H // G, dim=1)) * m["scale"]
    if m.get("softcap"):
        s = soft_cap(s, m["softcap"])
    share = softmax_with_sink(s, visible(T, m.get("mask")), w.get(p + "sink"))
    o = torch.einsum("hij,jhd->ihd", share, v.repeat_interleave(H // G, dim=1)).reshape(T, H * dv)
    return o @ w[p + "o"].T, own


# --------------------------------------------------------------------------- feed-forwards

def gated(w, p, a):
    return (gelu_tanh(a @ w[p + "gate"].T) * (a @ w[p + "up"].T)) @ w[p + "down"].T


def ungated(w, p, a):
    return relu_squared(a @ w[p + "up"].T) @ w[p + "down"].T


def experts(w, p, mlp, a):
    """Every token's ``top`` experts by router logit, weighed by the softmax over the chosen logits alone, plus a shared
    expert times the logistic of one projected number."""
    z = a @ w[p + "router"].T
    out = torch.zeros_like(a)
    for t in range(a.shape[0]):
        best = torch.topk(z[t], mlp["router"]["top"])
        for share, e in zip(torch.softmax(best.values, 0), best.indices.tolist()):
            out[t] = out[t] + share * ungated(w, f"{p}e{e}.", a[t:t + 1])[0]
    if mlp.get("shared"):
        out = out + torch.sigmoid(a @ w[p + "shared.sg"].T) * ungated(w, p + "shared.", a)
    return out


# --------------------------------------------------------------------------- the decoder

def embed(c, w, ids):
    x = w["embed"][torch.as_tensor(ids)]
    b = (c.get("embedding") or {}).get("bigram")
    if b:
        x = x + w["bigram"][torch.as_tensor(pair_rows(ids, b["buckets"], b["mul_prev"], b["mul_cur"]))]
    return x


def forward(c, w, ids, trace=None):
    """Logits [T, vocab] of every position; ``trace`` (a list) receives the residual stream after every layer."""
    eps = c["norm"]["eps"]
    x = embed(c, w, ids)
    first_values = None
    for i, layer in enumerate(c["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        y, values = attention(w, p + "mix.", m, x, eps, first_values if m.get("v_mix") else None)
        if m.get("v_mix") and first_values is None:
            first_values = values
        x = x + rms_norm(y, w[p + "norm1"], eps)
        mlp = layer.get("mlp")
        if mlp:
            y = gated(w, p + "mlp.", x) if mlp["kind"] == "dense" else experts(w, p + "mlp.", mlp, x)
            x = x + rms_norm(y, w[p + "norm2"], eps)
        if trace is not None:
            trace.append(x.clone())
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T
