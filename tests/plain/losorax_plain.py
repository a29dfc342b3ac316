"""Plain, slow, whole-sequence implementation of the Losorax decoder: the oracle of its tests.

Every mechanism is one function that walks a sequence in the precision it is given (float64 by default).
No cache, no batching, no kernels; nothing is shared with the ``return_b200`` package.  The configuration is
config.json as a plain dict, the weights a dict name -> tensor.

Notation.  a: a sublayer's input [T, width].  Linear maps are stored [out, in] and applied as ``a @ W.T``.
A recurrent state M of a head is a [key rows, value columns] matrix read out as ``M.T @ q``.  Positions start at 0.
"""
from __future__ import annotations

import json
import math
import os
import struct

import torch
import torch.nn.functional as F

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

def tanh_norm(w, name, x):
    """An elementwise squash in the place of a norm: no mean, no variance."""
    return torch.tanh(w[name + ".alpha"] * x) * w[name] + w[name + ".b"]


def rms(x, eps):
    """x over the root of (its mean square plus eps), along the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def blend_with_previous(a, mu):
    """Row t becomes a[t] + (a[t - 1] - a[t]) * mu; the row before the first is zero."""
    before = torch.cat([torch.zeros_like(a[:1]), a[:-1]], 0)
    return a + (before - a) * mu


def causal_conv(z, taps):
    """z [T, C], taps [C, K] with the last column for the token itself; what lies before the sequence is zero."""
    T, C = z.shape
    K = taps.shape[1]
    padded = torch.cat([z.new_zeros(K - 1, C), z], 0)
    out = z.new_zeros(T, C)
    for j in range(K):
        out = out + padded[j:j + T] * taps[:, j]
    return out


def bucket(n, rows, reach):
    """Row of a distance table of ``rows`` rows for distance n: one row a distance up to rows / 2, then rows that cover
    ever longer spans, spaced by the logarithm, the last one from about ``reach`` on."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(reach / half) * (rows - half)))


def temperature(T, coef, every, dtype):
    """The factor on the query at each position: it grows with the logarithm of how many whole runs of ``every``
    positions lie behind it."""
    p = torch.arange(T)
    return 1.0 + coef * torch.log((torch.div(p + 1, every, rounding_mode="floor") + 1).to(torch.float64)).to(dtype)


def softmax_plus_one(s, ok):
    """exp(s) over (1 + the sum of exp(s)) along the last axis, over the allowed columns."""
    s = s.masked_fill(~ok, float("-inf"))
    top = torch.clamp(s.max(-1, keepdim=True).values, min=0.0)
    e = torch.exp(s - top)
    return e / (torch.exp(-top) + e.sum(-1, keepdim=True))


# --------------------------------------------------------------------------- mixers

def attention(w, p, m, a, eps, shared=None):
    """Causal attention with convolved, normed queries and keys, a query temperature, a learned bias by distance and
    a softmax with one added below.  ``shared``: (k, v) of the layer whose keys and values this layer reads.
    Returns (output, (k, v))."""
    T = a.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]

    def projected(name):
        z = a @ w[p + name].T
        return causal_conv(z, w[p + name + ".conv"]) if m.get("conv") else z
    q = rms(projected("q").view(T, H, d), eps)
    if shared is None:
        k = rms(projected("k").view(T, G, d), eps)
        v = projected("v").view(T, G, dv)
    else:
        k, v = shared
    t = m.get("q_temp")
    if t:
        q = q * temperature(T, t["coef"], t["every"], q.dtype)[:, None, None]
    s = torch.einsum("ihd,jhd->hij", q, k.repeat_interleave(H // G, dim=1)) * m["scale"]
    table = w[p + "rel"]                                                             # [rows, H]
    of_distance = torch.tensor([bucket(n, table.shape[0], m["bias_max"]) for n in range(T)])
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    s = s + table[of_distance[(i - j).clamp(min=0)]].permute(2, 0, 1)
    o = torch.einsum("hij,jhd->ihd", softmax_plus_one(s, j <= i), v.repeat_interleave(H // G, dim=1))
    return o.reshape(T, H * dv) @ w[p + "o"].T, (k, v)


def general_delta(w, p, m, a, eps):
    """M <- diag(w) M - (r * u) (u^T M) + k v^T with both terms on the old M; o = M^T q.  w: a decay per head and key row,
    r: a removal rate per head and key row, u: the key as a unit vector."""
    T = a.shape[0]
    H, d = m["heads"], m["dim"]
    q = (a @ w[p + "r"].T).view(T, H, d)
    k = (a @ w[p + "k"].T).view(T, H, d)
    v = (a @ w[p + "v"].T).view(T, H, d)
    decay = torch.exp(-math.exp(-0.5) * torch.sigmoid(torch.tanh(a @ w[p + "w1"].T) @ w[p + "w2"].T + w[p + "w0"])).view(T, H, d)
    rate = torch.sigmoid(a @ w[p + "a"].T + w[p + "a.b"]).view(T, H, d)
    u = k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)
    M = a.new_zeros(H, d, d)
    out = a.new_zeros(T, H, d)
    for t in range(T):
        held = torch.einsum("hi,hij->hj", u[t], M)
        M = decay[t][:, :, None] * M - (rate[t] * u[t])[:, :, None] * held[:, None, :] + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hij,hi->hj", M, q[t])
    out = rms(out, eps).reshape(T, H * d) * w[p + "norm"] * torch.sigmoid(a @ w[p + "g"].T)
    return out @ w[p + "o"].T


# --------------------------------------------------------------------------- feed-forwards

def gated_unit(w, p, a):
    return (F.silu(a @ w[p + "gate"].T) * (a @ w[p + "up"].T)) @ w[p + "down"].T


def route(z, top):
    """z [T, E] router outputs -> (chosen experts [T, top], their scores [T, top], as they are)."""
    s = torch.sigmoid(z)
    picked = s.topk(top, dim=-1).indices
    return picked, s.gather(1, picked)


def experts(w, p, mlp, a):
    picked, weight = route(a @ w[p + "router"].T, mlp["router"]["top"])
    out = torch.zeros_like(a)
    for t in range(a.shape[0]):
        for e, c in zip(picked[t].tolist(), weight[t]):
            out[t] += gated_unit(w, f"{p}e{e}.", c * a[t:t + 1])[0]
    return out


# --------------------------------------------------------------------------- the model

def mixer(c, w, i, a, kept):
    layer = c["layers"][i]
    p, m, eps = f"l{i}.mix.", layer["mixer"], c["norm"]["eps"]
    if layer["type"] == "attention":
        src = m.get("kv_from")
        y, kv = attention(w, p, m, a, eps, kept[src] if src is not None else None)
        kept[i] = kv
        return y
    if layer["type"] == "general_delta":
        return general_delta(w, p, m, a, eps)
    raise ValueError(layer["type"])


def forward(c, w, ids, trace=None):
    """ids -> logits [T, vocab].  ``trace``: a list that receives the residual stream after every layer."""
    x = w["embed"][torch.as_tensor(ids, dtype=torch.long)]
    kept = {}
    for i, layer in enumerate(c["layers"]):
        p = f"l{i}."
        a = blend_with_previous(tanh_norm(w, p + "norm1", x), w[p + "shift"])
        x = x + tanh_norm(w, p + "norm1b", mixer(c, w, i, a, kept)) * w[p + "ls1"]
        mlp = layer.get("mlp")
        if mlp:
            a = tanh_norm(w, p + "norm2", x)
            y = gated_unit(w, p + "mlp.", a) if mlp["kind"] == "dense" else experts(w, p + "mlp.", mlp, a)
            x = x + tanh_norm(w, p + "norm2b", y) * w[p + "ls2"]
        if trace is not None:
            trace.append(x.clone())
    return tanh_norm(w, "final.norm", x) @ w["head"].T
