"""Causal grouped-query attention over the paged cache (rollout/monkey_patch/qwen3.py:25-56).

Projections q, k, v as one fused product (the reference runs three, :29-31; the fused weight is
their row-wise concatenation), per-head RMSNorm of q and k before the rotation (:29-30),
rotation and cache write in one kernel (for a step of single tokens: inside the attention kernel),
attention over the block table, output projection
(:55-56).  Sizes, window, norm and position encoding come from the specification, as do the options that the reference's
model has no use for: first keys kept beside a window, capped scores, a sink, values blended with an earlier layer's.
"""
from __future__ import annotations

import math

import torch

from ..ext import ops
from .base import MIXERS, NORMS, POSITION_ENCODINGS, KVCacheNeed, Mixer, ParamSpec, Tiling


@MIXERS.register("attention")
class PagedAttention(Mixer):
    def __init__(self, spec, env):
        super().__init__(spec, env)
        if spec.num_heads % spec.num_kv_heads:
            raise ValueError(f"num_heads={spec.num_heads} is not a multiple of num_kv_heads={spec.num_kv_heads}")
        if spec.head_dim % 16 or not (16 <= spec.head_dim <= 256):
            raise ValueError(f"head_dim={spec.head_dim}: the attention kernels take multiples of 16 from 16 to 256")
        if spec.window is not None and spec.window <= 0:
            raise ValueError("window must be positive")
        if spec.keep_first < 0 or (spec.keep_first and spec.window is None):
            raise ValueError("keep_first: not negative, and only beside a window")
        if spec.softcap is not None and not spec.softcap > 0:
            raise ValueError("softcap must be positive")
        if spec.value_mix not in (None, "source", "blend"):
            raise ValueError(f"value_mix={spec.value_mix!r}; known: None, 'source', 'blend'")
        self.q_norm = NORMS.build(spec.qk_norm, env) if spec.qk_norm is not None else None
        self.k_norm = NORMS.build(spec.qk_norm, env) if spec.qk_norm is not None else None
        if spec.qk_norm is not None and (spec.qk_norm.kind != "rmsnorm" or spec.qk_norm.size != (spec.key_dim or spec.head_dim)):
            raise ValueError("the fused q/k norm is an RMSNorm over a head's elements (its key_dim, or head_dim)")
        self.position = POSITION_ENCODINGS.build(spec.position, env) if spec.position is not None else None
        self.q_size = spec.num_heads * spec.head_dim
        self.kv_size = spec.num_kv_heads * spec.head_dim
        self._sink = None

    # ------------------------------------------------------------------ parameters and cache
    def params(self):
        s = self.spec
        p = {"qkv": ParamSpec((self.q_size + 2 * self.kv_size, s.hidden_size)),
             "o": ParamSpec((s.hidden_size, self.q_size))}
        if self.q_norm is not None:           # as long as the padded heads are
            weight = ParamSpec((s.head_dim,), role="vector", init=self.q_norm.params()["weight"].init)
            p["q_norm.weight"] = p["k_norm.weight"] = weight
        if s.sink:
            p["sink"] = ParamSpec((s.num_heads,), role="vector", init="normal:0.5")
        if s.value_mix == "blend":
            p["value_share"] = ParamSpec((1,), role="vector", init="uniform01")
        return p

    def bind(self, tensors):
        self.p_qkv = tensors["qkv"]
        self.p_o = tensors["o"]
        if self.q_norm is not None:
            self.q_norm.bind({"weight": tensors["q_norm.weight"]})
            self.k_norm.bind({"weight": tensors["k_norm.weight"]})
        if self.spec.sink:
            self._sink = tensors["sink"].float().contiguous()
        if self.spec.value_mix == "blend":
            self.value_share = tensors["value_share"].float().contiguous()

    def cache_need(self):
        return KVCacheNeed(self.spec.num_kv_heads, self.spec.head_dim, self.spec.window, self.spec.keep_first)

    def batch_tilings(self):
        """The row blocks of the tensor-core kernel for prompt portions that this head size runs on."""
        if self.env.act_dtype != torch.bfloat16:
            return {}
        if self.spec.head_dim in ops.TC5_ATTENTION_HEAD_DIMS:
            return {ops.TILES_TC5: Tiling(ops.TC5_TILE_ROWS, heaviest_first=True)}
        return {ops.TILES_MMA: Tiling(ops.MMA_TILE_ROWS)}

    def graph_variant(self, n_tokens, longest_context):
        """A captured step cannot change the grid of the split-KV decode kernel: the number of key splits
        is fixed per captured graph."""
        if self.env.act_dtype != torch.bfloat16:
            return {}
        s = self.spec
        seen = ops.keys_seen(s.window, s.keep_first)
        return {ops.decode_splits_key(s.num_heads, s.num_kv_heads, seen):
                ops.decode_splits_for(n_tokens, longest_context, s.num_heads, s.num_kv_heads, seen)}

    # ------------------------------------------------------------------ one step
    @property
    def _qkv_name(self):
        """A layer whose values later layers read keeps its projections in a buffer of its own until the step is over."""
        return "attention.qkv_source" if self.spec.value_mix == "source" else "attention.qkv"

    def forward(self, x, ctx):
        T = x.shape[0]
        qkv = ctx.buffer(self._qkv_name, (T, self.q_size + 2 * self.kv_size), x.dtype, x.device)
        ops.linear(x, self.p_qkv, qkv)
        o = self.core(qkv, ctx)
        y = ctx.buffer("attention.y", (T, self.spec.hidden_size), x.dtype, x.device)
        ops.linear(o, self.p_o, y)
        return y

    # A mixer that is "product, something in the middle, product" says so, and a block may then run the two
    # products in kernels of its own choosing (fused with the norms around them).
    def in_projection(self):
        """(weight [q + 2 kv, hidden], name of the buffer its output goes to)."""
        return self.p_qkv, self._qkv_name

    def out_projection(self):
        return self.p_o

    def core(self, qkv, ctx):
        """From the projections [T, q + 2 kv] to the attention output [T, q]: per-head norm, position encoding,
        blend of the values, cache write, attention over the block table."""
        s, b, kv = self.spec, ctx.batch, ctx.kv
        blend = self._blend(qkv, b)
        norm_size = s.qk_norm.size if s.qk_norm is not None else None
        seen = ops.keys_seen(s.window, s.keep_first)
        T = qkv.shape[0]
        qw = self.q_norm.p_weight if self.q_norm is not None else None
        kw = self.k_norm.p_weight if self.k_norm is not None else None
        eps = s.qk_norm.eps if s.qk_norm is not None else 0.0
        offset = s.qk_norm.offset if s.qk_norm is not None else 0.0
        tables = self.position.rotary_tables() if self.position is not None else None
        o = ctx.buffer("attention.o", (T, self.q_size), qkv.dtype, qkv.device)
        if (tables is not None or self.position is None) and ops.decode_only(b, qkv.dtype, s.num_heads, s.num_kv_heads, seen):
            # single decoded tokens only: norm, rotation, cache write and attention are one kernel
            cos, sin, rot = tables if tables is not None else (None, None, 0)
            ops.attention_decode_fused(qkv, qw, kw, eps, offset, cos, sin, rot, kv.k, kv.v, b, kv.block_table,
                                       kv.page_size, o, s.num_heads, s.num_kv_heads, s.head_dim, s.scale, s.window,
                                       write_kv=ctx.write_cache, norm_size=norm_size, blend=blend, sink=self._sink,
                                       softcap=s.softcap, keep=s.keep_first)
            return o
        if tables is not None or self.position is None:
            cos, sin, rot = tables if tables is not None else (None, None, 0)
            ops.qk_norm_rope_write(qkv, qw, kw, eps, cos, sin, rot, b.pos, b.tok_seg, kv.block_table,
                                   kv.page_size, kv.k, kv.v, s.num_heads, s.num_kv_heads, s.head_dim,
                                   write_kv=ctx.write_cache, offset=offset, norm_size=norm_size, blend=blend)
        else:
            # an encoding that is not a rotation of pairs: norm, then the encoding's own in-place
            # step on q and k, then the cache write
            ops.qk_norm_rope_write(qkv, qw, kw, eps, None, None, 0, b.pos, b.tok_seg, kv.block_table,
                                   kv.page_size, kv.k, kv.v, s.num_heads, s.num_kv_heads, s.head_dim,
                                   write_kv=False, offset=offset, norm_size=norm_size)
            self.position.apply(qkv, b, s.num_heads, s.num_kv_heads, s.head_dim)
            if ctx.write_cache:
                ops.qk_norm_rope_write(qkv, None, None, 0.0, None, None, 0, b.pos, b.tok_seg, kv.block_table,
                                       kv.page_size, kv.k, kv.v, s.num_heads, s.num_kv_heads, s.head_dim,
                                       write_kv=True, blend=blend)
        ops.paged_attention(qkv, kv.k, kv.v, b, kv.block_table, kv.page_size, o, s.num_heads,
                            s.num_kv_heads, s.head_dim, s.scale, s.window, self._sink, None, s.softcap, keep=s.keep_first)
        return o

    def _blend(self, qkv, batch):
        """What the cache write blends the step's values with (``ops.qk_norm_rope_write``), or None.  A "source" layer leaves
        its raw values, columns of its projections, under ``attention.source_values`` in the step's scratch."""
        s = self.spec
        if s.value_mix is None:
            return None
        held = getattr(batch, "scratch", None)
        if held is None:
            raise ValueError("layers that share values within a step need the step's map of buffers")
        if s.value_mix == "source":
            held["attention.source_values"] = (qkv[:, self.q_size + self.kv_size:], s.num_kv_heads, s.head_dim,
                                               s.value_dim or s.head_dim)
            return None
        first, heads, stride, n = held["attention.source_values"]
        if heads != s.num_kv_heads or n != (s.value_dim or s.head_dim):
            raise ValueError("values are blended head by head: both layers have as many key/value heads of the same value size")
        return first, stride, n, self.value_share


def distance_rows(rows: int, reach: float):
    """The row of a distance table of ``rows`` rows for every distance 0, 1, 2, ... up to the first that has the last row
    (all farther ones have it too): row n below half = rows // 2, then rows for ever longer spans,
    half + floor(ln(n / half) / ln(reach / half) * (rows - half)).  Worked out in float64."""
    half = rows // 2
    out, n = [], 0
    while not out or out[-1] != rows - 1:
        out.append(n if n < half else
                   min(rows - 1, half + math.floor(math.log(n / half) / math.log(reach / half) * (rows - half))))
        n += 1
    return out


@MIXERS.register("gated_attention")
class GatedAttention(Mixer):
    """``GatedAttentionSpec``: one product gives a row [q | k | v | gate] (k and v only if the layer owns its cache; v
    only if it has a value projection); one kernel prepares the row (biases, the norm over a whole projection, the
    rotation of neighbouring pairs, heads padded to the cache's head size, keys and values into their pages); the
    engine's paged attention kernels run with the layer's score options; the gate is applied and the heads are
    projected out.  A layer that reads another run's cache prepares its queries only.  Heads that are prepared one by
    one (a convolution over time, a norm per head, a query temperature) have a row kernel of their own
    (csrc/attention_conv.cu); the run keeps the last rows of its projections per request (``kept_floats``), also when the
    keys and values it attends to are another run's."""

    def __init__(self, spec, env):
        super().__init__(spec, env)
        s = spec
        if s.num_heads % s.num_kv_heads:
            raise ValueError(f"num_heads={s.num_heads} is not a multiple of num_kv_heads={s.num_kv_heads}")
        if s.window is not None and s.chunk is not None:
            raise ValueError("a window and a chunk exclude each other")
        if (s.window is not None and s.window <= 0) or (s.chunk is not None and s.chunk <= 0):
            raise ValueError("window and chunk must be positive")
        if s.gate not in (None, "head", "element"):
            raise ValueError(f"gate={s.gate!r}; known: None, 'head', 'element'")
        if s.values_are_keys and s.value_dim != s.key_dim:
            raise ValueError("values that are the keys have the keys' size")
        self.D = (max(s.key_dim, s.value_dim) + 15) // 16 * 16          # the head size of the cache and the kernels
        if not (16 <= self.D <= 256):
            raise ValueError(f"heads of {max(s.key_dim, s.value_dim)} elements: the attention kernels take up to 256")
        self.position = POSITION_ENCODINGS.build(s.position, env) if s.position is not None else None
        if self.position is not None and not getattr(self.position, "interleaved", False):
            raise ValueError("the row kernel rotates neighbouring pairs: the position encoding must be 'rope_interleaved'")
        if self.position is not None and s.position.rotary_dim > s.key_dim:
            raise ValueError("the rotary width is at most the key size")
        self.by_head = bool(s.conv_taps or s.head_norm_eps is not None or s.temperature is not None)
        if self.by_head and (s.bias or s.whole_norm_eps is not None or s.position is not None or s.values_are_keys):
            raise ValueError("heads that are prepared one by one (conv_taps, head_norm_eps, temperature) take no biases, norm over a "
                             "whole projection, rotation, or keys as values")
        if s.conv_taps is not None and not (1 <= s.conv_taps <= 33):
            raise ValueError("conv_taps: 1 to 33")
        if s.temperature is not None and int(s.temperature[1]) < 1:
            raise ValueError("temperature: a positive run length")
        if s.distance_bias is not None and (s.distance_bias[0] < 2 or not s.distance_bias[1] > s.distance_bias[0] // 2):
            raise ValueError("distance_bias: at least two rows, and a reach beyond half of them")
        if s.sink and s.fixed_sink is not None:
            raise ValueError("a learned sink and a fixed one exclude each other")
        self.nq = s.num_heads * s.key_dim
        self.nk = s.num_kv_heads * s.key_dim if s.own_cache else 0
        self.nv = s.num_kv_heads * s.value_dim if (s.own_cache and not s.values_are_keys) else 0
        self.ng = 0 if s.gate is None else s.num_heads if s.gate == "head" else s.num_heads * s.value_dim
        self._slopes = None
        self._sink = None
        self._taps = None
        self._bias = None

    # ------------------------------------------------------------------ parameters and cache
    def params(self):
        s = self.spec
        p = {"in": ParamSpec((self.nq + self.nk + self.nv + self.ng, s.hidden_size)),
             "o": ParamSpec((s.hidden_size, s.num_heads * self.D))}
        if s.bias:
            p["bias"] = ParamSpec((self.nq + self.nk + self.nv,), role="vector", init="normal:0.2")
        if s.whole_norm_eps is not None:
            p["q_norm"] = ParamSpec((self.nq,), role="vector", init="ones_normal")
            if s.own_cache:
                p["k_norm"] = ParamSpec((self.nk,), role="vector", init="ones_normal")
        if s.sink:
            p["sink"] = ParamSpec((s.num_heads,), role="vector", init="normal:0.5")
        if s.conv_taps:
            p["conv"] = ParamSpec((self.nq + self.nk + self.nv, s.conv_taps), role="vector", init="normal:0.5")
        if s.distance_bias is not None:
            p["rel"] = ParamSpec((s.distance_bias[0], s.num_heads), role="vector", init="normal:1.0")
        return p

    def bind(self, tensors):
        super().bind(tensors)
        s = self.spec
        if s.sink:
            self._sink = self.p_sink.float().contiguous()
        if s.slope_exponent is not None:
            h = torch.arange(1, s.num_heads + 1, dtype=torch.float64)
            self._slopes = torch.exp2(-float(s.slope_exponent) * h / s.num_heads).float().to(self.env.device)
        if s.fixed_sink is not None:
            self._sink = torch.full((s.num_heads,), float(s.fixed_sink), dtype=torch.float32, device=self.env.device)
        if self.by_head:                    # without a convolution: a filter of the token itself
            self._taps = self.p_conv.float().t().contiguous() if s.conv_taps else torch.ones(
                (1, self.nq + self.nk + self.nv), dtype=torch.float32, device=self.env.device)
        if s.distance_bias is not None:     # the table by distance instead of by row, [heads, distances]
            rows = torch.tensor(distance_rows(*s.distance_bias), dtype=torch.int64, device=self.p_rel.device)
            self._bias = self.p_rel.float()[rows].t().contiguous()

    def kept_floats(self):
        s = self.spec
        return (self.nq + self.nk + self.nv) * (s.conv_taps - 1) if s.conv_taps else 0

    def cache_need(self):
        s = self.spec
        return KVCacheNeed(s.num_kv_heads, self.D, s.cache_window) if s.own_cache else None

    def batch_tilings(self):
        if self.env.act_dtype != torch.bfloat16:
            return {}
        if self.D in ops.TC5_ATTENTION_HEAD_DIMS:
            return {ops.TILES_TC5: Tiling(ops.TC5_TILE_ROWS, heaviest_first=True)}
        return {ops.TILES_MMA: Tiling(ops.MMA_TILE_ROWS)}

    def graph_variant(self, n_tokens, longest_context):
        if self.env.act_dtype != torch.bfloat16:
            return {}
        s = self.spec
        bound = s.window or s.chunk
        return {ops.decode_splits_key(s.num_heads, s.num_kv_heads, bound):
                ops.decode_splits_for(n_tokens, longest_context, s.num_heads, s.num_kv_heads, bound)}

    def out_projection(self):
        return self.p_o

    # ------------------------------------------------------------------ one step
    def forward(self, x, ctx):
        s, b, kv = self.spec, ctx.batch, ctx.kv
        T, dev, dt = x.shape[0], x.device, x.dtype
        if kv is None:
            raise ValueError("a gated attention needs a paged cache: its own, or the one its schedule entry names")
        if kv.k.shape[-1] != self.D or kv.k.shape[1] != s.num_kv_heads:
            raise ValueError("the cache this layer reads has other heads than the layer")
        proj = ctx.buffer("gated_attention.proj", (T, self.nq + self.nk + self.nv + self.ng), dt, dev)
        ops.linear(x, self.p_in, proj)
        write = bool(ctx.write_cache and s.own_cache)
        q = ctx.buffer("gated_attention.q", (T, s.num_heads * self.D), dt, dev)
        if self.by_head:
            ops.attention_conv_prepare(proj, self._taps, ctx.kept, 0, b, kv, q, s.num_heads, s.num_kv_heads, s.key_dim, s.value_dim,
                                       self.D, s.head_norm_eps, s.temperature, own_kv=s.own_cache, write_kv=write)
        else:
            self._prepare_rows(proj, b, kv, q, write)
        o = ctx.buffer("gated_attention.o", (T, s.num_heads * self.D), dt, dev)
        ops.paged_attention(q, kv.k, kv.v, b, kv.block_table, kv.page_size, o, s.num_heads, s.num_kv_heads, self.D,
                            s.scale, s.window, self._sink, s.chunk, s.softcap, self._slopes, self._bias)
        if s.gate is not None:
            ops.attention_gate(o, proj, self.nq + self.nk + self.nv, s.gate == "head", s.num_heads, s.value_dim, self.D)
        y = ctx.buffer("gated_attention.y", (T, s.hidden_size), torch.float32, dev)
        ops.linear(o, self.p_o, y)
        return y

    def _prepare_rows(self, proj, b, kv, q, write: bool):
        s = self.spec
        biases = None
        if s.bias:
            bq, bk = self.p_bias[:self.nq], self.p_bias[self.nq:self.nq + self.nk]
            biases = (bq, bk if write else None, self.p_bias[self.nq + self.nk:] if write else None)
        norms = None
        if s.whole_norm_eps is not None:
            norms = (self.p_q_norm, self.p_k_norm if write else None)
        ops.attention_prepare(proj, 0, self.nq, -1 if (s.values_are_keys or not s.own_cache) else self.nq + self.nk,
                              biases, norms, float(s.whole_norm_eps or 0.0),
                              self.position.tables() if self.position is not None else None, b, kv, q,
                              s.num_heads, s.num_kv_heads, s.key_dim, s.value_dim, self.D, write_kv=write)
