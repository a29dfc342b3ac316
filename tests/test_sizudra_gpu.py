"""The Sizudra decoder through the engine against the plain implementation (tests/plain/sizudra_plain.py).

Every test makes a small configuration of its own with random weights (written as a bfloat16 checkpoint, as a model
folder holds them), replays a trace through the engine's step function and compares every logits row with the plain
implementation's, which walks the whole sequence in float64.  float32 path: every row within 1e-4 of its size.  bfloat16
path: rows weighed together (see ``assert_close``).  Where random weights would hide a fault (a key far back among hundreds,
a window that is one position off, a kept first key, a sink) scores are made sharp, and the test first shows that the plain
model itself moves by far more than the tolerance with that fault.
"""
import json
import math
import os
import random
import types

import numpy as np
import pytest
import torch

import helpers
from helpers import collect, mixed, pool_tokens, portions, random_ids, tail_decoded, whole
from plain import sizudra_plain as plain

pytestmark = pytest.mark.gpu

TOL = {"float32": 1e-4, "bfloat16": 1.0 / 12}
DTYPES = [torch.float32, torch.bfloat16]


# ------------------------------------------------------------------------------- configurations

def dense(ff=56):
    return {"kind": "dense", "ff": ff}


def moe(experts=6, top=2, ff=24, shared=16):
    m = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    return {**m, "shared": {"ff": shared}} if shared else m


def att(heads=4, kv_heads=2, dim=12, vdim=20, scale=None, rot=(300.0, 8), v_mix=True, mlp="default"):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else 1.5 * dim ** -0.5}
    if rot:
        m["rot"] = {"base": rot[0], "dims": rot[1]}
    if v_mix:
        m["v_mix"] = True
    return {"type": "attention", "mixer": m, "mlp": dense() if mlp == "default" else mlp}


def att2(size=11, keep_first=3, cap=5.0, **kw):
    layer = att(**kw)
    layer["type"] = "attention_2"
    layer["mixer"]["mask"] = {"size": size, "keep_first": keep_first}
    layer["mixer"]["softcap"] = cap
    return layer


def config(layers, vocab=97, width=40, eps=1e-5, bigram=(53, 7, 5)):
    c = {"architecture": "Sizudra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if bigram:
        c["embedding"] = {"bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))}
    return c


def full_config():
    """Both mixers and both feed-forwards in another order than any other test's, a layer without a feed-forward, one whose
    values are its own although an earlier layer's were blended, windows of several sizes."""
    return config([att2(v_mix=False, mlp=moe()), att(heads=6, rot=(1e4, 12), mlp=moe(5, 3, 16, 40)), att2(size=30, keep_first=7, dim=24, mlp=None),
                   att(heads=2, dim=16, v_mix=False, mlp=dense(33)), att2(size=5, keep_first=0, cap=2.0, mlp=moe(4, 1, 32, None)), att()])


def other_sizes_config():
    """The values one (a head, a key head, a window of one position, an expert, a bucket), sizes that fill no whole vector,
    keys wider than values and the other way round, a rotation of two elements, of all and of none, a window shorter than
    what it keeps, as many experts chosen as there are, a cap below and far above the scores, a width of odd pieces."""
    return config([att(heads=3, kv_heads=3, dim=7, vdim=33, rot=(50.0, 2), mlp=moe(1, 1, 9, 1)),
                   att2(heads=9, kv_heads=3, dim=34, vdim=33, rot=(90.0, 34), size=1, keep_first=4, cap=0.7, mlp=dense(9)),
                   att2(heads=6, kv_heads=3, dim=24, vdim=33, rot=None, size=3, keep_first=17, cap=900.0, mlp=moe(3, 3, 8, 5)),
                   att2(heads=5, kv_heads=1, dim=130, vdim=18, rot=(7.0, 6), size=200, keep_first=1, v_mix=False, mlp=None),
                   att(heads=1, kv_heads=1, dim=64, vdim=6, rot=(1e6, 64), v_mix=False, mlp=moe(33, 4, 7, 12)),
                   att(heads=3, kv_heads=3, dim=20, vdim=33, rot=(20.0, 20), mlp=dense(8))], vocab=61, width=36, eps=1e-3, bigram=(1, 0, 3))


def wide_config():
    """Sizes that pick the tensor-core kernels of prompts in bfloat16 (heads of 64 and 128, enough pairs for the grouped
    experts, enough rows for the woven gated product) and the 16-byte forms of the kernels around them."""
    return config([att(heads=4, kv_heads=2, dim=64, vdim=40, rot=(1e4, 32), mlp=moe(8, 2, 32, 64)),
                   att2(heads=8, kv_heads=2, dim=48, vdim=40, rot=(1e3, 48), size=150, keep_first=70, cap=8.0, mlp=dense(96)),
                   att2(heads=4, kv_heads=1, dim=128, vdim=128, rot=(1e5, 64), size=300, keep_first=4, v_mix=False, mlp=moe(4, 2, 64, 24)),
                   att(heads=4, kv_heads=2, dim=40, vdim=40, rot=(1e4, 16), mlp=None)], width=64)


_MODELS = {}


def model(tmp_path_factory, name, raw, seed=3, patch=None):
    """(model folder, (config, float64 weights), memo of plain logits), cached.  ``patch`` changes tensors (name -> tensor)
    before they are written."""
    if name not in _MODELS:
        from return_b200.config.sizudra_config import SizudraConfig
        from return_b200.weights import loader
        from return_b200.weights.safetensors_io import write_safetensors
        d = str(tmp_path_factory.mktemp(name))
        loader.write_random_model(d, SizudraConfig(raw), seed, torch.bfloat16)
        path = os.path.join(d, "model.safetensors")
        tensors = plain.read_safetensors(path)
        for i, layer in enumerate(raw["layers"]):                  # files hold a share for every layer that could blend
            if layer["mixer"].get("v_mix"):
                tensors.setdefault(f"l{i}.mix.vmix", torch.tensor(0.7))
        if patch is not None:
            patch(tensors)
        write_safetensors(path, [(n, t.bfloat16().contiguous()) for n, t in tensors.items()])
        _MODELS[name] = (d, plain.read_model(d), {})
    return _MODELS[name]


def plain_rows(entry, ids):
    d, (c, w), memo = entry
    key = tuple(ids)
    if key not in memo:
        memo[key] = plain.forward(c, w, list(ids)).float()
    return memo[key]


def close_calls(entry, ids):
    """[T] bool: tokens of which some router's last chosen and first unchosen logits are nearly tied (within 6 % of the logits'
    spread): rounding may choose the other expert there, and the row is then another one."""
    tied = torch.zeros(len(ids), dtype=torch.bool)
    true_experts = plain.experts

    def watched(w, p, mlp, a):
        z, top = a @ w[p + "router"].T, mlp["router"]["top"]
        if z.shape[1] > top:
            best = z.topk(top + 1, dim=1).values
            tied.logical_or_(best[:, -2] - best[:, -1] < 0.06 * z.std(dim=1))
        return true_experts(w, p, mlp, a)
    _run_with(entry, ids, experts=watched)
    return tied


def _run_with(entry, ids, **changed):
    """Plain logits with functions of the plain implementation replaced: what an engine with that fault would give."""
    kept = {n: getattr(plain, n) for n in changed}
    try:
        for n, f in changed.items():
            setattr(plain, n, f)
        return plain.forward(*entry[1], list(ids)).float()
    finally:
        for n, f in kept.items():
            setattr(plain, n, f)


def requests_for(entry, lens, seed=10):
    return {f"r{i}": random_ids(entry[1][0]["vocab"], n, seed + i) for i, n in enumerate(lens)}


def run_trace(model_dir, dtype, steps, page_size=16, max_reside=4, graph=False):
    from return_b200.engine.replay import TraceReplayer
    rp = TraceReplayer(model_dir, dtype, pool_tokens(steps), page_size=page_size, max_reside=max_reside, poison=True,
                       use_cuda_graph=graph)
    outs = []
    for st in steps:
        lg = rp.run_step(st)
        outs.append(None if lg is None else lg.float().cpu())
        rp.runner.manager.check()
    assert rp.runner.manager.num_requests == 0 and rp.runner.manager.pages_used() == [0] * len(rp.runner.manager.groups)
    return collect(steps, outs)


def row_errors(got, want):
    """The error of every row as a part of the row's size, both with their means taken off (as the softmax sees them)."""
    assert got.shape == want.shape and torch.isfinite(got).all()
    got, want = got - got.mean(1, keepdim=True), want - want.mean(1, keepdim=True)
    return (got - want).norm(dim=1) / want.norm(dim=1)


def assert_close(got, want, dtype, what="", mean=0.03, robust=False, tied=None):
    """float32: every row within 1e-4 of its size.  bfloat16: rounding moves single rows far more than the rest (a router
    whose best candidates are nearly tied, and then every row that looks at that one), so the rows are weighed together:
    their mean within 3 %, at most one row in ten (or two) beyond a twelfth, none but the ``tied`` ones (``close_calls``)
    beyond four tenths.  ``robust``: configurations drawn at random, where a single row
    may move by its own size but the middle row may not."""
    e = row_errors(got, want)
    if dtype == "float32":
        over = int((e > TOL[dtype]).sum())
        assert over == 0 or (robust and over <= 1 and float(e.median()) < 1e-5), (what, dtype, float(e.max()), int(e.argmax()))
        return
    over = int((e > TOL[dtype]).sum())
    if robust:
        assert over <= max(2, e.numel() // 10) and float(e.median()) < mean, (what, dtype, over, float(e.max()), float(e.median()))
        return
    clear = torch.cat([e if tied is None else e[~tied], e.new_zeros(1)])
    assert over <= max(2, e.numel() // 10) and float(clear.max()) < 0.4 and float(e.mean()) < mean, \
        (what, dtype, over, float(e.max()), float(e.mean()), int(e.argmax()))


def compare(entry, dtype, steps, requests, robust=False, **kw):
    got = run_trace(entry[0], dtype, steps, **kw)
    for rid, ids in requests.items():
        tied = close_calls(entry, ids) if dtype == "bfloat16" and not robust else None
        assert_close(got[rid], plain_rows(entry, ids), dtype, rid, robust=robust, tied=tied)


# ------------------------------------------------------------------------------- kernels of single mechanisms

def _step(lens, pos0, page, D, G, dtype, seed=0, tilings=True):
    """A step's tables and empty pools for segments of ``lens`` tokens behind ``pos0`` cached ones each."""
    from return_b200.ext import ops
    cu = np.concatenate([[0], np.cumsum(lens)]).astype(np.int32)
    n = len(lens)
    kv_len = np.asarray([p + m for p, m in zip(pos0, lens)], np.int32)
    blocks = int((kv_len.max() + page - 1) // page)
    g = torch.Generator().manual_seed(seed)
    table = torch.randperm(n * blocks, generator=g).view(n, blocks).int()
    i32 = lambda v: torch.as_tensor(np.asarray(v, np.int32)).cuda()
    decode = [i for i, m in enumerate(lens) if m == 1]
    multi = [i for i, m in enumerate(lens) if m > 1]
    tiles = {name: np.asarray([(i, r) for i in multi for r in range(0, lens[i], rows)], np.int32).reshape(-1, 2)
             for name, rows in ((ops.TILES_TC5, ops.TC5_TILE_ROWS), (ops.TILES_MMA, ops.MMA_TILE_ROWS))}
    host = types.SimpleNamespace(num_multi=len(multi), decode_segs=np.asarray(decode, np.int32), num_tokens=int(cu[-1]), seg_kv_len=kv_len,
                                 tiles=tiles)
    b = types.SimpleNamespace(
        host=host, scratch={}, variant={}, num_tokens=int(cu[-1]), num_segments=n, cu_q=i32(cu), seg_pos0=i32(pos0), seg_kv_len=i32(kv_len),
        decode_segs=i32(decode), tiles={k: i32(v) for k, v in tiles.items()},
        pos=i32([pos0[i] + k for i, m in enumerate(lens) for k in range(m)]), tok_seg=i32([i for i, m in enumerate(lens) for _ in range(m)]))
    pool = lambda: torch.full((n * blocks, G, page, D), float("nan"), dtype=dtype, device="cuda")
    return b, types.SimpleNamespace(k=pool(), v=pool(), block_table=table.cuda(), page_size=page), table


def _fill(pool, table, page, rows):
    """Writes rows[i] [positions, G, D] of segment i into its pages."""
    for i, r in enumerate(rows):
        pos = torch.arange(r.shape[0])
        pool[table[i, pos // page].long().cuda(), :, (pos % page).cuda()] = r.to(pool.dtype).cuda()


# segments: lengths and cached tokens before them; portions at starts that are no tile's, decoded tokens with short and long
# contexts, a portion of several row blocks
ATTENTION_STEPS = [([40, 1, 3, 1, 70], [0, 0, 90, 333, 33]), ([300, 2, 1], [417, 63, 1900])]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window,keep,cap,sink", [(24, 5, None, False), (64, 64, 3.0, True), (1, 1, None, True), (130, 3, 2.0, False),
                                                  (7, 100, 9.0, True), (40, 0, 4.0, True), (None, 0, 1.5, True), (500, 17, 0.2, False)])
@pytest.mark.parametrize("D,Hq,G", [(16, 4, 2), (48, 3, 1), (64, 4, 2), (128, 10, 1)])
def test_attention_over_a_window_and_kept_first_keys(D, Hq, G, window, keep, cap, sink, dtype):
    """Every query of a step against the formula: windows inside and across key tiles and pages, kept keys that end inside a
    tile, fill one or reach beyond the window's start, with and without capped scores (small and beyond the cap) and a
    sink; keys that no query of the step can see lie on pages that were given back."""
    from return_b200.ext import ops
    for si, (lens, pos0) in enumerate(ATTENTION_STEPS):
        page = (8, 16)[si]
        b, kv, table = _step(lens, pos0, page, D, G, dtype, seed=si)
        g = torch.Generator().manual_seed(D + si)
        rnd = lambda *s: torch.randn(s, generator=g)
        T = b.num_tokens
        keys, values = [rnd(p + n, G, D).to(dtype) for n, p in zip(lens, pos0)], [rnd(p + n, G, D).to(dtype) for n, p in zip(lens, pos0)]
        q = (rnd(T, Hq * D) * 1.5).to(dtype)
        _fill(kv.k, table, page, keys)
        _fill(kv.v, table, page, values)
        if window:                                     # blocks that the window has passed and that hold no kept key
            bt = table.clone()
            for i, p in enumerate(pos0):
                bt[i, (keep + page - 1) // page:max(0, p - window + 1) // page] = -1
            kv.block_table = bt.cuda()
        sk = rnd(Hq) if sink else None
        out = torch.empty((T, Hq * D), dtype=dtype, device="cuda")
        ops.paged_attention(q.cuda(), kv.k, kv.v, b, kv.block_table, page, out, Hq, G, D, D ** -0.5, window,
                            sk.cuda() if sink else None, None, cap, keep=keep)
        ops.check_status(out.device)
        got, row = out.cpu().double().view(T, Hq, D), 0
        for i, (n, p) in enumerate(zip(lens, pos0)):
            qs = torch.zeros(p + n, Hq, D, dtype=torch.float64)
            qs[p:] = q[row:row + n].double().view(n, Hq, D)
            s = torch.einsum("ihd,jhd->hij", qs[p:], keys[i].double().repeat_interleave(Hq // G, 1)) * D ** -0.5
            if cap:
                s = plain.soft_cap(s, cap)
            ok = plain.visible(p + n, {"size": window, "keep_first": keep} if window else None)[p:]
            share = plain.softmax_with_sink(s, ok, sk.double() if sink else None)
            want = torch.einsum("hij,jhd->ihd", share, values[i].double().repeat_interleave(Hq // G, 1))
            err = (got[row:row + n] - want).abs().max()
            assert err < (2e-5 if dtype == torch.float32 else 3e-2), (i, float(err))
            row += n


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("lens", [[3, 1, 40], [1, 1], [900, 1, 700]])
@pytest.mark.parametrize("Hq,G,dim,vdim,rot,blend", [(4, 2, 12, 20, 8, True), (3, 1, 64, 40, 32, True), (6, 2, 64, 64, 64, False),
                                                     (2, 2, 30, 128, 16, True), (4, 1, 128, 128, 48, True), (5, 5, 16, 7, 0, True),
                                                     (8, 2, 32, 32, 16, True), (2, 1, 130, 9, 4, True)])
def test_rows_normed_rotated_blended_and_cached(Hq, G, dim, vdim, rot, blend, lens, dtype):
    """Heads padded to the cache's size, normed over their own elements, partly rotated; values blended with another buffer's
    whose heads are padded otherwise; few rows and enough for the 16-byte form."""
    from return_b200.ext import ops
    D = (max(dim, vdim) + 15) // 16 * 16
    D1 = (vdim + 15) // 16 * 16 + 16                                 # the earlier layer's padded heads
    pos0 = [5 * i + 2 for i in range(len(lens))]
    page = 8
    b, kv, table = _step(lens, pos0, page, D, G, dtype, seed=dim)
    T = b.num_tokens
    g = torch.Generator().manual_seed(T + dim)
    rnd = lambda *s: torch.randn(s, generator=g)
    pad = lambda t, to: torch.nn.functional.pad(t, (0, to - t.shape[-1]))
    q, k, v, v1 = (rnd(T, n, m).to(dtype) for n, m in ((Hq, dim), (G, dim), (G, vdim), (G, vdim)))
    qkv = torch.cat([pad(x, D).reshape(T, -1) for x in (q, k, v)], 1).cuda()
    first = torch.cat([rnd(T, 24).to(dtype), pad(v1, D1).reshape(T, -1)], 1).cuda()[:, 24:]
    wq, wk, share = rnd(dim) + 1, rnd(dim) + 1, torch.tensor([0.3])
    top = max(p + n for n, p in zip(lens, pos0))
    f = torch.arange(max(rot // 2, 1), dtype=torch.float64)
    ang = torch.outer(torch.arange(top, dtype=torch.float64), 40.0 ** (-2 * f / max(rot, 1)))
    ops.qk_norm_rope_write(qkv, pad(wq, D).cuda(), pad(wk, D).cuda(), 1e-3, ang.cos().float().cuda() if rot else None,
                           ang.sin().float().cuda() if rot else None, rot, b.pos, b.tok_seg, kv.block_table, page, kv.k, kv.v, Hq, G, D,
                           norm_size=dim, blend=(first, D1, vdim, share.cuda()) if blend else None)
    got_q, kk, vv, row = qkv[:, :Hq * D].cpu().double().view(T, Hq, D), kv.k.cpu().double(), kv.v.cpu().double(), 0
    tol = 2e-5 if dtype == torch.float32 else 2e-2

    def check(got, want):
        assert ((got[..., :want.shape[-1]] - want).abs() <= tol * want.abs().clamp(min=1.0)).all() and (got[..., want.shape[-1]:] == 0).all()
    for i, (n, p) in enumerate(zip(lens, pos0)):
        r = slice(row, row + n)
        turn = lambda x, w: plain.rotate_halves(plain.rms_norm(x.double(), w.double(), 1e-3), 40.0, rot, p) if rot else plain.rms_norm(x.double(), w.double(), 1e-3)
        check(got_q[r], turn(q[r], wq))
        pos = torch.arange(p, p + n)
        pages = table[i, pos // page].long()
        check(kk[pages, :, pos % page], turn(k[r], wk))
        check(vv[pages, :, pos % page], plain.blend_values(v[r].double(), v1[r].double(), float(share)) if blend else v[r].double())
        kk[pages, :, pos % page] = vv[pages, :, pos % page] = float("nan")
        row += n
    assert kk.isnan().all() and vv.isnan().all()                          # nothing else was written


@pytest.mark.parametrize("window,keep,cap,sink", [(None, 0, None, False), (20, 6, 3.0, True), (300, 40, None, True), (None, 0, 1.0, False)])
@pytest.mark.parametrize("Hq,G,dim,vdim,rot", [(4, 2, 24, 40, 16), (3, 1, 64, 64, 64), (20, 1, 128, 96, 32)])
def test_decoding_in_one_kernel_is_decoding_in_two(Hq, G, dim, vdim, rot, window, keep, cap, sink):
    """The kernel that norms, rotates, blends, caches and attends for single tokens against the row kernel followed by the
    attention kernel: the same pages, outputs within a rounding."""
    from return_b200.ext import ops
    D = (max(dim, vdim) + 15) // 16 * 16
    pos0 = [0, 3, 15, 16, 31, 200, 777]
    lens, page = [1] * len(pos0), 16
    g = torch.Generator().manual_seed(dim)
    rnd = lambda *s: torch.randn(s, generator=g)
    T = len(lens)
    pad = lambda t, to: torch.nn.functional.pad(t, (0, to - t.shape[-1]))
    qkv = torch.cat([pad(rnd(T, n, m).bfloat16(), D).reshape(T, -1) for n, m in ((Hq, dim), (G, dim), (G, vdim))], 1).cuda()
    first = pad(rnd(T, G, vdim).bfloat16(), D).reshape(T, -1).cuda()
    w = pad(rnd(dim) + 1, D).cuda()
    ang = torch.outer(torch.arange(800, dtype=torch.float64), 90.0 ** (-2 * torch.arange(rot // 2, dtype=torch.float64) / rot))
    cos, sin = ang.cos().float().cuda(), ang.sin().float().cuda()
    sk, blend = rnd(Hq).cuda() if sink else None, (first, D, vdim, torch.tensor([0.4]).cuda())
    past = [(rnd(p, G, D), rnd(p, G, D)) for p in pos0]
    outs, pools = [], []
    for fused in (True, False):
        b, kv, table = _step(lens, pos0, page, D, G, torch.bfloat16, seed=1)
        _fill(kv.k, table, page, [a for a, _ in past])
        _fill(kv.v, table, page, [a for _, a in past])
        out = torch.empty((T, Hq * D), dtype=torch.bfloat16, device="cuda")
        if fused:
            ops.attention_decode_fused(qkv, w, w, 1e-5, 0.0, cos, sin, rot, kv.k, kv.v, b, kv.block_table, page, out, Hq, G, D, dim ** -0.5,
                                       window, norm_size=dim, blend=blend, sink=sk, softcap=cap, keep=keep)
        else:
            x = qkv.clone()
            ops.qk_norm_rope_write(x, w, w, 1e-5, cos, sin, rot, b.pos, b.tok_seg, kv.block_table, page, kv.k, kv.v, Hq, G, D,
                                   norm_size=dim, blend=blend)
            ops.paged_attention(x, kv.k, kv.v, b, kv.block_table, page, out, Hq, G, D, dim ** -0.5, window, sk, None, cap, keep=keep)
        outs.append(out.cpu().float())
        pools.append((kv.k.cpu().nan_to_num(9.0), kv.v.cpu().nan_to_num(9.0)))
    assert torch.equal(pools[0][0], pools[1][0]) and torch.equal(pools[0][1], pools[1][1])
    assert torch.isfinite(outs[0]).all() and (outs[0] - outs[1]).abs().max() < 2e-2


@pytest.mark.parametrize("cap", [0.3, 5.0, 200.0])
def test_capped_scores_on_both_sides_of_the_polynomial(cap):
    """One query row whose scores run from far below the cap to beyond it, so that key tiles take the polynomial and the
    exponential form of the tanh in turn: weights against the formula, in prompts and decoded, for two head sizes' kernels."""
    from return_b200.ext import ops
    for D in (32, 64):
        n, page = 384, 16
        for lens, pos0 in (([n], [0]), ([1], [n - 1])):
            b, kv, table = _step(lens, pos0, page, D, 1, torch.bfloat16)
            u = torch.zeros(D)
            u[0] = 8.0
            size = torch.linspace(0.0, 4.0 * cap, n)[torch.randperm(n, generator=torch.Generator().manual_seed(2))] if cap < 100 else \
                torch.linspace(-300.0, 300.0, n)
            k = torch.zeros(n, 1, D)
            k[:, 0, 0] = size
            v = torch.randn(n, 1, D, generator=torch.Generator().manual_seed(3)).bfloat16()
            k = k.bfloat16()
            _fill(kv.k, table, page, [k])
            _fill(kv.v, table, page, [v])
            q = u.bfloat16().expand(b.num_tokens, D).contiguous().cuda()
            out = torch.empty((b.num_tokens, D), dtype=torch.bfloat16, device="cuda")
            ops.paged_attention(q, kv.k, kv.v, b, kv.block_table, page, out, 1, 1, D, 0.125, None, None, None, cap)
            ops.check_status(out.device)
            s = plain.soft_cap(8.0 * k[:, 0, 0].double() * 0.125, cap).expand(n, n)[None]
            p = plain.softmax_with_sink(s, plain.visible(n, None))
            want = torch.einsum("hij,jhd->ihd", p, v.double())[pos0[0]:].reshape(b.num_tokens, D)
            assert (out.cpu().double() - want).abs().max() < 2e-2, (D, lens)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,H", [(1, 36), (5, 33), (3, 640), (700, 64), (2, 4096), (2, 6001)])
def test_joint_of_two_sublayers(T, H, dtype):
    """Norm of the output, add and copy, in every combination the blocks use, against the formulas."""
    from return_b200.ext import ops
    g = torch.Generator().manual_seed(H)
    rnd = lambda *s: torch.randn(s, generator=g)
    x, y, w, w2 = rnd(T, H), (rnd(T, H) * 3).to(dtype), rnd(H) + 1, rnd(H) + 1
    want = x.double() + plain.rms_norm(y.double(), w.double(), 1e-3)
    tol = 4e-6 if dtype == torch.float32 else 2e-2
    for nxt in (None, (w2.cuda(), 1e-2, 0.0)):
        s, out = x.cuda(), torch.empty((T, H), dtype=dtype, device="cuda")
        ops.postnorm_add_norm(s, y.cuda(), (w.cuda(), 1e-3, 0.0), nxt, out)
        assert (s.cpu().double() - want).abs().max() < 4e-6 * 8
        o = want if nxt is None else plain.rms_norm(want, w2.double(), 1e-2)
        assert ((out.cpu().double() - o).abs() <= tol * o.abs().clamp(min=2.0)).all()
    s = x.cuda()
    ops.postnorm_add_norm(s, y.cuda(), (w.cuda(), 1e-3, 0.0))                          # no rows wanted
    assert (s.cpu().double() - want).abs().max() < 4e-6 * 8
    s, out = x.cuda(), torch.empty((T, H), dtype=dtype, device="cuda")
    ops.postnorm_add_norm(s, None, None, None, out)                                    # nothing added: the stream itself
    assert torch.equal(s.cpu(), x) and torch.equal(out.cpu(), x.to(dtype))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("M", [1, 7, 30, 900])
@pytest.mark.parametrize("I,K,weave", [(48, 40, 8), (33, 36, 0), (256, 128, 8), (56, 64, 0)])
def test_units_gated_by_gelu(I, K, weave, M, dtype):
    """Few rows (the gate in the weight-streaming product), some (a kernel of its own), many (in the tcgen05 product)."""
    from return_b200.ext import ops
    g = torch.Generator().manual_seed(I + M)
    x, gate, up = (torch.randn(s, generator=g).to(dtype) for s in ((M, K), (I, K), (I, K)))
    gate, up = (gate * 0.3).to(dtype), (up * 0.3).to(dtype)
    w = torch.stack([gate.view(-1, 8, K), up.view(-1, 8, K)], 1).reshape(2 * I, K) if weave else torch.cat([gate, up])
    out = torch.empty((M, I), dtype=dtype, device="cuda")
    ops.gated_linear(x.cuda(), w.cuda(), out, weave, None, "gelu_tanh")
    ops.check_status(out.device)
    want = plain.gelu_tanh(x.double() @ gate.double().T) * (x.double() @ up.double().T)
    assert (out.cpu().double() - want).abs().max() < (2e-5 if dtype == torch.float32 else 3e-2) * float(want.abs().max())
    ops.gated_linear(x.cuda(), w.cuda(), out, weave)                                   # and silu as before
    a = x.double() @ gate.double().T
    want = a * torch.sigmoid(a) * (x.double() @ up.double().T)
    assert (out.cpu().double() - want).abs().max() < (2e-5 if dtype == torch.float32 else 3e-2) * float(want.abs().max())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,E,top,W,F,S", [(1, 6, 2, 40, 24, 16), (9, 5, 5, 36, 9, 7), (70, 12, 2, 64, 40, 24), (600, 9, 3, 72, 48, 96),
                                           (700, 33, 2, 128, 256, 0), (20, 1, 1, 32, 8, 8)])
def test_experts_without_a_gate_beside_a_gated_shared_one(T, E, top, W, F, S, dtype):
    """The part itself: pairs that stream their expert's weights, sorted pairs on the tensor cores, and on tcgen05."""
    from return_b200.ext import ops
    from return_b200.parts.base import FEED_FORWARDS, BuildEnv
    from return_b200.parts.spec import DenseMLPSpec, MoESpec
    g = torch.Generator().manual_seed(T + E)
    rnd = lambda *s: torch.randn(s, generator=g)
    mats = {"router": rnd(E, W), "sg": rnd(1, W) * W ** -0.5, "sup": rnd(max(S, 1), W) * W ** -0.5, "sdown": rnd(W, max(S, 1)) * 0.3}
    up, down = rnd(E, F, W) * W ** -0.5, rnd(E, W, F) * F ** -0.5
    mats = {n: t.to(dtype) for n, t in mats.items()}
    up, down, x = up.to(dtype), down.to(dtype), rnd(T, W).to(dtype)
    unit = lambda n: DenseMLPSpec(W, n, "relu2")
    ff = FEED_FORWARDS.build(MoESpec(W, E, top, unit(F), shared=unit(S) if S else None, renorm_tiny=0.0, shared_gate=bool(S)),
                             BuildEnv(dtype, torch.device("cuda")))
    tensors = {"router": torch.cat([mats["router"]] + ([mats["sg"]] if S else [])), "experts.up": up.reshape(E * F, W),
               "experts.down": down.reshape(E * W, F)}
    if S:
        tensors.update({"shared.up": mats["sup"], "shared.down": mats["sdown"]})
    assert {n: tuple(p.shape) for n, p in ff.params().items()} == {n: tuple(t.shape) for n, t in tensors.items()}
    ff.bind({n: t.cuda() for n, t in tensors.items()})
    got = ff.forward(x.cuda(), None).cpu().double()
    ops.check_status(torch.device("cuda", 0))
    w = {"router": mats["router"].double(), "shared.up": mats["sup"].double(), "shared.down": mats["sdown"].double(), "shared.sg": mats["sg"].double()}
    for e in range(E):
        w[f"e{e}.up"], w[f"e{e}.down"] = up[e].double(), down[e].double()
    want = plain.experts(w, "", {"router": {"experts": E, "top": top}, "shared": {"ff": S} if S else None}, x.double())
    z = x.double() @ w["router"].T
    best = z.topk(min(top + 1, E), dim=1).values
    clear = (best[:, -2] - best[:, -1] > 1e-3) if E > top else torch.ones(T, dtype=torch.bool)     # not a close call
    err = (got - want).norm(dim=1) / want.norm(dim=1).clamp(min=1e-3)
    assert float(err[clear].max()) < (2e-5 if dtype == torch.float32 else 4e-2) and clear.sum() >= T * 0.9


# ------------------------------------------------------------------------------- each mechanism alone, as a small model

ALONE = {
    "attention": lambda: config([att(mlp=None)], bigram=None),
    "attention_without_rotation": lambda: config([att(rot=None, v_mix=False, mlp=None)], bigram=None),
    "windowed": lambda: config([att2(mlp=None)], bigram=None),
    "pairs_of_tokens": lambda: config([att(mlp=None)], bigram=(29, 5, 3)),
    "blended_values": lambda: config([att(mlp=None), att2(dim=24, mlp=None), att(v_mix=False, mlp=None), att(heads=2, dim=30, mlp=None)], bigram=None),
    "gated_unit": lambda: config([att(mlp=dense(48))], bigram=None),
    "experts": lambda: config([att(mlp=moe(10, 3, 16, 24))], bigram=None),
    "experts_without_a_shared_one": lambda: config([att(mlp=moe(7, 2, 16, None))], bigram=None),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(ALONE))
def test_each_mechanism_alone(tmp_path_factory, name, dtype):
    """A model of one layer (more where values are blended): whole prompts, prompts against token-by-token decoding, and
    portions down to single first tokens."""
    entry = model(tmp_path_factory, "alone_" + name, ALONE[name](), seed=7)
    reqs = requests_for(entry, (70, 9), seed=40)
    compare(entry, dtype, whole(reqs), reqs)
    compare(entry, dtype, tail_decoded(reqs, tail=40), reqs, page_size=8)
    compare(entry, dtype, portions(reqs, [1, 1, 2, 17, 3, 30]), reqs, page_size=4)


# ------------------------------------------------------------------------------- the whole model under every schedule

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_whole_prompts_and_decoding(tmp_path_factory, dtype):
    entry = model(tmp_path_factory, "full", full_config())
    reqs = requests_for(entry, (130, 37, 1, 64), seed=10)
    compare(entry, dtype, whole(reqs), reqs)
    compare(entry, dtype, tail_decoded(reqs, tail=48), reqs)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_portions_of_several_sizes(tmp_path_factory, dtype):
    entry = model(tmp_path_factory, "full", full_config())
    reqs = requests_for(entry, (150, 33), seed=14)
    compare(entry, dtype, portions(reqs, [2, 29, 13, 2, 5, 40, 3]), reqs, page_size=8)
    compare(entry, dtype, portions(reqs, [64, 1, 2, 16]), reqs, page_size=16)
    compare(entry, dtype, portions(reqs, [2]), reqs, page_size=4)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_mixed_batches_with_pages_and_slots_used_again(tmp_path_factory, dtype):
    """Six requests through two and three slots, portions beside decoded tokens, requests that sit out a step: every
    request's rows are those of the request alone."""
    entry = model(tmp_path_factory, "full", full_config())
    reqs = requests_for(entry, (90, 41, 7, 66, 30, 2), seed=22)
    compare(entry, dtype, mixed(reqs, max_live=3, portion=19, decode_tail=12, seed=1), reqs, page_size=8, max_reside=3)
    compare(entry, dtype, mixed(reqs, max_live=2, portion=7, decode_tail=25, seed=2), reqs, page_size=4, max_reside=2)


def test_batching_and_cutting_do_not_change_float32_logits_at_all(tmp_path_factory):
    entry = model(tmp_path_factory, "full", full_config())
    reqs = requests_for(entry, (80, 35, 12), seed=31)
    a = run_trace(entry[0], "float32", whole(reqs))
    b = run_trace(entry[0], "float32", mixed(reqs, max_live=3, portion=9, decode_tail=10, seed=5), page_size=4, max_reside=3)
    c = run_trace(entry[0], "float32", portions(reqs, [2, 31, 1, 7]), page_size=8)
    for rid in reqs:
        assert torch.equal(a[rid], b[rid]) and torch.equal(a[rid], c[rid]), rid


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_other_sizes(tmp_path_factory, dtype):
    entry = model(tmp_path_factory, "other", other_sizes_config(), seed=11)
    reqs = requests_for(entry, (75, 20, 1), seed=20)
    compare(entry, dtype, whole(reqs), reqs)
    compare(entry, dtype, mixed(reqs, max_live=2, portion=11, decode_tail=9, seed=3), reqs, page_size=4, max_reside=2)
    compare(entry, dtype, tail_decoded(reqs, tail=70), reqs, page_size=16)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_many_query_heads_on_one_key_head(tmp_path_factory, dtype):
    """Twenty and thirty-six query heads a key head: the decode kernel packs a key head's query heads into tiles of 16
    rows, and every row keeps its own head's sink."""
    raw = config([att(heads=20, kv_heads=1, dim=16, vdim=16, mlp=None), att2(heads=36, kv_heads=1, dim=16, vdim=16, size=20, mlp=dense(24))], width=48)
    entry = model(tmp_path_factory, "many_heads", raw, seed=9)
    reqs = requests_for(entry, (70, 33), seed=44)
    compare(entry, dtype, tail_decoded(reqs, tail=45), reqs, page_size=8)
    compare(entry, dtype, mixed(reqs, max_live=2, portion=9, decode_tail=20, seed=7), reqs, page_size=4, max_reside=2)


def _random_config(rng):
    """A configuration no fixed case has: two to five layers of random kinds and sizes."""
    layers, shared_kv = [], (rng.choice([1, 2, 3]), rng.choice([5, 8, 16, 24, 40]))          # of the layers that blend values
    for _ in range(rng.randint(2, 5)):
        mlp = rng.choice([None, dense(rng.choice([7, 24, 40])), moe(*rng.choice([(4, 1, 16, 8), (6, 2, 8, None), (9, 3, 12, 20), (5, 5, 8, 3)]))])
        v_mix = rng.random() < 0.6
        kv, vdim = shared_kv if v_mix else (rng.choice([1, 2, 3]), rng.choice([7, 16, 33]))
        dim = rng.choice([7, 8, 16, 20, 48, 64])
        rot = rng.choice([None, (rng.choice([10.0, 1e4]), 2 * rng.randint(1, dim // 2))])
        opts = dict(heads=kv * rng.choice([1, 2, 3, 5]), kv_heads=kv, dim=dim, vdim=vdim, rot=rot, v_mix=v_mix, mlp=mlp)
        if rng.random() < 0.5:
            opts.update(size=rng.choice([1, 2, 9, 16, 33, 64]), keep_first=rng.choice([0, 1, 4, 16, 19]), cap=rng.choice([0.5, 3.0, 40.0]))
            layers.append(att2(**opts))
        else:
            layers.append(att(**opts))
    return config(layers, vocab=rng.randint(30, 200), width=rng.choice([24, 33, 36, 40, 56, 64]), eps=rng.choice([1e-6, 1e-5, 1e-3]),
                  bigram=rng.choice([None, (41, 3, 11)]))


@pytest.mark.parametrize("seed", list(range(12)))
def test_random_configurations_and_traces(tmp_path_factory, seed):
    rng = random.Random(500 + seed)
    raw = _random_config(rng)
    entry = model(tmp_path_factory, f"fuzz{seed}", raw, seed=seed)
    reqs = requests_for(entry, [rng.randint(1, 80) for _ in range(rng.randint(2, 4))], seed=100 + seed)
    steps = mixed(reqs, max_live=rng.randint(1, 3), portion=rng.randint(2, 30), decode_tail=rng.randint(0, 20), seed=seed)
    page = rng.choice([4, 8, 16, 32])
    for dtype in ("float32", "bfloat16"):
        try:
            compare(entry, dtype, steps, reqs, robust=True, page_size=page, max_reside=3)
        except AssertionError as e:
            raise AssertionError((raw, page, str(e)[:300]))


# ------------------------------------------------------------------------------- far keys, edges, sinks, blends, states

def _asking_pair(entry, scale_name="l0.mix."):
    """(token that asks, token that answers, filler tokens): without rotation and pairs of tokens, the query of the first
    scores the key of the second far above those of the fillers."""
    c, w = entry[1]
    m = c["layers"][0]["mixer"]
    x = w["embed"]
    q = plain.rms_norm((x @ w[scale_name + "q"].T)[:, :m["dim"]], w[scale_name + "q.norm"], c["norm"]["eps"])
    k = plain.rms_norm((x @ w[scale_name + "k"].T)[:, :m["dim"]], w[scale_name + "k.norm"], c["norm"]["eps"])
    s = q @ k.T * m["scale"]
    asks, answers = divmod(int((s - s.mean(1, keepdim=True)).argmax()), s.shape[1])
    fill = [int(t) for t in s[asks].argsort()[:25] if int(t) not in (asks, answers)]
    return asks, answers, fill


def _sharp(dim, layer):
    """One layer whose scores are spread widely: one head, no rotation, no feed-forward."""
    layer["mixer"]["scale"] = 9.0 / dim
    layer["mixer"].pop("rot", None)
    return config([layer], width=32, bigram=None)


SCHEDULES = [(lambda ids: whole({"x": ids}), 16), (lambda ids: tail_decoded({"x": ids}, tail=200), 16),
             (lambda ids: portions({"x": ids}, [301, 2, 148, 70, 2, 200]), 8)]


@pytest.mark.parametrize("dim", [16, 64, 128])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_one_key_far_back_among_hundreds(tmp_path_factory, dtype, dim):
    """A key that one query scores far above all others, in the first tokens, at a page's last and first place, and just
    before the asking token; asked for from a prompt and by decoded tokens.  Without that key the plain model gives other
    rows."""
    entry = model(tmp_path_factory, f"far{dim}", _sharp(dim, att(heads=2, kv_heads=1, dim=dim, vdim=16, v_mix=False, mlp=None)))
    b, a, fill = _asking_pair(entry)
    g = torch.Generator().manual_seed(1)
    ids = [fill[int(i)] for i in torch.randint(0, len(fill), (640,), generator=g)]
    asks = {300: 0, 450: 15, 520: 16, 601: 600, 639: 319}                # asking place: where its key lies
    for p, j in asks.items():
        ids[p], ids[j] = b, a
    hidden = [j for j in range(640) if ids[j] == a]
    true_visible = plain.visible

    def blind(T, mask):
        ok = true_visible(T, mask)
        ok[:, hidden] = False
        ok[0, 0] = True
        return ok
    want, lost = plain_rows(entry, ids), _run_with(entry, ids, visible=blind)
    places = sorted(asks)
    gone = row_errors(lost, want)[places]
    assert float(gone.min()) > 0.15
    for steps, page in SCHEDULES:
        got = run_trace(entry[0], dtype, steps(ids), page_size=page)["x"]
        assert_close(got, want, dtype, "far", mean=0.04)
        assert (row_errors(got, want)[places] < 0.25 * gone).all()


@pytest.mark.parametrize("dim,size,keep", [(16, 44, 5), (64, 64, 16), (64, 129, 70), (128, 33, 1), (16, 100, 130)])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_keys_just_inside_and_outside_the_window_and_the_kept_first(tmp_path_factory, dtype, dim, size, keep):
    """Answering keys exactly at the window's last position and one before it, at the last kept position and one behind it, at
    the first position; asked for in prompts, by decoded tokens and at the start of portions.  The plain model with a window
    or a kept run one larger or one smaller gives other rows at exactly those places."""
    layer = att2(heads=2, kv_heads=1, dim=dim, vdim=16, size=size, keep_first=keep, cap=50.0, v_mix=False, mlp=None)

    def patch(t):
        t["l0.mix.sink"].fill_(-3.0)
    entry = model(tmp_path_factory, f"edge{dim}_{size}_{keep}", _sharp(dim, layer), patch=patch)
    b, a, fill = _asking_pair(entry)
    g = torch.Generator().manual_seed(2)
    n = 640
    base = [fill[int(i)] for i in torch.randint(0, len(fill), (n,), generator=g)]
    true_visible = plain.visible
    faults = {"window +1": (1, 0), "window -1": (-1, 0), "kept +1": (0, 1), "kept -1": (0, -1)}
    # fault -> (where the answering keys lie, the places that ask): each place asks for one key that the fault adds or hides
    edges = {"window +1": [(p - size, p) for p in (350, 463, 600) if p - size >= keep], "window -1": [(p - size + 1, p) for p in (351, 464, 601) if p - size + 1 >= keep],
             "kept +1": [(keep, p) for p in (380, 500, 630) if keep <= p - size], "kept -1": [(keep - 1, p) for p in (381, 501, 631)]}
    for fault, pairs in edges.items():
        ds, dk = faults[fault]
        if not pairs or size + ds < 1:
            continue
        ids = list(base)
        for j, p in pairs:
            ids[j] = a
            ids[p] = b
        places = sorted({p for _, p in pairs})
        want = plain_rows(entry, ids)
        wrong = _run_with(entry, ids, visible=lambda T, m: true_visible(T, {"size": m["size"] + ds, "keep_first": m["keep_first"] + dk}))
        moved = row_errors(wrong, want)[places]
        assert float(moved.min()) > 0.08, (fault, moved)
        for steps, page in (SCHEDULES[0], (lambda x: tail_decoded({"x": x}, tail=n - 340), 16), (lambda x: portions({"x": x}, [350, 30, 83, 37, 100, 2]), 8)):
            got = run_trace(entry[0], dtype, steps(ids), page_size=page)["x"]
            assert_close(got, want, dtype, fault, mean=0.04)
            assert (row_errors(got, want)[places] < 0.25 * moved).all(), (fault, row_errors(got, want)[places], moved)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_sink_the_cap_and_the_norm_before_the_rotation(tmp_path_factory, dtype):
    """Sinks as large as the keys' scores, a cap well below them, norm weights far from one: without any of them, with the sink
    capped or scaled, or with the norm taken behind the rotation, the plain model gives other rows, the first ones too."""
    layer = att2(heads=4, kv_heads=2, dim=16, vdim=16, size=50, keep_first=2, cap=1.5, scale=0.8, rot=(30.0, 12), v_mix=False, mlp=None)

    def patch(t):
        t["l0.mix.sink"][:] = torch.tensor([2.5, 3.0, 1.0, 4.0])
        t["l0.mix.q.norm"][:] = torch.linspace(0.2, 2.2, 16)
        t["l0.mix.k.norm"][:] = torch.linspace(1.8, 0.1, 16)
    entry = model(tmp_path_factory, "sink_cap", config([layer], width=32, bigram=None), patch=patch)
    ids = requests_for(entry, (160,), seed=5)["r0"]
    want = plain_rows(entry, ids)
    sm, rn, rt = plain.softmax_with_sink, plain.rms_norm, plain.rotate_halves
    turn = lambda x: rt(x, 30.0, 12) if x.dim() == 3 and x.shape[-1] == 16 else x
    back = lambda x: x if x.dim() == 3 and x.shape[-1] == 16 else x
    faults = {"no sink": dict(softmax_with_sink=lambda s, ok, sink=None: sm(s, ok)),
              "capped sink": dict(softmax_with_sink=lambda s, ok, sink=None: sm(s, ok, plain.soft_cap(sink, 1.5))),
              "no cap": dict(soft_cap=lambda s, cap: s),
              "norm behind the rotation": dict(rms_norm=lambda x, w, eps: rn(turn(x), w, eps), rotate_halves=lambda x, base, dims: back(x))}
    moved = {n: row_errors(_run_with(entry, ids, **f), want) for n, f in faults.items()}
    assert all(float(e[1:].mean()) > 0.03 for e in moved.values()), {n: float(e[1:].mean()) for n, e in moved.items()}
    least = min(float(e[1:].mean()) for e in moved.values())
    for steps in (whole({"x": ids}), tail_decoded({"x": ids}, tail=157), portions({"x": ids}, [2, 4, 1, 7, 20])):
        got = run_trace(entry[0], dtype, steps, page_size=8)["x"]
        assert_close(got, want, dtype, "sink")
        assert float(row_errors(got, want).mean()) < 0.3 * least


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_blended_values_are_those_of_the_first_such_layer_and_are_cached_blended(tmp_path_factory, dtype):
    """Large shares: the plain model that takes the layer before instead of the first one, the blended values instead of the
    raw ones, or caches unblended values gives other rows."""
    raw = config([att(v_mix=False, mlp=None), att(mlp=None), att2(size=9, mlp=None), att(dim=24, mlp=None)], width=40)

    def patch(t):
        for n in t:
            if n.endswith(".vmix"):
                t[n] = torch.tensor({"l2": 0.6, "l3": 0.8}.get(n[:2], 0.3))
    entry = model(tmp_path_factory, "shares", raw, patch=patch)
    ids = requests_for(entry, (90,), seed=6)["r0"]
    want = plain_rows(entry, ids)
    true_att = plain.attention
    last = {}

    def previous(w, p, m, a, eps, first_values=None):
        y, own = true_att(w, p, m, a, eps, last.get("v") if first_values is not None else None)
        if m.get("v_mix"):
            last["v"] = own
        return y, own
    moved = [row_errors(_run_with(entry, ids, attention=previous), want),
             row_errors(_run_with(entry, ids, blend_values=lambda v, first, share: v), want),
             row_errors(_run_with(entry, ids, blend_values=lambda v, first, share: share * v + (1 - share) * first), want)]
    assert all(float(e.mean()) > 0.1 for e in moved), [float(e.mean()) for e in moved]
    for steps in (whole({"x": ids}), tail_decoded({"x": ids}, tail=80), portions({"x": ids}, [2, 4, 1, 7, 20])):
        got = run_trace(entry[0], dtype, steps, page_size=8)["x"]
        assert_close(got, want, dtype, "blend")
        assert float(row_errors(got, want).mean()) < 0.2 * min(float(e.mean()) for e in moved)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_slot_taken_again_inherits_no_token_and_a_portion_knows_the_one_before(tmp_path_factory, dtype):
    """Requests one after the other through one slot, cut everywhere: a first token has the pair table's last row, every other
    one the row of itself and its predecessor, which may lie in an earlier step or stand behind a step left out."""
    entry = model(tmp_path_factory, "alone_pairs_of_tokens", ALONE["pairs_of_tokens"](), seed=7)
    reqs = requests_for(entry, (24, 13, 1, 8), seed=12)
    ids = reqs["r0"]
    rows = plain.pair_rows(ids, 29, 5, 3)
    fresh = plain.pair_rows
    wrong = _run_with(entry, ids, pair_rows=lambda x, *a: [29 if t % 6 == 0 else r for t, r in enumerate(fresh(x, *a))])
    assert rows[0] == 29 and float(row_errors(wrong, plain_rows(entry, ids))[6::6].min()) > 0.1
    compare(entry, dtype, portions(reqs, [6, 1, 1, 4]), reqs, max_reside=1)
    compare(entry, dtype, mixed(reqs, max_live=2, portion=5, decode_tail=3, seed=4), reqs, max_reside=2)
    joined = plain_rows(entry, reqs["r0"] + reqs["r1"])[24:]
    assert float(row_errors(joined, plain_rows(entry, reqs["r1"]))[0]) > 0.1                        # inheriting would show


@pytest.mark.parametrize("dtype,graph", [("float32", False), ("bfloat16", True)])
def test_long_decoding(tmp_path_factory, dtype, graph):
    """Up to 160 tokens decoded one by one behind a prompt of three; in bfloat16 through the captured graphs of generation."""
    entry = model(tmp_path_factory, "full", full_config())
    reqs = dict(zip("xyz", requests_for(entry, (163, 150, 20), seed=8).values()))
    steps = []
    for k in range(161):
        entries = [{"id": rid, "tokens": ids[:3] if k == 0 else [ids[2 + k]], "want": [2] if k == 0 else [0]}
                   for rid, ids in reqs.items() if 2 + k < len(ids)]
        ended = [rid for rid, ids in reqs.items() if 2 + k == len(ids) - 1]
        steps.append({"step": k, "entries": entries, "end": ended})
    got = run_trace(entry[0], dtype, steps, graph=graph)
    for rid, ids in reqs.items():
        assert_close(got[rid], plain_rows(entry, ids)[2:], dtype, rid, tied=close_calls(entry, ids)[2:])


def test_a_prompt_of_many_rows(tmp_path_factory):
    """A portion long enough for the tensor-core kernels of prompts, beside a short request, then a shorter portion
    behind the long cached prefix (its keys split over CTAs) beside a decoded token, then decoded tokens; in bfloat16 also
    through the graphs."""
    entry = model(tmp_path_factory, "wide", wide_config(), seed=5)
    reqs = requests_for(entry, (1200, 40), seed=33)
    a, b = reqs["r0"], reqs["r1"]
    steps = [{"step": 0, "entries": [{"id": "r1", "tokens": b[:20], "want": list(range(20))}], "end": []},
             {"step": 1, "entries": [{"id": "r0", "tokens": a[:1100], "want": [0, 500, 1099]},
                                      {"id": "r1", "tokens": b[20:21], "want": [0]}], "end": []},
             {"step": 2, "entries": [{"id": "r0", "tokens": a[1100:1190], "want": list(range(90))},
                                      {"id": "r1", "tokens": b[21:22], "want": [0]}], "end": []}]
    for k in range(10):
        steps.append({"step": 3 + k, "entries": [{"id": "r0", "tokens": [a[1190 + k]], "want": [0]},
                                                  {"id": "r1", "tokens": [b[22 + k]], "want": [0]}],
                      "end": ["r0", "r1"] if k == 9 else []})
    want0, want1 = plain_rows(entry, a)[[0, 500, 1099] + list(range(1100, 1200))], plain_rows(entry, b)[:32]
    for dtype, graph in (("bfloat16", False), ("float32", False), ("bfloat16", True)):
        got = run_trace(entry[0], dtype, steps, graph=graph)
        assert_close(got["r0"], want0, dtype, "long")
        assert_close(got["r1"], want1, dtype, "short")


# ------------------------------------------------------------------------------- generation through the engine

def _greedy_plain(entry, prompt, n):
    c, w = entry[1]
    ids = list(prompt)
    for _ in range(n):
        ids.append(int(plain.forward(c, w, ids)[-1].argmax()))
    return ids[len(prompt):]


@pytest.mark.parametrize("graph", [False, True])
def test_greedy_generation_through_the_scheduler(tmp_path_factory, graph):
    """Five prompts through three slots, portions of 24 beside decoded tokens: the scheduler admits, cuts, frees and
    hands slots on; the tokens are the plain model's."""
    from return_b200.engine.config import EngineConfig
    from return_b200.engine.engine import Engine
    entry = model(tmp_path_factory, "full", full_config())
    prompts = list(requests_for(entry, (5, 29, 1, 40, 12), seed=30).values())
    eng = Engine(entry[0], EngineConfig(max_token=512, max_reside=3, page_size=16, prefill_chunk=24, dtype="float32",
                                        use_cuda_graph=graph))
    got = eng.generate(prompts, max_new_tokens=10, temperature=0.0)
    assert [r.output_ids for r in got] == [_greedy_plain(entry, p, 10) for p in prompts]
    assert eng.runner.manager.pages_used() == [0] * len(eng.runner.manager.groups)


def test_bfloat16_generation_picks_tokens_the_plain_model_rates_highest(tmp_path_factory):
    """Every generated token is the plain model's best or within a rounding of it; two in 24 may miss that where a token before
    them went to another expert."""
    from return_b200.engine.config import EngineConfig
    from return_b200.engine.engine import Engine
    entry = model(tmp_path_factory, "full", full_config())
    c, w = entry[1]
    prompts = list(requests_for(entry, (7, 33, 20), seed=50).values())
    eng = Engine(entry[0], EngineConfig(max_token=512, max_reside=4, page_size=16, prefill_chunk=32, dtype="bfloat16"))
    missed = 0
    for p, r in zip(prompts, eng.generate(prompts, max_new_tokens=8, temperature=0.0)):
        lg, tied = plain.forward(c, w, p + r.output_ids), close_calls(entry, p + r.output_ids)
        for k, tok in enumerate(r.output_ids):
            row = lg[len(p) - 1 + k]
            missed += int(row[tok] < row.max() - 0.15 * row.std())
            assert tied[len(p) - 1 + k] or row[tok] >= row.max() - 0.5 * row.std(), (k, tok)
    assert missed <= 2


def test_command_line_generates_and_replays(tmp_path_factory):
    import subprocess
    import sys
    entry = model(tmp_path_factory, "full", full_config())
    prompt = requests_for(entry, (9,), seed=60)["r0"]
    out = subprocess.run([sys.executable, "-m", "return_b200", "generate", "--model", entry[0], "--prompt-ids",
                          ",".join(map(str, prompt)), "--new", "6", "--temperature", "0", "--dtype", "float32",
                          "--max-token", "256", "--max-reside", "2"], capture_output=True, text=True, timeout=600,
                         cwd=helpers.ROOT)
    assert out.returncode == 0, out.stderr[-2000:]
    assert json.loads(out.stdout.strip().splitlines()[0])["output_ids"] == _greedy_plain(entry, prompt, 6)
    lines = [{"step": 0, "entries": [{"id": "a", "tokens": [1, 2, 3], "want": [2]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": [4], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": [5, 6], "want": [0, 1]}], "end": ["a"]}]
    out = subprocess.run([sys.executable, os.path.join(helpers.ROOT, "bin", "trace_run"), "--model", entry[0], "--dtype",
                          "float32", "--out", os.path.join(entry[0], "out"), "--max-tokens", "64"],
                         input="".join(json.dumps(line) + "\n" for line in lines), capture_output=True, text=True, timeout=600)
    assert out.returncode == 0 and all(f"done {i}" in out.stdout for i in range(3)), out.stderr[-2000:]
    assert not os.path.exists(os.path.join(entry[0], "out", "1.f32"))
    want = plain_rows(entry, [1, 2, 3, 4, 5, 6])
    for step, rows in ((0, [2]), (2, [4, 5])):
        got = torch.frombuffer(bytearray(open(os.path.join(entry[0], "out", f"{step}.f32"), "rb").read()), dtype=torch.float32)
        assert float(row_errors(got.view(len(rows), -1), want[rows]).max()) < TOL["float32"]
