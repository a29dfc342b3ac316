"""The Losorax decoder through the engine against the plain implementation (tests/plain/losorax_plain.py).

Every test makes a small configuration of its own with random weights (written as a bfloat16 checkpoint, as a model
folder holds them), replays a trace through the engine's step function and compares every logits row with the plain
implementation's, which walks the whole sequence in float64, token by token where there is a recurrence.
float32 path: every row within 1e-4 of its size.  bfloat16 path: rows weighed together (see ``assert_close``).
Where random weights would hide a fault (a key far back among hundreds, a bias row that is one distance off, a state that
was lost) the scores are made sharp or the decays slow, and the test first shows that the plain model itself moves by far
more than the tolerance when that key, row or state is wrong.
"""
import copy
import json
import math
import os
import types

import pytest
import torch

import helpers
from helpers import collect, mixed, pool_tokens, portions, random_ids, tail_decoded, whole
from plain import losorax_plain as plain

pytestmark = pytest.mark.gpu

TOL = {"float32": 1e-4, "bfloat16": 1.0 / 12}


# ------------------------------------------------------------------------------- configurations

def dense(ff=56):
    return {"kind": "dense", "ff": ff}


def moe(experts=6, top=2, ff=24):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}


def att_layer(heads=4, kv_heads=2, dim=12, vdim=20, scale=None, conv=3, rows=10, reach=33, temp=(0.4, 16), kv_from=None, mlp="default"):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else 1.5 * dim ** -0.5,
         "conv": conv, "bias_rows": rows, "bias_max": reach}
    if temp:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": dense() if mlp == "default" else mlp}


def delta_layer(heads=3, dim=10, rank=6, mlp="default"):
    return {"type": "general_delta", "mixer": {"heads": heads, "dim": dim, "decay_rank": rank}, "mlp": moe() if mlp == "default" else mlp}


def config(layers, vocab=97, width=40, eps=1e-5):
    return {"architecture": "Losorax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


def full_config():
    """Both mixers and both feed-forwards, layers without a feed-forward, layers that read an earlier layer's keys (one of
    them the layer right behind, one with more heads and another filter), tables of several sizes."""
    return config([att_layer(), att_layer(heads=6, conv=4, rows=8, reach=50, kv_from=0, mlp=moe(5, 3, 16)), delta_layer(mlp=None),
                   att_layer(heads=2, kv_heads=1, dim=16, vdim=8, conv=2, rows=16, reach=90, temp=(0.2, 40), mlp=None),
                   delta_layer(heads=2, dim=16, rank=4, mlp=dense(33)),
                   att_layer(heads=3, kv_heads=1, dim=16, vdim=8, rows=6, reach=20, temp=None, kv_from=3, mlp=moe(4, 1, 32))])


def other_sizes_config():
    """The values one (one head, one key head, one tap, one expert of one, a rank of one, runs of one position, a head of
    one number in the delta rule), sizes that fill no whole vector, keys wider than values and the other way round, long
    filters, no filter, tables of two and of many rows, of an odd number of rows, as many experts chosen as there are."""
    return config([att_layer(heads=1, kv_heads=1, dim=7, vdim=33, conv=1, rows=2, reach=2, temp=(0.9, 1), mlp=moe(1, 1, 9)),
                   delta_layer(heads=1, dim=72, rank=1, mlp=dense(9)),
                   att_layer(heads=6, kv_heads=3, dim=24, vdim=8, conv=7, rows=40, reach=41, temp=(-0.05, 5), mlp=moe(3, 3, 8)),
                   att_layer(heads=9, kv_heads=3, dim=24, vdim=8, conv=5, rows=5, reach=300, temp=(0.1, 1000), kv_from=2, mlp=None),
                   delta_layer(heads=5, dim=1, rank=3, mlp=None),
                   att_layer(heads=2, kv_heads=2, dim=130, vdim=18, conv=0, rows=12, reach=17, temp=None, mlp=moe(33, 4, 7)),
                   delta_layer(heads=2, dim=33, rank=9, mlp=moe(2, 2, 40))], vocab=61, width=36, eps=1e-6)


def wide_config():
    """Sizes that pick the tensor-core kernels of prompts in bfloat16 (heads of 64 and 128, enough pairs for the grouped
    experts, enough rows for the woven gated product) and the 16-byte forms of the kernels around them."""
    return config([att_layer(heads=4, kv_heads=2, dim=64, vdim=48, conv=4, rows=32, reach=400, temp=(0.3, 256), mlp=moe(8, 2, 32)),
                   delta_layer(heads=2, dim=128, rank=16, mlp=dense(96)),
                   att_layer(heads=8, kv_heads=2, dim=64, vdim=48, conv=4, rows=16, reach=100, kv_from=0, mlp=moe(4, 2, 64)),
                   att_layer(heads=4, kv_heads=1, dim=128, vdim=128, conv=3, rows=24, reach=700, mlp=None)], width=64)


_MODELS = {}


def model(tmp_path_factory, name, raw, seed=3, patch=None):
    """(model folder, (config, float64 weights), memo of plain logits), cached: the plain walk is slow.  ``patch``
    changes tensors (name -> tensor) before they are written."""
    if name not in _MODELS:
        from return_b200.config.losorax_config import LosoraxConfig
        from return_b200.weights import loader
        from return_b200.weights.safetensors_io import write_safetensors
        d = str(tmp_path_factory.mktemp(name))
        loader.write_random_model(d, LosoraxConfig(raw), seed, torch.bfloat16)
        if patch is not None:
            tensors = plain.read_safetensors(os.path.join(d, "model.safetensors"))
            patch(tensors)
            write_safetensors(os.path.join(d, "model.safetensors"), [(n, t.bfloat16().contiguous()) for n, t in tensors.items()])
        _MODELS[name] = (d, plain.read_model(d), {})
    return _MODELS[name]


def plain_rows(entry, ids):
    d, (c, w), memo = entry
    key = tuple(ids)
    if key not in memo:
        memo[key] = plain.forward(c, w, list(ids)).float()
    return memo[key]


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


def assert_close(got, want, dtype, what="", mean=0.03, robust=False):
    """float32: every row within 1e-4 of its size.  bfloat16: rounding moves single rows far more than the rest (a router
    whose best candidates are nearly tied, a read-out near zero that is divided by its own size), so the rows are weighed
    together: their mean within 3 %, at most one row in ten (or two) beyond a twelfth, none beyond six tenths.  A lost key,
    a wrong bias, a stale page or a lost state moves every row behind it, and the tests that aim at single rows compare
    those rows with what the fault would give.  ``robust``: configurations drawn at random, where a single row may move by
    its own size but the middle row may not."""
    e = row_errors(got, want)
    if dtype == "float32":
        assert float(e.max()) < TOL[dtype], (what, dtype, float(e.max()), int(e.argmax()))
        return
    over = int((e > TOL[dtype]).sum())
    if robust:
        assert over <= max(2, e.numel() // 10) and float(e.median()) < mean, (what, dtype, over, float(e.max()), float(e.median()))
        return
    assert over <= max(2, e.numel() // 10) and float(e.max()) < 0.6 and float(e.mean()) < mean, \
        (what, dtype, over, float(e.max()), float(e.mean()), int(e.argmax()))


def compare(entry, dtype, steps, requests, robust=False, **kw):
    got = run_trace(entry[0], dtype, steps, **kw)
    for rid, ids in requests.items():
        assert_close(got[rid], plain_rows(entry, ids), dtype, rid, robust=robust)


# ------------------------------------------------------------------------------- kernels of single mechanisms

def _segments(lens, slots, pos0=None):
    cu = [0]
    for n in lens:
        cu.append(cu[-1] + n)
    tok_seg = [i for i, n in enumerate(lens) for _ in range(n)]
    pos0 = pos0 or [0] * len(lens)
    pos = [pos0[i] + k for i, n in enumerate(lens) for k in range(n)]
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
    return types.SimpleNamespace(cu_q=i32(cu), tok_seg=i32(tok_seg), seg_slot=i32(slots), pos=i32(pos), num_segments=len(lens),
                                 num_tokens=cu[-1], spans=[(cu[i], cu[i + 1]) for i in range(len(lens))])


# segments of a step: lengths, state slots, positions of their first tokens.  Short ones beside long ones, more tokens
# than a run of one thread or warp, and (the last) enough to make the kernels walk their longest runs.
STEPS = [([5], [1], [0]), ([1, 1, 1], [2, 0, 1], [0, 7, 90]), ([3, 1, 2, 70, 1, 4], [0, 1, 2, 3, 4, 5], [0, 3, 1, 15, 0, 40]),
         ([2100, 1, 2, 3, 900], [4, 3, 2, 1, 0], [31, 0, 2, 5, 0])]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("step", range(len(STEPS)))
@pytest.mark.parametrize("H", [36, 33, 640])
def test_joint_of_two_sublayers(H, step, dtype):
    """Add, squash and blend in every combination the blocks use, against the formulas; the kept rows of the step's
    requests are renewed and no other slot is touched."""
    from return_b200.ext import ops
    lens, slots, pos0 = STEPS[step]
    b = _segments(lens, slots, pos0)
    g = torch.Generator().manual_seed(H + step)
    rnd = lambda *s: torch.randn(s, generator=g)
    T = b.num_tokens
    x, y, mu = rnd(T, H), rnd(T, H), torch.rand(H, generator=g)
    post, nxt = (rnd(1).abs() + 0.3, rnd(H), rnd(H)), (rnd(1).abs() + 0.3, rnd(H), rnd(H))
    off, stride = 8, (H + 8 + 3) // 4 * 4
    kept = rnd(7, stride)
    sq = lambda v, p: torch.tanh(p[0].double() * v) * p[1].double() + p[2].double()
    xs = x.double() + sq(y.to(dtype).double(), post)
    h = sq(xs, nxt)
    want, want_kept = h.clone(), kept.double().clone()
    for (lo, hi), s in zip(b.spans, slots):
        before = torch.cat([kept[s:s + 1, off:off + H].double(), h[lo:hi - 1]], 0)
        want[lo:hi] = h[lo:hi] + (before - h[lo:hi]) * mu.double()
        want_kept[s, off:off + H] = h[hi - 1]
    dev = lambda t: t.cuda().contiguous()
    cx, cpost, cnxt, ck = dev(x), tuple(map(dev, post)), tuple(map(dev, nxt)), dev(kept)
    out, x_out = torch.empty((T, H), dtype=dtype, device="cuda"), torch.empty((T, H), device="cuda")
    tol = 2e-6 if dtype == torch.float32 else 3e-2
    ops.tanh_joint(cx, x_out, dev(y.to(dtype)), cpost, cnxt, out, shift=(dev(mu), ck, off), batch=b)
    assert (x_out.cpu().double() - xs).abs().max() < 4e-6 and (out.cpu().double() - want).abs().max() < tol * 6
    assert (ck.cpu().double() - want_kept).abs().max() < 4e-6
    # without a blend, in place, the output in float32
    ops.tanh_joint(cx, cx, dev(y.to(dtype)), cpost, cnxt, out)
    assert (cx.cpu().double() - xs).abs().max() < 4e-6 and (out.cpu().double() - h).abs().max() < tol * 6
    # nothing added; a raw sum without a squash; listed rows that leave the stream alone
    cx = dev(x)
    ops.tanh_joint(cx, None, None, None, cnxt, out)
    assert (out.cpu().double() - sq(x.double(), nxt)).abs().max() < tol * 6
    rows = torch.randint(0, T, (5,), generator=g)
    out5 = torch.empty((5, H), dtype=dtype, device="cuda")
    ops.tanh_joint(cx, None, dev(y), None, cnxt, out5, rows=rows.int().cuda())
    assert (out5.cpu().double() - sq(x.double() + y.double(), nxt)[rows]).abs().max() < tol * 6 and torch.equal(cx.cpu(), x)
    ops.tanh_joint(cx, cx, dev(y), None, None, None)
    assert (cx.cpu().double() - (x.double() + y.double())).abs().max() < 1e-6


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("step", range(len(STEPS)))
@pytest.mark.parametrize("Hq,G,dim,vdim,K,own", [(4, 2, 12, 20, 3, True), (3, 1, 64, 48, 4, True), (5, 1, 16, 8, 4, False),
                                                 (2, 2, 7, 33, 1, True), (9, 3, 128, 128, 4, True), (2, 1, 40, 24, 9, True),
                                                 (3, 3, 130, 18, 2, True)])
def test_rows_of_convolved_heads(Hq, G, dim, vdim, K, own, step, dtype):
    """Filters over tokens of this step and kept ones, head norms, temperature, padding, pages and the kept rows afterwards."""
    from return_b200.ext import ops
    lens, slots, pos0 = STEPS[step]
    b = _segments(lens, slots, pos0)
    T, page = b.num_tokens, 8
    D = (max(dim, vdim) + 15) // 16 * 16
    C = Hq * dim + (G * (dim + vdim) if own else 0)
    g = torch.Generator().manual_seed(1000 * step + dim + K)
    rnd = lambda *s: torch.randn(s, generator=g)
    proj, taps = rnd(T, C).to(dtype), rnd(C, K) * 0.6
    kept = torch.zeros(7, (K - 1) * C + 12)
    kept[:, 4:4 + (K - 1) * C] = rnd(7, (K - 1) * C).to(dtype).float()
    blocks = max((p + n + page - 1) // page for n, p in zip(lens, pos0))
    table = torch.randperm(len(lens) * blocks, generator=g).view(len(lens), blocks).int()
    pool = lambda: torch.full((len(lens) * blocks, G, page, D), 9.0, dtype=dtype, device="cuda")
    kv = types.SimpleNamespace(k=pool(), v=pool(), block_table=table.cuda(), page_size=page)
    q = torch.empty((T, Hq * D), dtype=dtype, device="cuda")
    eps, temp = 1e-3, (0.7, 12)
    ck = kept.cuda()
    ops.attention_conv_prepare(proj.cuda(), taps.t().contiguous().cuda(), ck if K > 1 else None, 4, b, kv, q, Hq, G, dim, vdim, D, eps,
                               temp, own_kv=own, write_kv=own)
    tol = 3e-5 if dtype == torch.float32 else 3e-2
    q, kk, vv, ck = q.cpu().double().view(T, Hq, D), kv.k.cpu().double(), kv.v.cpu().double(), ck.cpu()
    for i, ((lo, hi), s, p0) in enumerate(zip(b.spans, slots, pos0)):
        before = kept[s, 4:4 + (K - 1) * C].view(K - 1, C).double()
        seen = torch.cat([before, proj[lo:hi].double()], 0)
        y = sum(seen[j:j + hi - lo] * taps[:, j].double() for j in range(K))
        if K > 1:
            assert torch.equal(ck[s, 4:4 + (K - 1) * C].view(K - 1, C).double(), seen[-(K - 1):])
        f = plain.temperature(p0 + hi - lo, *temp, torch.float64)[p0:, None, None]
        wq = plain.rms(y[:, :Hq * dim].view(-1, Hq, dim), eps) * f
        assert (q[lo:hi, :, :dim] - wq).abs().max() < tol * max(1.0, float(wq.abs().max())) and (q[lo:hi, :, dim:] == 0).all()
        if not own:
            continue
        wk = plain.rms(y[:, Hq * dim:(Hq + G) * dim].view(-1, G, dim), eps)
        wv = y[:, (Hq + G) * dim:].view(-1, G, vdim)
        pos = torch.arange(p0, p0 + hi - lo)
        pages = table[i, pos // page].long()
        gk, gv = kk[pages, :, pos % page], vv[pages, :, pos % page]
        assert (gk[..., :dim] - wk).abs().max() < tol * float(wk.abs().max()) and (gk[..., dim:] == 0).all()
        assert (gv[..., :vdim] - wv).abs().max() < tol * float(wv.abs().max()) and (gv[..., vdim:] == 0).all()
        kk[pages, :, pos % page], vv[pages, :, pos % page] = 9.0, 9.0
    assert (kk == 9.0).all() and (vv == 9.0).all()                          # nothing else was written
    untouched = [s for s in range(7) if s not in slots]
    assert torch.equal(ck[untouched], kept[untouched]) and torch.equal(ck[:, :4], kept[:, :4])


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,D,rank", [(3, 10, 6), (2, 16, 8), (1, 72, 1), (5, 1, 3), (2, 33, 9), (2, 128, 16), (1, 200, 5), (4, 64, 24)])
def test_general_delta_kernels(H, D, rank, dtype):
    """Preparation and scan over a sequence cut into three steps beside another request, against the plain recurrence from
    the projections on; the other slots stay as they are."""
    from return_b200.ext import ops
    g = torch.Generator().manual_seed(D + H)
    HD, T = H * D, 43
    rnd = lambda *s: torch.randn(s, generator=g)
    proj, low = rnd(T, 5 * HD + rank).to(dtype), rnd(T, HD)
    bias, w0 = rnd(HD) * 0.5, rnd(HD) - 1.0
    c = math.exp(-0.5)
    r, k, v, a = (proj.double()[:, i * HD:(i + 1) * HD].view(T, H, D) for i in (0, 1, 2, 4))
    decay = torch.exp(-c * torch.sigmoid(low.double() + w0.double())).view(T, H, D)
    rate = torch.sigmoid(a + bias.double().view(H, D))
    u = k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)
    M, want = torch.zeros(H, D, D, dtype=torch.float64), []
    for t in range(T):
        held = torch.einsum("hi,hij->hj", u[t], M)
        M = decay[t][:, :, None] * M - (rate[t] * u[t])[:, :, None] * held[:, None, :] + k[t][:, :, None] * v[t][:, None, :]
        want.append(torch.einsum("hij,hi->hj", M, r[t]).reshape(HD))
    want = torch.stack(want)
    DR = (D + 3) // 4 * 4
    state = torch.full((3, H * D * DR + 8), 7.0, device="cuda")
    state[1, 4:4 + H * D * DR] = 0.0
    state[2, 4:4 + H * D * DR] = 0.0
    got = []
    for lo, hi in ((0, 1), (1, 21), (21, T)):
        n = hi - lo
        b = _segments([2, n], [2, 1], [0, lo])
        x = torch.cat([proj[:2], proj[lo:hi]], 0).cuda()
        dec = torch.cat([low[:2], low[lo:hi]], 0).cuda()
        rem = torch.empty_like(dec)
        ops.general_delta_prep(x, HD, 4 * HD, bias.cuda(), w0.cuda(), c, 1e-6, dec, rem, H, D)
        out = torch.empty((n + 2, HD), device="cuda")
        ops.general_delta_scan(x, x[:, HD:], x[:, 2 * HD:], dec, rem, state, 4, b, out, H, D)
        got.append(out[2:].cpu().double())
    got = torch.cat(got)
    assert ((got - want).abs().amax(1) / want.abs().amax(1).clamp(min=1.0)).max() < 2e-5
    S = state[1, 4:4 + H * D * DR].view(H, D, DR).cpu().double()
    assert (S[:, :, :D].transpose(1, 2) - M).abs().max() < 2e-5 * max(1.0, float(M.abs().max())) and (S[:, :, D:] == 0).all()
    assert (state[0] == 7.0).all() and (state[1, :4] == 7.0).all() and (state[1, 4 + H * D * DR:] == 7.0).all()


@pytest.mark.parametrize("E,top", [(15, 2), (6, 6), (35, 4), (1, 1)])
def test_scores_taken_as_they_are(E, top):
    from return_b200.ext import ops
    g = torch.Generator().manual_seed(E * 7 + top)
    z = torch.randn((50, E), generator=g) * 2.0
    picked, weight = plain.route(z.double(), top)
    expert_of = torch.empty((50, top), dtype=torch.int32, device="cuda")
    got = torch.empty((50, top), dtype=torch.float32, device="cuda")
    ops.moe_route(z.cuda(), expert_of, got, top, score="sigmoid", renorm=False)
    assert torch.equal(expert_of.cpu().long(), picked) and (got.cpu().double() - weight).abs().max() < 1e-6


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,E,top,F,H", [(5, 6, 2, 24, 40), (9, 3, 3, 7, 36), (90, 8, 1, 32, 64), (700, 8, 2, 32, 64)])
def test_weights_on_the_experts_input(T, E, top, F, H, dtype):
    """sum_k expert(weight * x) on every path of the experts (single pairs, grouped tiles, tcgen05 tiles).  The weights are
    small, so an expert that weighed its output instead would be far off: silu(w g) (w u) is not w silu(g) u."""
    from return_b200.ext import ops
    g = torch.Generator().manual_seed(T + E)
    rnd = lambda *s: torch.randn(s, generator=g)
    x, gu, down = rnd(T, H).to(dtype), (rnd(E, 2 * F, H) * H ** -0.5).to(dtype), (rnd(E, H, F) * F ** -0.5).to(dtype)
    expert_of = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(T)])
    weight = torch.rand((T, top), generator=g) * 0.5 + 0.1
    want, wrong = torch.zeros(T, H, dtype=torch.float64), torch.zeros(T, H, dtype=torch.float64)
    for k in range(top):
        W1, W2, c = gu.double()[expert_of[:, k]], down.double()[expert_of[:, k]], weight[:, k:k + 1].double()
        run = lambda v: torch.einsum("thf,tf->th", W2, torch.nn.functional.silu((p := torch.einsum("tfh,th->tf", W1, v))[:, :F]) * p[:, F:])
        want += run(c * x.double())
        wrong += c * run(x.double())
    out = torch.empty((T, H), dtype=dtype, device="cuda")
    ops.moe_experts(x.cuda(), gu.cuda(), down.cuda(), expert_of.int().cuda().contiguous(), weight.cuda(), None, out, float("inf"), 1.0,
                    shift=0.0, weigh_input=True)
    err = (out.cpu().double() - want).norm() / want.norm()
    assert err < (2e-6 if dtype == torch.float32 else 1e-2) and (wrong - want).norm() / want.norm() > 0.3
    ops.check_status(torch.device("cuda:0"))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_sandwich_of_rms_norms_takes_scales_and_a_blend(dtype):
    """The options of the sandwich block with RMSNorms (whose joints are other kernels): two blocks of a plain mixer in a
    row, a sequence cut in two steps."""
    from return_b200.parts.base import MIXERS, BuildEnv, LayerContext, Mixer
    from return_b200.parts.block import SandwichBlock
    from return_b200.parts.spec import NormSpec, SandwichBlockSpec

    class Doubling(Mixer):
        def forward(self, x, ctx):
            return (x * 2.0).contiguous()
    MIXERS.register("doubling", Doubling)
    try:
        H, T, eps, g = 40, 11, 1e-5, torch.Generator().manual_seed(5)
        spec = SandwichBlockSpec(types.SimpleNamespace(kind="doubling"), None, NormSpec(H, eps), NormSpec(H, eps), layer_scale=True, token_shift=True)
        env = BuildEnv(dtype, torch.device("cuda:0"))
        blocks, ws = [], []
        for _ in range(2):
            blk = SandwichBlock(spec, env)
            w = {n: torch.rand(p.shape, generator=g) + 0.2 for n, p in blk.params().items()}
            assert set(w) == {"mixer_norm.weight", "mixer_post_norm.weight", "mixer_scale", "shift"}
            blk.bind({n: t.cuda() for n, t in w.items()})
            blocks.append(blk)
            ws.append({n: t.double() for n, t in w.items()})
        x = torch.randn((T, H), generator=g)
        want = x.double()
        for w in ws:
            a = plain.blend_with_previous(plain.rms(want, eps) * w["mixer_norm.weight"], w["shift"])
            want = want + plain.rms(2.0 * a, eps) * w["mixer_post_norm.weight"] * w["mixer_scale"]
        kept = [torch.zeros((2,) + blk.kept_need().shape, device="cuda") for blk in blocks]
        got = []
        for lo, hi in ((0, 4), (4, T)):
            b = _segments([hi - lo], [1], [lo])
            b.scratch = {}
            stream = x[lo:hi].cuda()
            for i, blk in enumerate(blocks):
                ctx = LayerContext(batch=b, kept=kept[i], position=i, next_block=blocks[1] if i == 0 else None)
                assert blk.forward(stream, None, ctx) is None
            got.append(stream.cpu().double())
        err = (torch.cat(got) - want).norm() / want.norm()
        assert err < (1e-6 if dtype == torch.float32 else 1e-2)
    finally:
        MIXERS.unregister("doubling")


# ------------------------------------------------------------------------------- each mechanism alone, as a small model

ALONE = {
    "attention": lambda: config([att_layer(mlp=None)]),
    "attention_without_options": lambda: config([att_layer(conv=0, temp=None, mlp=None)]),
    "shared_keys": lambda: config([att_layer(mlp=None), att_layer(heads=2, conv=4, kv_from=0, mlp=None)]),
    "general_delta": lambda: config([delta_layer(mlp=None)]),
    "gated_unit": lambda: config([delta_layer(mlp=dense(48))]),
    "experts": lambda: config([delta_layer(mlp=moe(10, 3, 16))]),
}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(ALONE))
def test_each_mechanism_alone(tmp_path_factory, name, dtype):
    """A model of one layer (two where a layer reads another's keys): whole prompts, prompts against token-by-token
    decoding, and portions down to single first tokens."""
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


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_many_query_heads_on_one_key_head(tmp_path_factory, dtype):
    """Twenty and thirty-six query heads a key head: the decode kernel packs a key head's query heads into tiles of 16
    rows, and every row keeps its own head's bias."""
    raw = config([att_layer(heads=20, kv_heads=1, dim=16, vdim=16, mlp=None), delta_layer(heads=4, dim=8),
                  att_layer(heads=36, kv_heads=1, dim=16, vdim=16, rows=7, reach=60, kv_from=0, mlp=dense(24))], width=48)
    entry = model(tmp_path_factory, "many_heads", raw, seed=9)
    reqs = requests_for(entry, (70, 33), seed=44)
    compare(entry, dtype, tail_decoded(reqs, tail=45), reqs, page_size=8)
    compare(entry, dtype, mixed(reqs, max_live=2, portion=9, decode_tail=20, seed=7), reqs, page_size=4, max_reside=2)


def _random_config(rng):
    """A configuration no fixed case has: two to five layers of random kinds and sizes, later attentions reading an earlier
    one's keys."""
    layers, owners = [], []                                    # owners: (layer, kv_heads, dim, vdim) of attentions with keys
    for i in range(rng.randint(2, 5)):
        mlp = rng.choice([None, dense(rng.choice([7, 24, 40])), moe(*rng.choice([(4, 1, 16), (6, 2, 8), (9, 3, 12), (5, 5, 8), (16, 4, 8)]))])
        if rng.random() < 0.35:
            layers.append(delta_layer(rng.choice([1, 2, 3, 5]), rng.choice([3, 8, 12, 16, 33, 65]), rng.choice([1, 3, 8, 20]), mlp))
            continue
        rows = rng.choice([2, 4, 7, 16, 30])
        opts = dict(conv=rng.randint(0, 6), rows=rows, reach=rng.choice([rows // 2 + 1, rows, 3 * rows, 500]), mlp=mlp,
                    temp=rng.choice([None, (0.3, 1), (0.5, 17), (-0.1, 8)]))
        if owners and rng.random() < 0.5:
            src, kv, dim, vdim = rng.choice(owners)
            layers.append(att_layer(kv * rng.choice([1, 2, 4]), kv, dim, vdim, kv_from=src, **opts))
        else:
            kv, dim, vdim = rng.choice([1, 2, 3]), rng.choice([7, 8, 16, 20, 48]), rng.choice([5, 8, 16, 24, 40])
            owners.append((i, kv, dim, vdim))
            layers.append(att_layer(kv * rng.choice([1, 2, 3, 5]), kv, dim, vdim, **opts))
    return config(layers, vocab=rng.randint(30, 200), width=rng.choice([24, 33, 36, 40, 56, 64]), eps=rng.choice([1e-6, 1e-5, 1e-3]))


@pytest.mark.parametrize("seed", list(range(12)))
def test_random_configurations_and_traces(tmp_path_factory, seed):
    import random
    rng = random.Random(900 + seed)
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


# ------------------------------------------------------------------------------- far keys, bias rows, states, slots

def _by_token_alone(tensors):
    """No blend and filters of the token itself: a token's query and key then depend on the token alone."""
    for name, t in tensors.items():
        if name.endswith(".shift"):
            t.zero_()
        if name.endswith(".conv"):
            t.zero_()
            t[:, -1] = 1.0


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


@pytest.mark.parametrize("dim", [16, 64, 128])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_one_key_far_back_among_hundreds(tmp_path_factory, dtype, dim):
    """A key that one query scores far above all others, in the first tokens, at a page's last and first place, and just
    before the asking token; asked for from a prompt and by decoded tokens.  Without that key the plain model gives other
    rows."""
    raw = config([att_layer(heads=2, kv_heads=1, dim=dim, vdim=16, scale=9.0 / dim, rows=8, reach=600, mlp=None)], width=32)

    def patch(t):
        _by_token_alone(t)
        t["l0.mix.rel"] *= 0.2
    entry = model(tmp_path_factory, f"far{dim}", raw, patch=patch)
    c, w = entry[1]
    h = plain.tanh_norm(w, "l0.norm1", w["embed"])
    q, k = plain.rms((h @ w["l0.mix.q"].T)[:, :dim], 1e-5), plain.rms(h @ w["l0.mix.k"].T, 1e-5)
    s = q @ k.T * 9.0 / dim
    b, a = divmod(int((s - s.mean(1, keepdim=True)).argmax()), s.shape[1])
    fill = [int(x) for x in s[b].argsort()[:25] if int(x) not in (a, b)]
    g = torch.Generator().manual_seed(1)
    ids = [fill[int(i)] for i in torch.randint(0, len(fill), (640,), generator=g)]
    asks = {300: 0, 450: 15, 520: 16, 601: 600, 639: 319}                # asking place: where its key lies
    for p, j in asks.items():
        ids[p], ids[j] = b, a
    # the rows of one asking place with every answering key before it hidden from it
    true_softmax = plain.softmax_plus_one
    hidden = [j for j in range(640) if ids[j] == a]

    def blind(s, ok):
        ok = ok.clone()
        ok[:, hidden] = False
        return true_softmax(s, ok)
    want, lost = plain_rows(entry, ids), _run_with(entry, ids, softmax_plus_one=blind)
    places = sorted(asks)
    gone = row_errors(lost, want)[places]
    assert float(gone.min()) > 0.15
    for steps, page in ((whole({"x": ids}), 16), (tail_decoded({"x": ids}, tail=200), 16), (portions({"x": ids}, [301, 2, 148, 70, 2, 200]), 8)):
        got = run_trace(entry[0], dtype, steps, page_size=page)["x"]
        assert_close(got, want, dtype, "far", mean=0.04)
        assert (row_errors(got, want)[places] < 0.25 * gone).all()


@pytest.mark.parametrize("dim", [16, 64, 128])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_bias_rows_change_at_the_right_distance(tmp_path_factory, dtype, dim):
    """Bias rows far apart, so that a key one distance off its row shows: the plain model with every distance taken one too
    large, or one too small, gives other rows.  The table reaches 150 positions: rows of one distance, rows of many,
    behind them the last row; prompts, decoded tokens (over splits of the keys), portions that begin at a row's edge."""
    raw = config([att_layer(heads=4, kv_heads=2, dim=dim, vdim=16, scale=0.5 / dim, rows=12, reach=150, mlp=None)], width=32)

    def patch(t):
        _by_token_alone(t)
        t["l0.mix.rel"][:] = torch.where(torch.arange(12)[:, None] % 2 == torch.arange(4)[None] % 2, 1.5, -3.5)
        t["l0.ls1"].fill_(3.0)
    entry = model(tmp_path_factory, f"bias{dim}", raw, patch=patch)
    ids = requests_for(entry, (420,), seed=3)["r0"]
    true_bucket = plain.bucket
    want = plain_rows(entry, ids)
    off = [row_errors(_run_with(entry, ids, bucket=lambda n, *a, by=by: true_bucket(max(0, n + by), *a)), want) for by in (1, -1)]
    assert min(float(e[20:].mean()) for e in off) > 0.04
    for steps, page in ((whole({"x": ids}), 16), (tail_decoded({"x": ids}, tail=90), 16), (portions({"x": ids}, [6, 2, 5, 151, 20, 236]), 8)):
        got = run_trace(entry[0], dtype, steps, page_size=page)["x"]
        assert_close(got, want, dtype, "bias", mean=0.04)
        assert float(row_errors(got, want)[20:].mean()) < 0.25 * min(float(e[20:].mean()) for e in off)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_one_below_the_softmax_and_the_temperature(tmp_path_factory, dtype):
    """Scores pushed down by the bias so that the one in the denominator weighs as much as the keys, most of all for the first
    tokens, and a temperature that steps every seven positions: without either, or with the steps one position late, the
    plain model gives other rows."""
    raw = config([att_layer(heads=2, kv_heads=1, dim=16, vdim=16, scale=0.3, rows=4, reach=9, temp=(0.8, 7), mlp=None)], width=32)

    def patch(t):
        t["l0.mix.rel"] -= 5.0
        t["l0.ls1"].fill_(3.0)
        t["l0.norm1b.alpha"].fill_(3.0)
    entry = model(tmp_path_factory, "sink", raw, patch=patch)
    ids = requests_for(entry, (120,), seed=5)["r0"]
    want = plain_rows(entry, ids)
    no_sink = row_errors(_run_with(entry, ids, softmax_plus_one=lambda s, ok: torch.softmax(s.masked_fill(~ok, float("-inf")), -1)), want)
    true_temp = plain.temperature
    cold = row_errors(_run_with(entry, ids, temperature=lambda T, c, e, d: torch.ones(T, dtype=d)), want)
    late = row_errors(_run_with(entry, ids, temperature=lambda T, c, e, d: torch.cat([torch.ones(1, dtype=d), true_temp(T, c, e, d)[:-1]])), want)
    steps_at = [p for p in range(6, 120, 7)]
    assert float(no_sink.mean()) > 0.1 and float(no_sink[:3].min()) > 0.1 and float(cold[10:].mean()) > 0.1
    assert float(late[steps_at[:4]].mean()) > 0.012 and float(late[7:13].max()) == 0.0
    for steps in (whole({"x": ids}), tail_decoded({"x": ids}, tail=117), portions({"x": ids}, [2, 4, 1, 7, 20])):
        got = run_trace(entry[0], dtype, steps, page_size=8)["x"]
        assert_close(got, want, dtype, "sink")
        e = row_errors(got, want)
        assert float(e.mean()) < 0.2 * float(no_sink.mean()) and float(e[:3].max()) < 0.2 * float(no_sink[:3].min())
        if dtype == "float32":
            assert float(e[steps_at[:4]].mean()) < 0.01 * float(late[steps_at[:4]].mean())


def _slow_decays(tensors):
    """States that hardly forget and hardly remove: what a request saw far back still shows at its end."""
    for name, t in tensors.items():
        if name.endswith("mix.w0"):
            t.fill_(-8.0)
        if name.endswith("mix.a.b"):
            t.fill_(-6.0)


def states_config():
    return config([delta_layer(heads=2, dim=16, mlp=None), delta_layer(heads=3, dim=12, mlp=None)], width=32)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_states_far_back(tmp_path_factory, dtype):
    """With slow decays the last rows lean on the first two hundred tokens: without them the plain model gives other rows."""
    entry = model(tmp_path_factory, "slow_states", states_config(), patch=_slow_decays)
    ids = requests_for(entry, (330,), seed=6)["r0"]
    want = plain_rows(entry, ids)
    lost = row_errors(plain.forward(*entry[1], ids[200:]).float()[-20:], want[-20:])
    assert float(lost.mean()) > 0.08
    reqs = {"far": ids}
    for steps, page in ((tail_decoded(reqs, tail=36), 16), (portions(reqs, [250, 6, 10, 2, 62]), 8)):
        got = run_trace(entry[0], dtype, steps, page_size=page)["far"]
        assert_close(got, want, dtype, "far", mean=0.06)
        assert float(row_errors(got[-20:], want[-20:]).mean()) < 0.25 * float(lost.mean())


@pytest.mark.parametrize("kind", ["states", "attention"])
def test_a_slot_taken_again_inherits_nothing(tmp_path_factory, kind):
    """Two requests one after the other through one slot: the second starts from zero states, zero filter inputs and nothing
    to blend its first row with (the plain walk of the second alone)."""
    if kind == "states":
        entry = model(tmp_path_factory, "slow_states", states_config(), patch=_slow_decays)
    else:
        entry = model(tmp_path_factory, "alone_shared_keys", ALONE["shared_keys"](), seed=7)
    reqs = requests_for(entry, (50, 30), seed=12)
    for dtype in ("float32", "bfloat16"):
        compare(entry, dtype, portions(reqs, [7, 1, 20]), reqs, max_reside=1)
        compare(entry, dtype, tail_decoded(reqs, tail=29), reqs, max_reside=1)
    joined = plain_rows(entry, reqs["r0"] + reqs["r1"])[50:]
    assert float(row_errors(joined, plain_rows(entry, reqs["r1"]))[:3].mean()) > 0.08                # inheriting would show


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
        assert_close(got[rid], plain_rows(entry, ids)[2:], dtype, rid)


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
    from return_b200.engine.config import EngineConfig
    from return_b200.engine.engine import Engine
    entry = model(tmp_path_factory, "full", full_config())
    c, w = entry[1]
    prompts = list(requests_for(entry, (7, 33, 20), seed=50).values())
    eng = Engine(entry[0], EngineConfig(max_token=512, max_reside=4, page_size=16, prefill_chunk=32, dtype="bfloat16"))
    for p, r in zip(prompts, eng.generate(prompts, max_new_tokens=8, temperature=0.0)):
        lg = plain.forward(c, w, p + r.output_ids)
        for k, tok in enumerate(r.output_ids):
            row = lg[len(p) - 1 + k]
            assert row[tok] >= row.max() - 0.15 * row.std(), (k, tok)


def test_command_line_generates_and_replays(tmp_path_factory):
    import subprocess
    import sys
    raw = full_config()
    entry = model(tmp_path_factory, "full", raw)
    path = os.path.join(entry[0], "config.json")                  # as a model folder has it: sizes that tensors give are absent
    bare = copy.deepcopy(entry[1][0])
    for layer in bare["layers"]:
        layer["mixer"].pop("bias_rows", None)
        layer["mixer"].pop("decay_rank", None)
    with open(path, "w") as f:
        json.dump(bare, f)
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
                         input="".join(json.dumps(l) + "\n" for l in lines), capture_output=True, text=True, timeout=600)
    assert out.returncode == 0 and all(f"done {i}" in out.stdout for i in range(3)), out.stderr[-2000:]
    assert not os.path.exists(os.path.join(entry[0], "out", "1.f32"))
    want = plain_rows(entry, [1, 2, 3, 4, 5, 6])
    for step, rows in ((0, [2]), (2, [4, 5])):
        got = torch.frombuffer(bytearray(open(os.path.join(entry[0], "out", f"{step}.f32"), "rb").read()), dtype=torch.float32)
        assert float(row_errors(got.view(len(rows), -1), want[rows]).max()) < TOL["float32"]
