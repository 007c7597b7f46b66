"""Sonalix on the GPU against the plain restatement in tests/sonalix_ref.py: each mechanism alone (as a kernel and as a
one-layer model), whole prompts against token-by-token decoding, portions down to two tokens, unequal batches against
each request alone, pages and slots that are used again, keys far back, at page borders and just inside / just outside
the window with inputs made so that one key stands out, routers whose bias decides, values mixed with an earlier
layer's, the first tokens of a sequence, long decoding, several sizes (also sizes of one), and greedy generation through
LLMEngine.  fp32 runs are held to 2e-4 of the logits' spread, bf16 runs to 6e-2; models with routed experts are compared at
the 0.9 quantile of their rows in bf16, where 16-bit operands can flip a near-tied expert choice at single rows."""
import json
import struct
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

import sonalix_ref as R
from fidasun_util import Driver, rel_err
from sonalix_util import dense_cfg, full_cfg, layer, make_cfg, moe_cfg, random_layers, random_tensors
from zalalix_util import random_schedule

pytestmark = pytest.mark.gpu
F32_TOL, BF16_TOL = 2e-4, 6e-2
D64 = torch.float64


def ref_logits(cfg, tensors, tokens):
    return R.forward(cfg, tensors, tokens).numpy()


def toks(n, vocab, seed):
    return np.random.default_rng(seed).integers(0, vocab, size=n).tolist()


def _i32(a):
    return torch.tensor(a, dtype=torch.int32, device="cuda")


def bounds(dtype, routed=True):
    """(tolerance, quantile of the rows it applies to)."""
    if dtype == torch.float32:
        return F32_TOL, 1.0
    return BF16_TOL, 0.9 if routed else 1.0


def frequencies(dims, base):
    return torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=D64)


def halves_from_pairs(n, dims):
    """x[..., these] lays the interleaved pairs among the first `dims` of n entries out as two halves."""
    return torch.tensor(list(range(0, dims, 2)) + list(range(1, dims, 2)) + list(range(dims, n)))


def turned_at(x, pos, dims, base):
    """R.turn at listed positions: x [T, heads, d]."""
    rows = []
    for t, p in enumerate(pos):
        long = torch.zeros(p + 1, *x.shape[1:], dtype=D64)
        long[p] = x[t]
        rows.append(R.turn(long, dims, base)[p])
    return torch.stack(rows)


# ------------------------------------------------------------------ row kernels
@pytest.mark.parametrize("heads,dim,dims", [(4, 24, 12), (1, 2, 2), (3, 130, 128), (10, 7, 0), (2, 64, 64), (40, 33, 30)])
def test_rotary_rows_op(lib, heads, dim, dims):
    """Both pair layouts, a factor on cos and sin, entries past the rotated part and past the last head untouched."""
    from vllm_rs_b200 import ops
    g = torch.Generator().manual_seed(heads * dim)
    pos = [0, 1, 63, 64, 1500]
    x = torch.randn(len(pos), heads * dim + 3, generator=g)
    f = frequencies(dims, 500.0) if dims else torch.zeros(0, dtype=D64)
    at = torch.tensor(pos).cuda()
    half = ops.rotary_rows(x.cuda(), f.cuda(), at, heads=heads, dim=dim).cpu().double()
    want = turned_at(x.double()[:, :-3].view(len(pos), heads, dim), pos, dims, 500.0).reshape(len(pos), -1)
    assert torch.equal(half[:, -3:], x.double()[:, -3:])
    assert torch.allclose(half[:, :-3], want, atol=1e-5)
    inter = ops.rotary_rows(x.cuda(), f.cuda(), at, heads=heads, dim=dim, rot_half=False, rot_mag=1.5).cpu().double()
    perm = halves_from_pairs(dim, dims)
    y = x.double()[:, :-3].view(len(pos), heads, dim)[..., perm]
    y = turned_at(y, pos, dims, 500.0)
    y[..., :dims] *= 1.5
    want = torch.empty_like(y)
    want[..., perm] = y
    assert torch.allclose(inter[:, :-3], want.reshape(len(pos), -1), atol=2e-5)


@pytest.mark.parametrize("n,ld", [(5, 5), (40, 43), (64, 64), (2048, 2052), (1, 9)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_gate_rows_and_rmsnorm_rows_ops(lib, n, ld, dtype):
    from vllm_rs_b200 import ops
    g = torch.Generator().manual_seed(n)
    tol = 2e-6 if dtype == torch.float32 else 1e-2
    x, gate, w = torch.randn(9, n, generator=g), torch.randn(9, ld, generator=g) * 3, torch.randn(n, generator=g)
    out = ops.gate_rows(x.cuda(), gate.cuda(), dtype).cpu().double()
    want = x.double() * torch.sigmoid(gate.double()[:, :n])
    assert (out - want).abs().max() <= tol * max(1.0, want.abs().max().item())
    out = ops.rmsnorm_rows(gate.cuda(), n, w.cuda(), 1e-2, 0.0, dtype).cpu().double()
    want = R.unit_rms(gate.double()[:, :n], 1e-2) * w.double()
    assert (out - want).abs().max() <= 2 * tol * max(1.0, want.abs().max().item())


@pytest.mark.parametrize("D", [40, 33, 2048])
def test_norm_that_takes_over_the_experts_sum(lib, D):
    """One stream: x += the weighed expert rows, then the dynamic-tanh norm, in one pass -- all rows, and listed rows only."""
    from vllm_rs_b200 import ops
    g = torch.Generator().manual_seed(D)
    T, top = 6, 3
    rnd = lambda *s: torch.randn(*s, generator=g)                     # noqa: E731
    x, rows, w, b, wt = rnd(1, T, D), rnd(T * top, D), rnd(D), rnd(D), rnd(T, top)
    slot = torch.randperm(T * top, generator=g).to(torch.int32)
    new = x[0].double() + (wt.double()[:, :, None] * rows.double()[slot.long()].view(T, top, D)).sum(1)
    want = torch.tanh(0.6 * new) * w.double() + b.double()
    ex = (rows.cuda(), slot.cuda(), wt.cuda())
    got, out = ops.hyper_step(x.cuda(), experts=ex, w=w.cuda(), bias=b.cuda(), kind="dyntanh", alpha=0.6)
    assert torch.allclose(got.cpu()[0].double(), new, atol=1e-5) and torch.allclose(out.cpu().double(), want, atol=1e-5)
    pick = torch.tensor([4, 0], dtype=torch.int32)
    none, out = ops.hyper_step(x.cuda(), experts=ex, w=w.cuda(), bias=b.cuda(), kind="dyntanh", alpha=0.6, rows=pick.cuda())
    assert none is None and torch.allclose(out.cpu().double(), want[pick.long()], atol=1e-5)


# ------------------------------------------------------------------ latent attention
@pytest.mark.parametrize("rot_dim,dims", [(8, 8), (6, 2), (5, 0)])
def test_latent_prep_with_latent_queries(lib, rot_dim, dims):
    """Queries and raw latents from different buffers, rotation in the two-halves and the interleaved layout."""
    from vllm_rs_b200 import ops
    g = torch.Generator().manual_seed(7)
    H, dim, kvr, eps = 3, 10, 12, 1e-2
    pos, slots = [0, 1, 64, 900, 17], torch.tensor([3, 64, 2, 0, 130])
    T = len(pos)
    q, low = torch.randn(T, H * (dim + rot_dim), generator=g), torch.randn(T, kvr + rot_dim + 4, generator=g)
    wn, f = torch.randn(kvr, generator=g), (frequencies(dims, 80.0) if dims else torch.zeros(1, dtype=D64))
    qd = q.double().view(T, H, dim + rot_dim)
    kd = low.double()[:, None, kvr:kvr + rot_dim]
    inter = halves_from_pairs(rot_dim, dims)
    for rot_half in (True, False):
        cache = torch.zeros(3, 64, kvr + rot_dim, device="cuda")
        plain, full = ops.latent_prep_ex(q.cuda(), low.cuda(), cache, wn.cuda(), f.cuda(), 1.0, torch.tensor(pos).cuda(),
                                         slots.cuda(), heads=H, dim=dim, rot_dim=rot_dim, rot_dims=dims, kv_rank=kvr, eps=eps,
                                         rot_half=rot_half)

        def turn(x):
            if rot_half:
                return turned_at(x, pos, dims, 80.0)
            y = turned_at(x[..., inter], pos, dims, 80.0)
            z = torch.empty_like(y)
            z[..., inter] = y
            return z

        assert torch.equal(plain.cpu(), q.view(T, H, dim + rot_dim)[..., :dim])
        assert torch.allclose(full.cpu().double()[..., kvr:], turn(qd[..., dim:]), atol=1e-5)
        want = torch.cat([R.unit_rms(low.double()[:, :kvr], eps) * wn.double(), turn(kd)[:, 0]], -1)
        for t in range(T):
            s = int(slots[t])
            assert torch.allclose(cache.cpu()[s // 64, s % 64].double(), want[t], atol=1e-5)


# ------------------------------------------------------------------ attention: window, sink and cap together
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("split", [True, False])
@pytest.mark.parametrize("dk,dv,H,G,size", [(12, 20, 4, 2, 37), (32, 32, 3, 1, 64), (16, 48, 34, 2, 65), (80, 144, 2, 2, 1), (48, 160, 4, 1, 128)])
def test_attention_op_at_the_window_edge(lib, dtype, split, dk, dv, H, G, size):
    """Every query asks for one key by far: the last one its window keeps, the first one it has lost (what is left then is
    the sink and a flat rest), or the row's own.  Prompt rows and single decoded rows, shuffled block table, a sink per
    head, capped scores."""
    from vllm_rs_b200 import ops
    g = torch.Generator().manual_seed(dk + size)
    n, cap, tol = 260, 9.0, (2e-5 if dtype == torch.float32 else 3e-2)
    pages = [4, 0, 3, 1, 2]
    kc, vc = torch.zeros(5, 64, G, dk, dtype=dtype), torch.zeros(5, 64, G, dv, dtype=dtype)
    k = torch.randn(n, G, dk, generator=g) * 0.1
    v = torch.randn(n, G, dv, generator=g).to(dtype)
    # key j carries the point (cos, sin) of an angle that steps by one radian; a query aimed at j scores highest there
    ang = torch.arange(n, dtype=torch.float32)
    k[:, :, 0], k[:, :, 1] = (2 * torch.cos(ang))[:, None], (2 * torch.sin(ang))[:, None]
    k = k.to(dtype)
    for j in range(n):
        kc[pages[j // 64], j % 64], vc[pages[j // 64], j % 64] = k[j], v[j]
    sink = torch.randn(H, generator=g) + 4.0
    for rows_pos in (range(n), range(n - 1, n), range(130, 132), range(0, 3)):
        T = len(rows_pos)
        pos = torch.tensor(list(rows_pos), dtype=torch.float32)
        for back in (size - 1, size, 0):
            aim = (pos - back).clamp(min=0)
            q = torch.randn(T, H, dk, generator=g) * 0.05
            q[:, :, 0], q[:, :, 1] = (20 * torch.cos(aim))[:, None], (20 * torch.sin(aim))[:, None]
            q = q.to(dtype).float()
            out = ops.window_attn(q.cuda(), kc.cuda(), vc.cuda(), sink.cuda(), None, _i32([0, T]), _i32([rows_pos[-1] + 1]),
                                  _i32([pages]), window=size, keep_first=0, scale=0.4, softcap=cap, split=split).float().cpu()
            kk, vv = (z.double().repeat_interleave(H // G, 1) for z in (k, v))
            s = torch.zeros(H, n, n, dtype=D64)
            s[:, rows_pos] = torch.einsum("ihd,jhd->hij", q.double(), kk) * 0.4
            a = R.softmax_seen(R.cap(s, cap), size, sink.double())[:, rows_pos]
            want = torch.einsum("hij,jhd->ihd", a, vv)
            assert (out.double() - want).abs().max() <= tol * max(1.0, want.abs().max().item()), (rows_pos[0], T, back)


# ------------------------------------------------------------------ router and experts
@pytest.mark.parametrize("E,top", [(7, 3), (1, 1), (40, 40), (16, 2), (64, 33), (5, 1)])
def test_router_op_softmax_over_the_chosen(lib, E, top):
    from vllm_rs_b200 import ops
    g = torch.Generator().manual_seed(E)
    z, b = torch.randn(60, E, generator=g) * 4, torch.randn(E, generator=g) * 3
    z[1] += 300.0                         # large logits: the weights come from differences
    idx, wt = ops.moe_route_full(z.cuda(), b.cuda(), top, 0.7, score="chosen")
    idx, wt = idx.cpu(), wt.cpu()
    for t in range(60):
        want_idx, want_w = R.route((z[t] + b).double(), top)
        assert idx[t].tolist() == want_idx, t
        assert torch.allclose(wt[t].double(), 0.7 * want_w, atol=1e-6)


@pytest.mark.parametrize("T,D,F", [(70, 40, 24), (3, 33, 7), (130, 64, 96)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_clamped_experts_op(lib, T, D, F, dtype):
    """Gate clamped from above only, up clamped on both sides, other constants than the design's; summed and as rows."""
    from vllm_rs_b200 import ops
    g = torch.Generator().manual_seed(T)
    E, top, tol = 5, 3, (1e-5 if dtype == torch.float32 else 2e-2)
    h = torch.randn(T, D, generator=g).to(dtype)
    wu = (torch.randn(E, 2 * F, D, generator=g) * 3 / D ** 0.5).to(dtype)
    wd = (torch.randn(E, D, F, generator=g) / F ** 0.5).to(dtype)
    idx = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(T)]).to(torch.int32)
    wt, x = torch.rand(T, top, generator=g), torch.randn(T, D, generator=g)
    for limit, alpha, add in ((1.5, 1.702, 1.0), (0.4, 1.0, 0.25)):
        def one(t, e):
            u = wu[e].double() @ h[t].double()
            gg, uu = torch.clamp(u[:F], max=limit), torch.clamp(u[F:], -limit, limit)
            return wd[e].double() @ (gg * torch.sigmoid(alpha * gg) * (uu + add))
        if alpha == 1.702:
            p = {"gate": wu[0, :F].double(), "up": wu[0, F:].double(), "down": wd[0].double()}
            assert torch.allclose(one(0, 0), R.expert(h[0].double(), p, "", limit))
        want = torch.stack([torch.stack([one(t, int(idx[t, j])) for j in range(top)]) for t in range(T)])
        kw = dict(act="clamped", limit=limit, alpha=alpha, up_add=add)
        out = ops.moe_experts_ex(x.cuda(), h.cuda(), idx.cuda(), wt.cuda(), wu.cuda(), wd.cuda(), **kw).cpu().double()
        total = x.double() + (wt.double()[:, :, None] * want).sum(1)
        assert (out - total).abs().max() <= 2 * tol * max(1.0, total.abs().max().item())
        rows, slot = ops.moe_experts_rows(h.cuda(), idx.cuda(), wu.cuda(), wd.cuda(), **kw)
        got = rows.cpu().double()[slot.cpu().long()].view(T, top, D)
        assert (got - want).abs().max() <= 2 * tol * max(1.0, want.abs().max().item())


# ------------------------------------------------------------------ one-layer models
@pytest.mark.parametrize("kind,mlp,kw", [
    ("attention", None, {}),
    ("attention", None, dict(heads=3, kv_heads=1, dim=32, vdim=64, mask={"size": 64})),       # tensor-core forms
    ("attention", None, dict(heads=34, kv_heads=2, dim=16, vdim=32)),                         # a group wider than an MMA tile
    ("attention", None, dict(heads=5, kv_heads=5, mask={"size": 1}, v_mix=False)),            # a window of the token itself
    ("retention", None, {}),
    ("retention", None, dict(heads=3, dim=130, vdim=50, rot={"base": 30.0, "dims": 130}, decay=[0.9, 0.25, 0.999])),
    ("latent_attention", None, {}),
    ("latent_attention", None, dict(heads=17, dim=16, rot_dim=16, vdim=32, kv_rank=64, q_rank=80)),     # tensor-core forms
    ("latent_attention", None, dict(heads=2, dim=12, rot_dim=64, vdim=64, kv_rank=128, q_rank=20)),
    ("retention", dense_cfg(), {}),
    ("latent_attention", moe_cfg(), {}),
    ("attention", moe_cfg(experts=1, top=1, limit=0.1), {}),
    ("retention", moe_cfg(experts=6, top=6), {}),
])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_one_layer_alone(lib, kind, mlp, kw, dtype):
    cfg = make_cfg([layer(kind, mlp, **kw)])
    w = random_tensors(cfg, seed=3)
    t = toks(120, cfg["vocab"], 1)
    d = Driver(cfg, w, dtype, trace=True)
    d.step([("a", t)])
    tr = []
    want = R.forward(cfg, w, t, D64, tr).numpy()
    resid = d.runner.trace[0, :len(t)].cpu().numpy()
    tol, q = bounds(dtype, routed=bool(mlp) and mlp["kind"] == "moe")
    row_err = np.abs(resid - tr[0].numpy()).max(-1)
    assert np.quantile(row_err, q) <= tol * np.abs(tr[0].numpy()).max()
    assert rel_err(d.result("a"), want, q) <= tol
    d2 = Driver(cfg, w, dtype)                                        # without the trace the experts' sum joins the final norm
    d2.step([("a", t[:100])])
    for x in t[100:]:                                                 # decode forms
        d2.step([("a", [x])])
    assert rel_err(d2.result("a"), want, q) <= tol


def test_residual_stream_after_every_layer(lib):
    cfg = full_cfg()
    w = random_tensors(cfg, seed=5)
    t = toks(100, cfg["vocab"], 1)
    tr = []
    R.forward(cfg, w, t, D64, tr)
    d = Driver(cfg, w, torch.float32, trace=True)
    d.step([("a", t)])
    for i, want in enumerate(tr):
        got = d.runner.trace[i, :len(t)].cpu().double()
        assert (got - want).abs().max() <= F32_TOL * want.abs().max(), i


# ------------------------------------------------------------------ what must show in the logits
@pytest.mark.parametrize("where", ["prompt", "decoded"])
@pytest.mark.parametrize("size", [37, 64, 65])
def test_window_edges_show_in_logits(lib, where, size):
    """A one-layer model: windows one longer or one shorter give other logits by far more than the tolerance (the score scale
    makes single keys count), and the framework follows the right one, in a prompt portion and for tokens decoded alone."""
    kw = dict(scale=1.5, heads=4, kv_heads=2)
    cfg = make_cfg([layer("attention", None, mask={"size": size}, **kw)])
    w = random_tensors(cfg, seed=4)
    t = toks(2 * size + 5, cfg["vocab"], 5)
    want = ref_logits(cfg, w, t)
    for other in (size - 1, size + 1):
        cfg2 = make_cfg([layer("attention", None, mask={"size": other}, **kw)])
        first = min(size, other)                                      # the first position the two windows treat differently
        lg = ref_logits(cfg2, w, t)
        assert rel_err(want[first:], lg[first:]) > 50 * F32_TOL
        assert rel_err(want[:first], lg[:first]) < 1e-12
    d = Driver(cfg, w, torch.float32)
    if where == "prompt":
        d.step([("a", t[:size - 1])]), d.step([("a", t[size - 1:])])
    else:
        d.step([("a", t[:size])])
        for x in t[size:]:
            d.step([("a", [x])])
    assert rel_err(d.result("a"), want) <= F32_TOL


@pytest.mark.parametrize("what", ["sink", "softcap", "k_scale", "q_latent_norm", "bias_only_chooses"])
def test_small_rules_show_in_logits(lib, what):
    """Each model and a variant with one rule changed differ by far more than the tolerance; the framework follows the rule."""
    kind = {"sink": "attention", "softcap": "attention", "k_scale": "retention", "q_latent_norm": "latent_attention",
            "bias_only_chooses": "retention"}[what]
    kw = {"softcap": dict(softcap=1.0, scale=1.0), "k_scale": dict(dim=16, rot={"base": 50.0, "dims": 16})}.get(what, {})
    eps = 0.1 if what == "k_scale" else 1e-5                          # with eps near the outputs' size the key factor shows
    cfg = make_cfg([layer(kind, moe_cfg() if what == "bias_only_chooses" else None, **kw)], eps=eps)
    w = random_tensors(cfg, seed=8)
    t = toks(70, cfg["vocab"], 3)
    want = ref_logits(cfg, w, t)
    w2, cfg2, route = dict(w), cfg, R.route
    if what == "sink":
        w2["l0.mix.sink"] = torch.full_like(w["l0.mix.sink"], -50.0)
    elif what == "softcap":
        cfg2 = make_cfg([layer(kind, None, **{**kw, "softcap": 1000.0})], eps=eps)
    elif what == "k_scale":
        w2["l0.mix.k"] = (w["l0.mix.k"].float() * 4).to(torch.bfloat16)
    elif what == "q_latent_norm":
        w2["l0.mix.dq.norm"] = torch.ones_like(w["l0.mix.dq.norm"])
    else:
        bias = w["l0.mlp.router.b"].double()
        R.route = lambda z, top: (lambda c: (c, torch.softmax((z - bias)[c], 0)))(route(z, top)[0])
    try:
        other = ref_logits(cfg2, w2, t)
    finally:
        R.route = route
    assert rel_err(want, other) > 50 * F32_TOL
    d = Driver(cfg, w, torch.float32)
    d.step([("a", t[:40])]), d.step([("a", t[40:])])
    assert rel_err(d.result("a"), want) <= F32_TOL


@pytest.mark.parametrize("kind", ["attention", "latent_attention", "retention"])
def test_a_far_token_shows_in_logits(lib, kind):
    """Replacing the very first token of a 300-token prompt changes the last row's logits of the plain model by far more
    than the tolerance, and the framework follows, the last row decoded alone after portions that end at and just after a
    page border.  Attentions: the query projection is made to turn the last token's input into the first token's key (and
    rotated entries stay out of the scores), so that one score stands out among hundreds.  Retention: decays of almost
    one, so the first token's write is still in the state."""
    n, D = 300, 48
    a, b = 94, 95                                                      # the first and the last token
    if kind == "attention":
        cfg = make_cfg([layer(kind, None, heads=2, kv_heads=1, dim=64, vdim=16, scale=0.5, softcap=60.0, mask={"size": 300},
                              rot={"base": 100.0, "dims": 2}, v_mix=False)])
    elif kind == "latent_attention":
        cfg = make_cfg([layer(kind, None, heads=1, dim=64, rot_dim=2, vdim=16, kv_rank=64, q_rank=64, scale=0.5)])
    else:
        cfg = make_cfg([layer(kind, None, decay=[0.9990234375, 1.0, 1.0, 0.9990234375])])
    w = random_tensors(cfg, seed=11)
    x = w["embed"].double() * cfg["embedding"]["scale"]
    W = {k: v.double() for k, v in w.items()}
    ha, hb = (R.dynamic_tanh(x[i], W, "l0.norm1") for i in (a, b))

    def aim(key_rows):                    # a projection like the keys' that maps hb to the key of ha
        return (key_rows + torch.outer(key_rows @ (ha - hb), hb) / (hb @ hb)).to(torch.bfloat16)

    if kind == "attention":
        q = aim(W["l0.mix.k"])
        w["l0.mix.q"] = torch.cat([q, q])
        w["l0.mix.q.norm"], w["l0.mix.k.norm"] = torch.ones(64).bfloat16(), torch.ones(64).bfloat16()
        w["l0.mix.q.norm"][:2] = 0.0
        w["l0.mix.sink"] = torch.zeros(2).bfloat16()
    elif kind == "latent_attention":
        w["l0.mix.dq"] = aim(W["l0.mix.dkv"][:64])
        for name in ("dq.norm", "dkv.norm"):
            w["l0.mix." + name] = torch.ones(64).bfloat16()
        w["l0.mix.uk"] = torch.eye(64).bfloat16()
        w["l0.mix.uq"] = torch.cat([torch.eye(64), torch.zeros(2, 64)]).bfloat16()
    base = toks(n, 90, 5)
    base[-1] = b
    t = list(base)
    t[0] = a
    want, other = ref_logits(cfg, w, t), ref_logits(cfg, w, base)
    assert rel_err(want[-1:], other[-1:]) > (200 if kind != "retention" else 50) * F32_TOL
    for dtype in (torch.float32, torch.bfloat16):
        d = Driver(cfg, w, dtype)
        d.step([("a", t[:64])]), d.step([("a", t[64:129])]), d.step([("a", t[129:n - 1])]), d.step([("a", t[n - 1:])])
        assert rel_err(d.result("a"), want) <= bounds(dtype, False)[0]


def test_value_mixing_follows_the_first_mixing_layer(lib):
    """Values come from the first attention with v_mix (not from layer 0, not from the layer before), un-mixed and of the
    same token, in batches whose rows belong to several requests; layers of other kinds lie in between."""
    kw = dict(heads=4, kv_heads=2, dim=16, vdim=16)
    cfg = make_cfg([layer("attention", None, v_mix=False, **kw), layer("attention", dense_cfg(), **kw), layer("retention", None),
                    layer("attention", None, **kw), layer("latent_attention", None), layer("attention", dense_cfg(24), **kw)])
    w = random_tensors(cfg, seed=6)
    a, b = toks(90, cfg["vocab"], 7), toks(70, cfg["vocab"], 8)
    wa, wb = ref_logits(cfg, w, a), ref_logits(cfg, w, b)
    for i in (0, 1, 5):                                               # other readings of the rule give other logits
        other = make_cfg([dict(L, mixer=dict(L["mixer"])) for L in cfg["layers"]])
        other["layers"][i]["mixer"]["v_mix"] = not other["layers"][i]["mixer"]["v_mix"]
        w2 = dict(w)
        w2.setdefault("l0.mix.vmix", w["l1.mix.vmix"])
        assert rel_err(ref_logits(other, w2, a), wa) > 50 * F32_TOL, i
    d = Driver(cfg, w, torch.float32)
    d.step([("b", b[:3]), ("a", a[:64])]), d.step([("a", a[64:66]), ("b", b[3:60])])
    for i in range(66, 90):
        d.step([("a", [a[i]])] + ([("b", [b[i - 6]])] if i - 6 < 70 else []))
    assert rel_err(d.result("a"), wa) <= F32_TOL
    assert rel_err(d.result("b"), wb[:len(d.result("b"))]) <= F32_TOL


# ------------------------------------------------------------------ schedules
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_whole_decode_and_portions_agree_with_the_plain_model(lib, dtype):
    cfg = full_cfg()
    w = random_tensors(cfg, seed=7)
    t = toks(150, cfg["vocab"], 3)
    want = ref_logits(cfg, w, t)
    tol, q = bounds(dtype)
    d = Driver(cfg, w, dtype)
    d.step([("whole", t)])
    assert rel_err(d.result("whole"), want, q) <= tol
    d.close("whole")
    d.step([("dec", t[:60])])
    for x in t[60:]:
        d.step([("dec", [x])])
    assert rel_err(d.result("dec"), want, q) <= tol
    d.close("dec")
    cuts = [2, 1, 2, 61, 2, 3, 64, 2, 13]                            # 150 tokens; cuts inside and at the ends of pages
    at = 0
    for c in cuts:
        d.step([("cut", t[at:at + c])])
        at += c
    assert at == len(t)
    assert rel_err(d.result("cut"), want, q) <= tol
    if dtype == torch.float32:                                       # the cut must not matter beyond rounding
        assert rel_err(d.result("cut"), d.result("dec")) <= 2e-5


def test_unequal_batches_and_reuse_of_pages_and_slots(lib):
    cfg = full_cfg()
    w = random_tensors(cfg, seed=9)
    V = cfg["vocab"]
    reqs = {"a": toks(130, V, 1), "b": toks(3, V, 2), "c": toks(70, V, 3), "d": toks(65, V, 4), "e": toks(40, V, 5),
            "f": toks(129, V, 6)}
    want = {k: ref_logits(cfg, w, v) for k, v in reqs.items()}
    d = Driver(cfg, w, torch.float32, num_blocks=7, max_seqs=4, slots=4)      # 7 pages: a(3) + c(2) + d(2) fill it
    at = {k: 0 for k in reqs}

    def portion(k, n):
        p = (k, reqs[k][at[k]:at[k] + n])
        at[k] += n
        return p

    d.step([portion("a", 64), portion("b", 2)])
    d.step([portion("a", 1), portion("b", 1), portion("c", 30)])
    d.close("b")                                                      # its page and slot go back
    d.step([portion("c", 40), portion("a", 2), portion("d", 65)])
    d.step([portion("a", 63)])
    d.close("a"), d.close("c")
    assert d.sched.num_free_blocks == 5 and d.sched.num_free_state_slots == 3
    d.step([portion("e", 39), portion("f", 128)])                     # reuses a's and c's pages and slots
    d.step([portion("f", 1), portion("e", 1)])
    for k in "abcdef":
        assert at[k] == len(reqs[k])
        assert rel_err(d.result(k), want[k]) <= F32_TOL, k


def test_first_tokens_and_long_decoding(lib):
    cfg = full_cfg()
    w = random_tensors(cfg, seed=13)
    t = toks(260, cfg["vocab"], 8)
    want = ref_logits(cfg, w, t)
    d = Driver(cfg, w, torch.float32)
    for x in t:                                                       # every token alone, from the very first
        d.step([("a", [x])])
    got = d.result("a")
    assert rel_err(got[:6], want[:6]) <= F32_TOL
    assert rel_err(got, want) <= F32_TOL


def test_other_sizes(lib):
    """Sizes of one and values that coincide elsewhere: one head, heads of one or two entries, a window of one token, no cap,
    ranks of one, one expert, a feed-forward of one unit, a factor of one on the sublayers, an embedding scale of one."""
    cfg = make_cfg([layer("attention", dense_cfg(7), heads=1, kv_heads=1, dim=2, vdim=1, scale=1.0, softcap=0.0,
                          rot={"base": 2.0, "dims": 2}, mask={"size": 1}),
                    layer("retention", dense_cfg(1), heads=1, dim=2, vdim=5, decay=[1.0], rot={"base": 9.0, "dims": 2}),
                    layer("latent_attention", moe_cfg(ff=1, experts=1, top=1), heads=1, dim=1, rot_dim=2, vdim=1, kv_rank=1, q_rank=1),
                    layer("attention", moe_cfg(ff=3, experts=2, top=2), heads=7, kv_heads=1, dim=8, vdim=1, rot={"base": 1e4, "dims": 4},
                          mask={"size": 1000}),
                    layer("latent_attention", dense_cfg(130), heads=7, dim=3, rot_dim=6, vdim=130, kv_rank=5, q_rank=130),
                    layer("retention", None, heads=7, dim=130, vdim=1, decay=[0.125 * (i + 1) for i in range(7)], rot={"base": 9.0, "dims": 4})],
                   width=24, vocab=50, eps=1e-3, mult=1.0, embed_scale=1.0)
    w = random_tensors(cfg, seed=17)
    t = toks(80, cfg["vocab"], 9)
    want = ref_logits(cfg, w, t)
    d = Driver(cfg, w, torch.float32)
    d.step([("a", t[:7])]), d.step([("a", t[7:9])]), d.step([("a", t[9:])])
    assert rel_err(d.result("a"), want) <= F32_TOL


def test_greedy_generation_through_the_engine(lib):
    """LLMEngine (schedule -> chunked prefill -> decode, state slots from the scheduler) against greedy decoding with
    the plain model."""
    from vllm_rs_b200 import engine, models
    cfg = full_cfg()
    w = random_tensors(cfg, seed=21)
    V = cfg["vocab"]
    prompts = [toks(75, V, 1), toks(5, V, 2), toks(40, V, 3)]
    new = 12
    runner = models.build_runner(cfg, w, dtype=torch.float32, device="cuda", num_blocks=12, max_blocks_per_seq=4,
                                 max_seqs=5, max_tokens=64, num_state_slots=5)
    eng = engine.LLMEngine(runner, 12, 3, chunk_size=32)              # prompts longer than a chunk are cut
    sids = [eng.add_request(p, new) for p in prompts]
    out = eng.run_to_completion()
    for sid, p in zip(sids, prompts):
        seq, want = list(p), []
        for _ in range(new):
            lg = ref_logits(cfg, w, seq)[-1]
            top2 = np.sort(lg)[-2:]
            nxt = int(lg.argmax())
            if top2[1] - top2[0] < 1e-3:                              # a near tie may flip in fp32: stop comparing there
                break
            want.append(nxt)
            seq.append(nxt)
        assert out[sid][:len(want)] == want
    assert eng.sched.num_free_state_slots == 5


# ------------------------------------------------------------------ random configurations under random schedules
@pytest.mark.parametrize("seed", [11, 12, 13, 14, 15, 16])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_random_configurations_under_random_schedules(lib, seed, dtype):
    """Sizes, layer orders and constants drawn at random (odd sizes, groups wider than an MMA tile, partial rotations,
    windows of 1 .. 200 positions, ranks that fit the tensor-core forms and ranks that do not); five requests of 5 .. 420
    tokens share four state slots and just enough pages, so both are used again."""
    rng = np.random.default_rng(seed)
    pick = lambda *xs: xs[int(rng.integers(len(xs)))]              # noqa: E731
    cfg = make_cfg(random_layers(rng, int(rng.integers(2, 7))), width=pick(64, 128, 200), vocab=pick(300, 512),
                   eps=pick(1e-6, 1e-5), mult=pick(0.6, 1.0), embed_scale=pick(0.8, 3.0))
    w = random_tensors(cfg, seed=seed)
    reqs = {f"r{i}": toks(pick(5, 40, 150, 260, 420), cfg["vocab"], seed + i) for i in range(5)}
    pages = sum(sorted((len(v) + 63) // 64 for v in reqs.values())[-4:])
    d = Driver(cfg, w, dtype, num_blocks=pages, max_seqs=4, slots=4)
    for st, ends in random_schedule(rng, reqs):
        d.step(st)
        for k in ends:
            d.close(k)
    tol, q = bounds(dtype, any(L["mlp"] and L["mlp"]["kind"] == "moe" for L in cfg["layers"]))
    for k in reqs:
        assert rel_err(d.result(k), ref_logits(cfg, w, reqs[k]), q) <= tol, (k, [L["type"] for L in cfg["layers"]])


# ------------------------------------------------------------------ a model folder through the command line
def _write_model_folder(path, cfg, tensors):
    """config.json and model.safetensors (8-byte little-endian header length, JSON header, raw data), bf16 tensors."""
    header, blobs, at = {}, [], 0
    for name, t in tensors.items():
        raw = t.contiguous().view(torch.int16).numpy().tobytes()
        header[name] = {"dtype": "BF16", "shape": list(t.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    hj = json.dumps(header).encode()
    with open(path / "model.safetensors", "wb") as f:
        f.write(struct.pack("<Q", len(hj)) + hj + b"".join(blobs))
    with open(path / "config.json", "w") as f:
        json.dump(cfg, f)


def test_model_folder_through_trace_runner_and_generate(lib, tmp_path):
    """The registry picks the model by config.json; the trace runner replays two interleaved requests on a pool of
    three pages (the second request reuses the first one's page and slot), `generate` decodes greedily."""
    root = Path(__file__).resolve().parent.parent
    cfg = full_cfg()
    w = random_tensors(cfg, seed=23)
    assert all(t.dtype == torch.bfloat16 for t in w.values())
    _write_model_folder(tmp_path, cfg, w)
    V = cfg["vocab"]
    a, b, c = toks(70, V, 1), toks(9, V, 2), toks(64, V, 3)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:40], "want": [0, 39]}, {"id": "b", "tokens": b[:2], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[2:], "want": [6]}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[40:69], "want": [28]}, {"id": "c", "tokens": c, "want": [63]}], "end": ["c"]},
             {"step": 3, "entries": [{"id": "a", "tokens": a[69:], "want": [0]}], "end": ["a"]}]
    out = tmp_path / "out"
    r = subprocess.run([str(root / "bin" / "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out", str(out),
                        "--max-tokens", "192"], input="".join(json.dumps(s) + "\n" for s in steps), text=True,
                       capture_output=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [ln for ln in r.stdout.split("\n") if ln.startswith("done")] == [f"done {i}" for i in range(4)]
    ra, rb, rc = ref_logits(cfg, w, a), ref_logits(cfg, w, b), ref_logits(cfg, w, c)
    want = {0: ra[[0, 39]], 1: rb[[8]], 2: np.stack([ra[68], rc[63]]), 3: ra[[69]]}
    for i, ref in want.items():
        got = np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(-1, V)
        assert rel_err(got, ref) <= 2 * F32_TOL, i
    r = subprocess.run([sys.executable, "-m", "vllm_rs_b200", "generate", "--model", str(tmp_path), "--dtype", "float32",
                        "--prompt-ids", ",".join(map(str, b)), "--max-new-tokens", "5"], cwd=root, text=True,
                       capture_output=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    got = json.loads(r.stdout.strip().split("\n")[-1])["output_ids"]
    seq = list(b)
    for k in range(5):
        lg = ref_logits(cfg, w, seq)[-1]
        top2 = np.sort(lg)[-2:]
        if top2[1] - top2[0] < 1e-3:
            break
        assert got[k] == int(lg.argmax()), k
        seq.append(int(lg.argmax()))
