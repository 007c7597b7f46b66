"""Zufulix on the GPU against the plain restatement in tests/zufulix_ref.py: each mechanism alone (as a kernel and as a
one-layer model), whole prompts against token-by-token decoding, portions down to two tokens, unequal batches against
each request alone, pages and slots that are used again, keys far back, at page borders and at the edges of the distance
buckets with inputs made so that one key stands out, routers whose groups decide the choice, values mixed with an
earlier layer's, the first tokens of a sequence, long decoding, several sizes, and greedy generation through LLMEngine.
fp32 runs are held to 2e-4 of the logits' spread, bf16 runs to 6e-2; models with routed experts are compared at the 0.9
quantile of their rows in bf16, where 16-bit operands can flip a near-tied expert choice at single rows."""
import numpy as np
import pytest
import torch

import zufulix_ref as R
from fidasun_util import Driver, rel_err
from zalalix_util import random_schedule
from zufulix_util import dense_cfg, full_cfg, layer, make_cfg, moe_cfg, random_layers, random_tensors

pytestmark = pytest.mark.gpu
F32_TOL, BF16_TOL = 2e-4, 6e-2


def ref_logits(cfg, tensors, tokens):
    return R.forward(cfg, tensors, tokens, torch.float64).numpy()


def toks(n, vocab, seed):
    return np.random.default_rng(seed).integers(0, vocab, size=n).tolist()


def _i32(a):
    return torch.tensor(a, dtype=torch.int32, device="cuda")


def bounds(dtype, routed=True):
    """(tolerance, quantile of the rows it applies to)."""
    if dtype == torch.float32:
        return F32_TOL, 1.0
    return BF16_TOL, 0.9 if routed else 1.0


# ------------------------------------------------------------------ row kernels
@pytest.mark.parametrize("S,D", [(1, 40), (2, 33), (3, 1028), (4, 2048), (5, 300), (8, 64), (16, 36), (13, 7)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_hyper_step_op(lib, S, D, dtype):
    """Update, read and norm in one pass; streams that are all equal (stored once); the read without an update; the norm
    of listed rows only; the sublayer's rows given as unsummed expert rows; every kind of norm."""
    from vllm_rs_b200 import ops
    g = torch.Generator().manual_seed(S * 1000 + D)
    T, eps = 9, 1e-3
    rnd = lambda *s: torch.randn(*s, generator=g)                     # noqa: E731
    x, y, mix, ow, iw = rnd(S, T, D) * 2 + 0.5, rnd(T, D), rnd(S, S), rnd(S), rnd(S)
    w, b = rnd(D), rnd(D)
    tol = 2e-5 if dtype == torch.float32 else 1e-2
    d = lambda t: t.double()                                          # noqa: E731
    c = lambda t: t.cuda().contiguous()                               # noqa: E731

    def near(got, want, what):
        assert (got.cpu().double() - want).abs().max() <= tol * max(1.0, want.abs().max().item()), what

    kw = dict(mix=c(mix), out_w=c(ow), in_w=c(iw), w=c(w), bias=c(b), eps=eps, dtype=dtype)
    for xs, equal in ((x, 0), (x[0], S)):
        old = [d(xs[s]) for s in range(S)] if not equal else [d(xs)] * S
        new = R.update_streams(old, d(mix), d(ow), d(y))
        z, h = ops.hyper_step(c(xs), y=c(y), equal_streams=equal, **kw)
        want_h = R.layer_norm(R.read_streams(new, d(iw)), d(w), d(b), eps)
        for t in range(S):
            assert (z[t].cpu().double() - new[t]).abs().max() <= 2e-5 * max(1.0, new[t].abs().max().item()), (t, equal)
        near(h, want_h, "norm")
        z, h = ops.hyper_step(c(xs), equal_streams=equal, **{k: v for k, v in kw.items() if k not in ("mix", "out_w")})
        assert z is None
        near(h, R.layer_norm(R.read_streams(old, d(iw)), d(w), d(b), eps), "read only")
        rows = [7, 0, 7, 3]
        _, h = ops.hyper_step(c(xs), y=c(y), equal_streams=equal, rows=_i32(rows), **{**kw, "in_w": None})
        near(h, R.layer_norm(sum(new)[rows], d(w), d(b), eps), "rows, plain sum")
    new = R.read_streams(R.update_streams([d(x[s]) for s in range(S)], d(mix), d(ow), d(y)), d(iw))
    _, h = ops.hyper_step(c(x), y=c(y), **{**kw, "bias": None}, kind="rms", w_offset=1.0)
    near(h, R.unit_rms(new, eps) * (1 + d(w)), "rms")
    _, h = ops.hyper_step(c(x), y=c(y), **kw, kind="dyntanh", alpha=0.4)
    near(h, torch.tanh(0.4 * new) * d(w) + d(b), "dynamic tanh")
    top = 3
    slot = torch.randperm(T * top, generator=g).to(torch.int32)
    er, tw = rnd(T * top, D), torch.rand(T, top, generator=g)
    ye = sum(d(tw[:, j:j + 1]) * d(er[slot.view(T, top)[:, j].long()]) for j in range(top))
    z, _ = ops.hyper_step(c(x), experts=(c(er), c(slot), c(tw)), mix=c(mix), out_w=c(ow), in_w=c(iw))
    want = R.update_streams([d(x[s]) for s in range(S)], d(mix), d(ow), ye)
    for t in range(S):
        assert (z[t].cpu().double() - want[t]).abs().max() <= 2e-5 * max(1.0, want[t].abs().max().item()), t


def test_layer_norm_kind_and_gelu_ops(lib):
    from vllm_rs_b200 import ops
    g = torch.Generator().manual_seed(1)
    x, w, b = torch.randn(11, 130, generator=g) * 3 + 40.0, torch.randn(130, generator=g), torch.randn(130, generator=g)
    got = ops.stream_norm(x.cuda(), w.cuda(), b.cuda(), kind="layer", eps=1e-5).cpu().double()
    assert torch.allclose(got, R.layer_norm(x.double(), w.double(), b.double(), 1e-5), atol=2e-4)   # a mean far above the spread
    up, bias = torch.randn(7, 50, generator=g) * 3, torch.randn(41, generator=g)
    got = ops.ff_act(up.cuda(), bias.cuda(), "gelu", n=41).cpu().double()
    assert torch.allclose(got, R.gelu(up[:, :41].double() + bias.double()), atol=3e-6)
    got = ops.ff_act(up.cuda(), None, "relu2", dtype=torch.bfloat16).cpu().double()
    assert torch.allclose(got, torch.relu(up.double()) ** 2, rtol=1e-2)


# ------------------------------------------------------------------ attention: learned distance bias, prep
def _plain_attention(q, k, v, rows_pos, scale, rel, far):
    T, H, _ = q.shape
    G, dv = k.shape[1], v.shape[2]
    out = torch.zeros(T, H, dv, dtype=torch.float64)
    bias = R.distance_bias_rows(rel, rows_pos, k.shape[0], far)
    for r, i in enumerate(rows_pos):
        for h in range(H):
            a = h // (H // G)
            p = torch.softmax((k[:i + 1, a] @ q[r, h]) * scale + bias[h, r, :i + 1], 0)
            out[r, h] = (p[:, None] * v[:i + 1, a]).sum(0)
    return out


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("split", [True, False])
@pytest.mark.parametrize("dk,dv,H,G", [(12, 20, 4, 2), (32, 32, 3, 1), (16, 48, 34, 2), (80, 144, 2, 2), (48, 160, 4, 1)])
def test_attention_op_with_a_learned_distance_bias(lib, dtype, split, dk, dv, H, G):
    """Random tables, and tables in which one bucket stands out by far: the row's own position, the last distance of the
    linear half, the first of the geometric half, the last distance before the open bucket (nothing further may be
    counted in), and the open bucket (whose keys share the weight).  A query that asks for a far key or for the key at a
    page border has to overcome the bias.  Prompt rows and single decoded rows, shuffled block table."""
    from vllm_rs_b200 import ops
    from vllm_rs_b200.models.zufulix import distance_table
    n, B, far = 330, 16, 120
    pages = [5, 2, 7, 0, 3, 6]
    g = torch.Generator().manual_seed(0)
    u = (torch.arange(n) - 160.0) / 256.0
    k = torch.randn(n, G, dk, generator=g) * 0.05
    k[:, :, 0], k[:, :, 1] = u[:, None], (u * u)[:, None]
    v = torch.randn(n, G, dv, generator=g)
    kc = torch.zeros(8, 64, G, dk, dtype=dtype, device="cuda")
    vc = torch.zeros(8, 64, G, dv, dtype=dtype, device="cuda")
    for j in range(n):
        kc[pages[j // 64], j % 64], vc[pages[j // 64], j % 64] = k[j].to(dtype).cuda(), v[j].to(dtype).cuda()
    kr, vr = k.to(dtype).double(), v.to(dtype).double()
    tol = 3e-3 if dtype == torch.float32 else 4e-2
    sharp = 16384.0
    forms = [("flat", None), ("first", None), ("border", None)] + [("bucket", b) for b in (0, 1, B // 2 - 1, B // 2, B - 2, B - 1)]
    for rows_pos in ([329], [64], [63], [0], list(range(200, 329)), list(range(0, 70)), list(range(250, 260))):
        T = len(rows_pos)
        pos = torch.tensor(rows_pos, dtype=torch.float32)
        for form, bucket in forms:
            q = torch.randn(T, H, dk, generator=g) * 0.1
            rel = torch.randn(B, H, generator=g)
            if form == "bucket":
                rel[bucket] += 40.0
            elif form != "flat":
                target = torch.zeros(T) if form == "first" else torch.full((T,), 127.0).minimum(pos)
                q[:, :, 0], q[:, :, 1] = (2.0 * sharp * (target - 160.0) / 256.0)[:, None], -sharp
            q = q.to(dtype).float()
            out = ops.window_attn(q.cuda().contiguous(), kc, vc, None, None, _i32([0, T]), _i32([rows_pos[-1] + 1]),
                                  _i32([pages]), window=0, keep_first=0, scale=1.0, split=split,
                                  dist_bias=distance_table(rel, far).cuda()).float().cpu()
            want = _plain_attention(q.double(), kr, vr, rows_pos, 1.0, rel.double(), far)
            assert (out.double() - want).abs().max() <= tol * max(1.0, want.abs().max().item()), (rows_pos[0], T, form, bucket)


def test_a_table_too_large_for_shared_memory(lib):
    """More distances than the kernels stage: the table is read from global memory."""
    from vllm_rs_b200 import ops
    from vllm_rs_b200.models.zufulix import distance_table
    g = torch.Generator().manual_seed(4)
    n, H, G, dk, dv, B, far = 200, 2, 1, 16, 16, 6, 400000
    k, v = torch.randn(n, G, dk, generator=g).bfloat16(), torch.randn(n, G, dv, generator=g).bfloat16()
    kc, vc = torch.zeros(4, 64, G, dk, dtype=torch.bfloat16), torch.zeros(4, 64, G, dv, dtype=torch.bfloat16)
    kc.view(-1, G, dk)[:n], vc.view(-1, G, dv)[:n] = k, v
    rel = torch.randn(B, H, generator=g) * 3
    table = distance_table(rel, far)
    assert table.shape[1] > 2048
    q = torch.randn(n, H, dk, generator=g).bfloat16().float()
    out = ops.window_attn(q.cuda(), kc.cuda(), vc.cuda(), None, None, _i32([0, n]), _i32([n]), _i32([[0, 1, 2, 3]]), window=0,
                          keep_first=0, scale=0.3, dist_bias=table.cuda()).float().cpu()
    want = _plain_attention(q.double(), k.double(), v.double(), range(n), 0.3, rel.double(), far)
    assert (out.double() - want).abs().max() <= 4e-2


def test_attention_prep_op_weightless_norms_and_mixed_values(lib):
    from vllm_rs_b200 import ops
    g = torch.Generator().manual_seed(3)
    H, G, dk, dv, eps, lam = 6, 2, 10, 7, 1e-2, 0.3
    T = 6
    slots = torch.tensor([3, 64, 2, 0, 130, 191])
    proj = torch.randn(T, H * dk + G * dk + G * dv + 5, generator=g)
    bias = torch.randn(H * dk + G * dk + G * dv, generator=g)
    pos = torch.arange(T)
    kept = torch.zeros(T, G * dv, device="cuda")
    x = proj.double()[:, :bias.numel()] + bias.double()
    first = torch.randn(T, G * dv, generator=g)
    for kw in (dict(v_first_out=kept), dict(v_first=first.cuda(), v_mix=lam)):
        kc, vc = torch.zeros(3, 64, G, dk, device="cuda"), torch.zeros(3, 64, G, dv, device="cuda")
        q = ops.window_attn_prep(proj.cuda(), bias.cuda(), None, None, None, pos.cuda(), slots.cuda(), kc, vc, heads=H,
                                 rot_dims=0, eps=eps, head_norm=2, **kw).cpu()
        own = x[:, (H + G) * dk:]
        want_v = own if "v_first_out" in kw else R.mix_values(own, first.double(), lam)
        for t in range(T):
            s = int(slots[t])
            assert torch.allclose(q[t].double(), R.unit_rms(x[t, :H * dk].view(H, dk), eps), atol=1e-5)
            assert torch.allclose(kc.cpu()[s // 64, s % 64].double(), R.unit_rms(x[t, H * dk:(H + G) * dk].view(G, dk), eps), atol=1e-5)
            assert torch.allclose(vc.cpu()[s // 64, s % 64].double().reshape(-1), want_v[t], atol=1e-6)
    assert torch.allclose(kept.cpu().double(), x[:, (H + G) * dk:], atol=1e-6)


# ------------------------------------------------------------------ router and experts
@pytest.mark.parametrize("E,top,groups,keep", [(12, 4, 4, 2), (12, 3, 3, 1), (16, 5, 0, 0), (6, 2, 6, 3), (40, 7, 5, 5), (1, 1, 1, 1),
                                               (64, 33, 2, 2)])
def test_router_op_sigmoid_group_sums_and_normalised_weights(lib, E, top, groups, keep):
    from vllm_rs_b200 import ops
    g = torch.Generator().manual_seed(E)
    z = torch.randn(60, E, generator=g) * 2
    if groups == 3:                       # one token whose best single expert sits in a group that loses on the pair
        z[0] = -4.0
        z[0, 0], z[0, 5], z[0, 6] = 3.0, 2.0, 1.9
    idx, wt = ops.moe_route_full(z.cuda(), None, top, 1.0, groups, keep, score="sigmoid", group_top=2, renorm=True)
    idx, wt = idx.cpu(), wt.cpu()
    for t in range(60):
        want_idx, want_w = R.route(z[t].double(), top, groups, keep)
        assert idx[t].tolist() == want_idx, t
        assert torch.allclose(wt[t].double(), torch.stack(want_w), atol=1e-6)
    if groups == 3:
        assert 0 not in idx[0].tolist() and idx[0, :2].tolist() == [5, 6]


def test_expert_rows_op(lib):
    """The unsummed rows, weighed by the caller, are the experts' sum."""
    from vllm_rs_b200 import ops
    g = torch.Generator().manual_seed(8)
    T, D, F, E, top = 70, 40, 24, 5, 3
    for dtype, tol in ((torch.float32, 1e-5), (torch.bfloat16, 2e-2)):
        h = torch.randn(T, D, generator=g).to(dtype)
        wu, wd = (torch.randn(E, F, D, generator=g) / 6).to(dtype), (torch.randn(E, D, F, generator=g) / 5).to(dtype)
        idx = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(T)]).to(torch.int32)
        rows, slot = ops.moe_experts_rows(h.cuda(), idx.cuda(), wu.cuda(), wd.cuda(), act="relu2")
        assert sorted(slot.tolist()) == list(range(T * top))
        got = rows.cpu().double()[slot.cpu().long()].view(T, top, D)
        for t in range(T):
            for j in range(top):
                e = int(idx[t, j])
                want = R.expert(h[t].double(), {"up": wu[e].double(), "down": wd[e].double()}, "")
                assert (got[t, j] - want).abs().max() <= tol * max(1.0, want.abs().max().item())


# ------------------------------------------------------------------ one-layer models
@pytest.mark.parametrize("mlp,kw,streams", [
    (None, {}, 3),
    (None, dict(heads=5, kv_heads=5, dim=24, v_mix=False), 1),                             # no grouping, one stream
    (None, dict(heads=3, kv_heads=1, dim=32, vdim=64, buckets=2, bias_max=7), 4),          # tensor-core forms
    (None, dict(heads=34, kv_heads=2, dim=16, vdim=32), 2),                                # a group wider than an MMA tile
    (None, dict(heads=1, kv_heads=1, dim=1, vdim=1, buckets=1), 6),
    (dense_cfg(), {}, 2),
    (moe_cfg(), {}, 4),
    (moe_cfg(experts=4, top=1, groups=None), {}, 5),
    (moe_cfg(experts=6, top=2, groups=(6, 2)), {}, 3),                                     # groups of one expert
    (moe_cfg(experts=1, top=1, groups=(1, 1)), {}, 1),
])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_one_layer_alone(lib, mlp, kw, streams, dtype):
    if dtype == torch.bfloat16 and kw.get("vdim") == 1:
        pytest.skip("one-element heads: a single 16-bit rounding is the whole value, nothing averages out")
    cfg = make_cfg([layer(mlp, **kw)], streams=streams)
    w = random_tensors(cfg, seed=3)
    t = toks(90, cfg["vocab"], 1)
    d = Driver(cfg, w, dtype, trace=True)
    d.step([("a", t)])
    tr = []
    want = R.forward(cfg, w, t, torch.float64, tr).numpy()
    resid = d.runner.trace[0, :len(t)].cpu().numpy()
    tol, q = bounds(dtype, routed=bool(mlp) and mlp["kind"] == "moe")
    row_err = np.abs(resid - tr[0].numpy()).max(-1)
    assert np.quantile(row_err, q) <= tol * np.abs(tr[0].numpy()).max()
    assert rel_err(d.result("a"), want, q) <= tol
    d2 = Driver(cfg, w, dtype)                                         # without the trace the last update is never stored
    d2.step([("a", t)])
    assert rel_err(d2.result("a"), d.result("a")) <= 1e-5


def test_residual_streams_after_every_layer(lib):
    cfg = full_cfg()
    w = random_tensors(cfg, seed=5)
    t = toks(100, cfg["vocab"], 1)
    tr = []
    R.forward(cfg, w, t, torch.float64, tr)
    d = Driver(cfg, w, torch.float32, trace=True)
    d.step([("a", t)])
    for i, want in enumerate(tr):
        got = d.runner.trace[i, :len(t)].cpu().double()
        assert (got - want).abs().max() <= F32_TOL * want.abs().max(), i


# ------------------------------------------------------------------ what must show in the logits
@pytest.mark.parametrize("where", ["prompt", "decoded"])
@pytest.mark.parametrize("edge", ["half", "last"])
def test_bucket_edges_show_in_logits(lib, where, edge):
    """A one-layer model in which one bucket's bias stands out.  Moving that bucket's edge by one place (another bias_max, or
    the restated bucket of the single distance at the edge) changes the plain model's logits by far more than the tolerance, and
    the framework follows the right one, in a prompt portion and for tokens decoded alone."""
    B, far = 12, 40
    half = B // 2
    bucket = half if edge == "half" else B - 1
    first = next(n for n in range(1000) if R.distance_bucket(n, B, far) == bucket)       # first distance in the bucket
    cfg = make_cfg([layer(None, buckets=B, bias_max=far, v_mix=False)])
    w = random_tensors(cfg, seed=4)
    w["l0.mix.rel"][bucket] = 12.0
    t = toks(3 * far, cfg["vocab"], 5)
    want = ref_logits(cfg, w, t)
    plain = R.distance_bucket
    try:                                  # the plain model with the edge one place later
        R.distance_bucket = lambda n, b, f: plain(n - 1 if n == first else n, b, f)
        other = ref_logits(cfg, w, t)
    finally:
        R.distance_bucket = plain
    assert rel_err(want[first:first + 1], other[first:first + 1]) > 50 * F32_TOL
    assert rel_err(want[:first], other[:first]) < 1e-12
    d = Driver(cfg, w, torch.float32)
    if where == "prompt":
        d.step([("a", t[:first - 1])]), d.step([("a", t[first - 1:])])
    else:
        d.step([("a", t[:first])])
        for x in t[first:]:
            d.step([("a", [x])])
    assert rel_err(d.result("a"), want) <= F32_TOL


def test_a_far_token_shows_in_logits(lib):
    """Replacing the very first token of a 300-token prompt changes the last row's logits of the plain model by far more
    than the tolerance, and the framework follows, the last row decoded alone after portions that end at and just after a
    page border.  The last token equals the first and keys are projected like the first head's queries, so that score is
    the largest there is; the scale makes it stand out among hundreds, and the bias of distance 0 keeps the last token from
    answering itself."""
    cfg = make_cfg([layer(None, heads=2, kv_heads=1, dim=48, vdim=16, scale=0.5, v_mix=False)])
    w = random_tensors(cfg, seed=11)
    w["l0.mix.k"], w["l0.mix.k.b"] = w["l0.mix.q"][:48].clone(), w["l0.mix.q.b"][:48].clone()
    w["l0.mix.rel"][0] = -40.0
    n = 300
    base = toks(n, cfg["vocab"] - 1, 5)
    base[-1] = cfg["vocab"] - 1
    t = list(base)
    t[0] = cfg["vocab"] - 1
    want, other = ref_logits(cfg, w, t), ref_logits(cfg, w, base)
    assert rel_err(want[-1:], other[-1:]) > 50 * F32_TOL
    d = Driver(cfg, w, torch.float32)
    d.step([("a", t[:64])]), d.step([("a", t[64:129])]), d.step([("a", t[129:n - 1])]), d.step([("a", t[n - 1:])])
    assert rel_err(d.result("a"), want) <= F32_TOL


def test_value_mixing_follows_the_first_mixing_layer(lib):
    """Values come from the first layer with v_mix (not from layer 0, not from the layer before), un-mixed and of the same
    token, in batches whose rows belong to several requests; the mixed values are what later steps find in the cache."""
    kw = dict(heads=4, kv_heads=2, dim=16, vdim=16)
    cfg = make_cfg([layer(None, v_mix=False, **kw), layer(dense_cfg(), **kw), layer(None, **kw), layer(None, v_mix=False, **kw),
                    layer(dense_cfg(24), **kw)])
    w = random_tensors(cfg, seed=6)
    a, b = toks(90, cfg["vocab"], 7), toks(70, cfg["vocab"], 8)
    wa, wb = ref_logits(cfg, w, a), ref_logits(cfg, w, b)
    for i in (0, 1, 4):                                               # other readings of the rule give other logits
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


def test_groups_decide_the_logits(lib):
    """A router whose groups are ranked by their two best members against one without groups: both agree with the plain
    model and differ from each other."""
    w, outs = None, []
    t = toks(60, 96, 3)
    for groups in ((3, 1), None):
        cfg = make_cfg([layer(moe_cfg(experts=6, top=2, groups=groups))])
        w = w or random_tensors(cfg, seed=9)
        d = Driver(cfg, w, torch.float32)
        d.step([("a", t)])
        assert rel_err(d.result("a"), ref_logits(cfg, w, t)) <= F32_TOL
        outs.append(d.result("a"))
    assert rel_err(outs[0], outs[1]) > 50 * F32_TOL


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
    """Sizes of one and values that coincide elsewhere: one head, as many key / value heads as query heads, a table of one
    or two buckets, an odd number of buckets, a range just above the linear half, one stream, one expert with top one, one
    group that is always kept, a feed-forward of one unit, no feed-forward at all, more streams than tokens."""
    for streams in (1, 7):
        cfg = make_cfg([layer(dense_cfg(1), heads=1, kv_heads=1, dim=2, vdim=130, scale=1.0, buckets=1, v_mix=False),
                        layer(moe_cfg(ff=1, experts=1, top=1, groups=(1, 1)), heads=1, kv_heads=1, dim=1, vdim=3, buckets=2, bias_max=2,
                              scale=2.0),
                        layer(None, heads=7, kv_heads=1, dim=130, vdim=3, buckets=7, bias_max=4),
                        layer(moe_cfg(ff=130, experts=5, top=5, groups=(5, 5)), heads=7, kv_heads=7, dim=8, v_mix=False,
                              buckets=9, bias_max=5)],
                       width=26, vocab=50, eps=1e-3, streams=streams, embed_scale=1.0)
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
            want.append(nxt)
            seq.append(nxt)
            if top2[1] - top2[0] < 1e-3:                              # a near tie may flip in fp32: stop comparing there
                break
        assert out[sid][:len(want)] == want
    assert eng.sched.num_free_state_slots == 5


# ------------------------------------------------------------------ random configurations under random schedules
@pytest.mark.parametrize("seed", [11, 12, 13, 14, 15, 16, 17, 18])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_random_configurations_under_random_schedules(lib, seed, dtype):
    """Sizes, layer orders and constants drawn at random (odd sizes, groups wider than an MMA tile, tables of 2 .. 48
    buckets over short and long ranges, routers with and without groups, 1 .. 6 streams); five requests of 5 .. 420 tokens
    share four state slots and just enough pages, so both are used again.  bf16 runs are compared at the 0.9 quantile of all
    requests' rows together: with 16-bit operands a near-tied expert choice can flip at single rows."""
    rng = np.random.default_rng(seed)
    pick = lambda *xs: xs[int(rng.integers(len(xs)))]              # noqa: E731
    cfg = make_cfg(random_layers(rng, int(rng.integers(2, 6))), width=pick(64, 128, 200), vocab=pick(300, 512),
                   eps=pick(1e-6, 1e-5), streams=pick(1, 2, 3, 4, 6), embed_scale=pick(0.3, 1.0, 2.0))
    w = random_tensors(cfg, seed=seed)
    reqs = {f"r{i}": toks(pick(5, 40, 150, 260, 420), cfg["vocab"], seed + i) for i in range(5)}
    pages = sum(sorted((len(v) + 63) // 64 for v in reqs.values())[-4:])
    d = Driver(cfg, w, dtype, num_blocks=pages, max_seqs=4, slots=4)
    for st, ends in random_schedule(rng, reqs):
        d.step(st)
        for k in ends:
            d.close(k)
    tol, q = bounds(dtype)
    want = {k: ref_logits(cfg, w, v) for k, v in reqs.items()}
    got, ref = np.concatenate([d.result(k) for k in reqs]), np.concatenate([want[k] for k in reqs])
    assert rel_err(got, ref, q) <= tol
    if dtype == torch.float32:
        for k in reqs:
            assert rel_err(d.result(k), want[k]) <= tol, k


# ------------------------------------------------------------------ a model folder through the command line
def _write_model_folder(path, cfg, tensors):
    """config.json and model.safetensors (8-byte little-endian header length, JSON header, raw data), bf16 tensors."""
    import json
    import struct
    header, blobs, at = {}, [], 0
    for name, t in tensors.items():
        raw = t.contiguous().view(torch.uint8).numpy().tobytes() if t.dtype != torch.bfloat16 else \
            t.contiguous().view(torch.int16).numpy().tobytes()
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
    import json
    import subprocess
    import sys
    from pathlib import Path
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
