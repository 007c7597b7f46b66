"""Small Zufulix configurations with random weights.  Test infrastructure; the driver that feeds portions through the
scheduler and the runner is fidasun_util.Driver, the random schedules come from zalalix_util.random_schedule (both are
model-agnostic)."""
from __future__ import annotations

import torch


def attn_cfg(**kw):
    """`buckets` (rows of the bias table) is read by random_tensors only; the model file reads the tensor's shape."""
    m = dict(heads=6, kv_heads=2, dim=24, vdim=20, scale=0.3, bias_max=50, v_mix=True, buckets=12)
    m.update(kw)
    return m


def dense_cfg(ff=56):
    return {"kind": "dense", "ff": ff}


def moe_cfg(ff=24, experts=12, top=4, groups=(4, 2)):
    r = dict(experts=experts, top=top)
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": r}


def layer(mlp=None, **kw):
    return {"type": "attention", "mixer": attn_cfg(**kw), "mlp": mlp}


def make_cfg(layers, width=48, vocab=96, eps=1e-5, streams=3, embed_scale=0.7):
    return {"architecture": "Zufulix", "width": width, "vocab": vocab, "streams": streams, "norm": {"eps": eps},
            "embedding": {"scale": embed_scale}, "layers": layers}


def full_cfg(**kw):
    """Every feed-forward kind, a first layer that does not mix values, sizes pairwise different."""
    return make_cfg([layer(dense_cfg(), v_mix=False, heads=4, kv_heads=4, dim=16, vdim=32, buckets=8, bias_max=30),
                     layer(moe_cfg()),
                     layer(moe_cfg(ff=40, experts=5, top=2, groups=None), heads=2, dim=32, scale=0.2, bias_max=140, buckets=32),
                     layer(None, v_mix=False, heads=3, kv_heads=1, dim=40, vdim=16),
                     layer(dense_cfg(40), heads=8, dim=16, bias_max=16, buckets=20)], **kw)


def random_tensors(cfg, seed=0):
    """name -> CPU tensor; everything is bf16 (exact in both operand dtypes)."""
    g = torch.Generator().manual_seed(seed)
    D, S, out = cfg["width"], cfg["streams"], {}

    def lin(n, k, gain=1.0):
        return (torch.randn(n, k, generator=g) * gain / k ** 0.5).to(torch.bfloat16)

    def vec(n, mean=0.0, std=0.2):
        return (mean + std * torch.randn(n, generator=g)).to(torch.bfloat16)

    def norm(name):
        out[name], out[name + ".b"] = vec(D, 1.0, 0.3), vec(D, 0.0, 0.2)

    def connection(name):                 # every stream keeps most of itself, takes some of the others and some of y
        out[name + ".in"] = vec(S, 1.0 / S, 0.4)
        out[name + ".mix"] = (0.8 * torch.eye(S) + 0.25 * torch.randn(S, S, generator=g) / S ** 0.5).to(torch.bfloat16)
        out[name + ".out"] = vec(S, 0.7, 0.4)

    out["embed"] = torch.randn(cfg["vocab"], D, generator=g).to(torch.bfloat16)
    norm("final.norm")
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        norm(p + "norm1"), connection(p + "hc1")
        H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        q = p + "mix."
        for n, rows in (("q", H * dk), ("k", G * dk), ("v", G * dv)):
            out[q + n], out[q + n + ".b"] = lin(rows, D, 2.0), vec(rows, 0.0, 0.5)
        out[q + "rel"] = vec(m["buckets"] * H, 0.0, 1.0).reshape(m["buckets"], H)
        if m.get("v_mix"):
            out[q + "vmix"] = (0.2 + 0.6 * torch.rand((), generator=g)).to(torch.bfloat16)
        out[q + "o"] = lin(D, H * dv)
        mlp = L.get("mlp")
        if not mlp:
            continue
        norm(p + "norm2"), connection(p + "hc2")
        q = p + "mlp."
        if mlp["kind"] == "dense":
            out[q + "up"], out[q + "down"] = lin(mlp["ff"], D, 2.0), lin(D, mlp["ff"], 2.0)
        else:
            E, F = mlp["router"]["experts"], mlp["expert"]["ff"]
            out[q + "router"] = lin(E, D, 2.0)
            for e in range(E):
                out[f"{q}e{e}.up"], out[f"{q}e{e}.down"] = lin(F, D, 2.0), lin(D, F, 2.0)
    return out


def random_layers(rng, count):
    """`count` layers drawn at random; the layers that mix values have the same kv_heads and vdim."""
    pick = lambda *xs: xs[int(rng.integers(len(xs)))]              # noqa: E731
    layers, shared = [], (pick(1, 2, 3), pick(8, 16, 32, 50, 96, 128))
    for _ in range(count):
        mix = rng.random() < 0.65
        G, dv = shared if mix else (pick(1, 2, 3), pick(8, 16, 20, 32, 64, 144))
        B = pick(2, 4, 7, 16, 32, 48)
        m = dict(heads=G * pick(1, 2, 4, 9, 17), kv_heads=G, dim=pick(8, 16, 32, 40, 80), vdim=dv, scale=pick(0.125, 0.3),
                 bias_max=B // 2 + pick(1, 9, 40, 200, 3000), v_mix=bool(mix), buckets=B)
        r = rng.random()
        if r < 0.2:
            mlp = None
        elif r < 0.5:
            mlp = dense_cfg(pick(1, 24, 64, 100))
        else:
            groups = pick(None, (1, 1), (2, 1), (3, 2), (4, 3))
            per = pick(1, 2, 3, 5)
            E = per * groups[0] if groups else pick(1, 3, 8, 40)
            mlp = moe_cfg(ff=pick(8, 40, 72), experts=E, top=min(pick(1, 2, 3), per * groups[1] if groups else E), groups=groups)
        layers.append({"type": "attention", "mixer": m, "mlp": mlp})
    return layers
