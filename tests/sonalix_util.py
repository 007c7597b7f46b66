"""Small Sonalix configurations with random weights.  Test infrastructure; the driver that feeds portions through the
scheduler and the runner is fidasun_util.Driver, the random schedules come from zalalix_util.random_schedule (both are
model-agnostic)."""
from __future__ import annotations

import torch


def attn_cfg(**kw):
    m = dict(heads=6, kv_heads=2, dim=24, vdim=20, scale=0.3, softcap=20.0, rot={"base": 3000.0, "dims": 16},
             mask={"size": 37}, v_mix=True)
    m.update(kw)
    return m


def ret_cfg(**kw):
    m = dict(heads=4, dim=24, vdim=40, rot={"base": 7000.0, "dims": 12}, decay=[0.5, 0.96875, 0.9921875, 1.0])
    m.update(kw)
    return m


def latent_cfg(**kw):
    """rot.dims always equals rot_dim: only `rot_dim` and `base` are given."""
    m = dict(heads=5, dim=20, rot_dim=8, vdim=28, kv_rank=36, q_rank=44, scale=0.25, base=900.0)
    m.update(kw)
    m["rot"] = {"base": m.pop("base"), "dims": m["rot_dim"]}
    return m


def dense_cfg(ff=56):
    return {"kind": "dense", "ff": ff}


def moe_cfg(ff=24, experts=7, top=3, limit=0.8):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}


def layer(kind, mlp=None, **kw):
    m = {"attention": attn_cfg, "retention": ret_cfg, "latent_attention": latent_cfg}[kind](**kw)
    return {"type": kind, "mixer": m, "mlp": mlp}


def make_cfg(layers, width=48, vocab=96, eps=1e-5, mult=0.7, embed_scale=1.5):
    return {"architecture": "Sonalix", "width": width, "vocab": vocab, "norm": {"eps": eps}, "residual_mult": mult,
            "embedding": {"scale": embed_scale}, "layers": layers}


def full_cfg(**kw):
    """Every mixer and feed-forward kind, a first attention that does not mix values, experts at the end, in the middle and
    before a layer without a feed-forward; sizes pairwise different."""
    return make_cfg([layer("attention", dense_cfg(), v_mix=False, heads=4, kv_heads=4, dim=16, vdim=32, mask={"size": 64}),
                     layer("latent_attention", moe_cfg()),
                     layer("attention", moe_cfg(ff=40, experts=5, top=1, limit=2.0)),
                     layer("retention", None),
                     layer("attention", dense_cfg(40), heads=2, dim=32, scale=0.2, softcap=5.0,
                           rot={"base": 500.0, "dims": 32}, mask={"size": 5}),
                     layer("retention", moe_cfg(ff=16, experts=9, top=4), heads=2, dim=16, vdim=24, decay=[0.75, 0.998046875],
                           rot={"base": 100.0, "dims": 16}),
                     layer("latent_attention", moe_cfg(), heads=3, dim=12, rot_dim=4, vdim=16, kv_rank=24, q_rank=52)], **kw)


def random_tensors(cfg, seed=0):
    """name -> CPU tensor; everything is bf16 (exact in both operand dtypes)."""
    g = torch.Generator().manual_seed(seed)
    D, out = cfg["width"], {}

    def lin(n, k, gain=1.0):
        return (torch.randn(n, k, generator=g) * gain / k ** 0.5).to(torch.bfloat16)

    def vec(n, mean=0.0, std=0.2):
        return (mean + std * torch.randn(n, generator=g)).to(torch.bfloat16)

    def norm(name):
        out[name], out[name + ".b"] = vec(D, 1.0, 0.3), vec(D, 0.0, 0.2)
        out[name + ".alpha"] = (0.4 + 0.6 * torch.rand((), generator=g)).to(torch.bfloat16)

    out["embed"], out["head"] = torch.randn(cfg["vocab"], D, generator=g).to(torch.bfloat16), lin(cfg["vocab"], D)
    norm("final.norm")
    for i, L in enumerate(cfg["layers"]):
        p, q, m = f"l{i}.", f"l{i}.mix.", L["mixer"]
        norm(p + "norm1")
        H, dk, dv = m["heads"], m["dim"], m["vdim"]
        if L["type"] == "attention":
            G = m["kv_heads"]
            for n, rows in (("q", H * dk), ("k", G * dk), ("v", G * dv)):
                out[q + n] = lin(rows, D, 2.0)
            out[q + "q.norm"], out[q + "k.norm"], out[q + "sink"] = vec(dk, 1.0, 0.3), vec(dk, 1.0, 0.3), vec(H, 0.5, 1.0)
            if m.get("v_mix"):
                out[q + "vmix"] = (0.2 + 0.6 * torch.rand((), generator=g)).to(torch.bfloat16)
        elif L["type"] == "retention":
            for n, rows in (("q", H * dk), ("k", H * dk), ("v", H * dv), ("g", H * dv)):
                out[q + n] = lin(rows, D, 2.0)
        else:
            R, Q, dr = m["kv_rank"], m["q_rank"], m["rot_dim"]
            out.update({q + "dq": lin(Q, D, 2.0), q + "dq.norm": vec(Q, 1.0, 0.3), q + "uq": lin(H * (dk + dr), Q),
                        q + "dkv": lin(R + dr, D, 2.0), q + "dkv.norm": vec(R, 1.0, 0.3), q + "uk": lin(H * dk, R),
                        q + "uv": lin(H * dv, R), q + "g": lin(H * dv, D)})
        out[q + "o"] = lin(D, H * dv)
        mlp = L.get("mlp")
        if not mlp:
            continue
        norm(p + "norm2")
        q = p + "mlp."
        if mlp["kind"] == "dense":
            F = mlp["ff"]
            out[q + "gate"], out[q + "up"], out[q + "down"] = lin(F, D, 2.0), lin(F, D, 2.0), lin(D, F)
        else:
            E, F = mlp["router"]["experts"], mlp["expert"]["ff"]
            out[q + "router"], out[q + "router.b"] = lin(E, D, 2.0), vec(E, 0.0, 0.7)
            for e in range(E):
                out[f"{q}e{e}.gate"], out[f"{q}e{e}.up"], out[f"{q}e{e}.down"] = lin(F, D, 2.0), lin(F, D, 2.0), lin(D, F)
    return out


def random_layers(rng, count):
    """`count` layers drawn at random; the layers that mix values have the same kv_heads and vdim."""
    pick = lambda *xs: xs[int(rng.integers(len(xs)))]              # noqa: E731
    layers, shared = [], (pick(1, 2, 3), pick(8, 16, 32, 50, 96, 128))
    for _ in range(count):
        kind = pick("attention", "attention", "retention", "latent_attention")
        if kind == "attention":
            mix = bool(rng.random() < 0.65)
            G, dv = shared if mix else (pick(1, 2, 3), pick(8, 16, 20, 32, 64, 144))
            dk = pick(8, 16, 32, 40, 80)
            kw = dict(heads=G * pick(1, 2, 4, 9, 17), kv_heads=G, dim=dk, vdim=dv, scale=pick(0.125, 0.3), softcap=pick(3.0, 30.0),
                      rot={"base": pick(100.0, 1e4, 1e6), "dims": pick(2, 4, dk)}, mask={"size": pick(1, 2, 17, 64, 65, 200)},
                      v_mix=mix)
        elif kind == "retention":
            H, dk = pick(1, 2, 3, 5), pick(8, 16, 24, 40, 64, 130)
            kw = dict(heads=H, dim=dk, vdim=pick(8, 16, 20, 48, 80), rot={"base": pick(100.0, 1e4, 1e6), "dims": pick(2, 8, dk)},
                      decay=[float(pick(0.5, 0.96875, 0.9921875, 0.9990234375, 1.0)) for _ in range(H)])
        else:
            kw = dict(heads=pick(1, 2, 5, 17), dim=pick(8, 12, 32, 48), rot_dim=pick(2, 8, 16, 64), vdim=pick(8, 20, 32, 64),
                      kv_rank=pick(12, 40, 64, 128), q_rank=pick(16, 40, 100), scale=pick(0.125, 0.3), base=pick(100.0, 1e4, 1e6))
        r = rng.random()
        if r < 0.2:
            mlp = None
        elif r < 0.5:
            mlp = dense_cfg(pick(1, 24, 64, 100))
        else:
            E = pick(1, 3, 8, 40)
            mlp = moe_cfg(ff=pick(8, 40, 72), experts=E, top=min(pick(1, 2, 3), E), limit=pick(0.5, 1.0, 7.0))
        layers.append(layer(kind, mlp, **kw))
    return layers
