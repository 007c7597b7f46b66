"""Throughput of the Zufulix decoder at layer sizes that resemble a real model (random weights), next to the closest
existing model of the framework, the Gibevik decoder (grouped-head attention with a distance bias, squared-ReLU experts
behind a router with groups, on the same runner), at equal width, depth, head counts and expert sizes:
`python bench.py --config zufulix`.

Per size: prefill tokens/s (one prompt of `prefill` tokens in one step) and decode tokens/s (`batch` sequences at
context `ctx`, one token each) of both models, CUDA events after warm-up, and a table of the new design's kernels timed
alone at the same shapes with their algorithmic bytes / flops against the measured copy bandwidth and cuBLAS bf16 peak.
Every row of a kernel that gained an option is followed by a `like` row: the same kernel at the same shape as the closest
model uses it, or the closest model's kernel for the same job."""
from __future__ import annotations

import numpy as np
import torch

from . import bench_gibevik, ops
from .bench_hybrid import _meta, _say, _time
from .models.gibevik import head_slopes
from .models.zufulix import distance_table

SIZES = {
    "w2048": dict(width=2048, vocab=32000, streams=4, ff=8448, attn=dict(heads=16, kv_heads=4, dim=128, buckets=32, far=128),
                  moe=dict(experts=16, top=4, ff=1024, groups=4, keep=2)),
    "w4096": dict(width=4096, vocab=32000, streams=4, ff=16512, attn=dict(heads=32, kv_heads=8, dim=128, buckets=32, far=128),
                  moe=dict(experts=32, top=4, ff=1024, groups=4, keep=2)),
}
MOE_FROM = 1                              # the first layer has a dense feed-forward, the others routed experts


def config(size, layers):
    s = SIZES[size]
    a, mo = s["attn"], s["moe"]
    mixer = dict(heads=a["heads"], kv_heads=a["kv_heads"], dim=a["dim"], vdim=a["dim"], scale=a["dim"] ** -0.5,
                 bias_max=a["far"], v_mix=True)
    moe = {"kind": "moe", "expert": {"ff": mo["ff"]},
           "router": {"experts": mo["experts"], "top": mo["top"], "groups": {"count": mo["groups"], "keep": mo["keep"]}}}
    return {"architecture": "Zufulix", "width": s["width"], "vocab": s["vocab"], "streams": s["streams"],
            "norm": {"eps": 1e-6}, "embedding": {"scale": 1.0},
            "layers": [{"type": "attention", "mixer": mixer, "mlp": moe if i >= MOE_FROM else {"kind": "dense", "ff": s["ff"]}}
                       for i in range(layers)]}


def like_config(size, layers):
    """Gibevik layers of the same head counts, expert sizes and dense feed-forward parameters (its dense form is gated)."""
    s = SIZES[size]
    a, mo = s["attn"], s["moe"]
    mixer = dict(heads=a["heads"], kv_heads=a["kv_heads"], dim=a["dim"], vdim=a["dim"], scale=a["dim"] ** -0.5,
                 q_temp={"coef": 0.1, "every": 512})
    moe = {"kind": "moe", "expert": {"ff": mo["ff"]}, "shared": None,
           "router": {"experts": mo["experts"], "identity": 0, "top": mo["top"],
                      "groups": {"count": mo["groups"], "keep": mo["keep"]}}}
    return {"architecture": "Gibevik", "width": s["width"], "vocab": s["vocab"], "norm": {"eps": 1e-6},
            "layers": [{"type": "attention", "mixer": mixer,
                        "mlp": moe if i >= MOE_FROM else {"kind": "dense", "ff": s["ff"] * 2 // 3}} for i in range(layers)]}


def random_tensors(cfg, seed=0):
    g = torch.Generator().manual_seed(seed)
    D, S, out = cfg["width"], cfg["streams"], {}
    lin = lambda n, k: (torch.randn(n, k, generator=g) / k ** 0.5).to(torch.bfloat16)         # noqa: E731
    vec = lambda n, m=0.0, s=0.1: (m + s * torch.randn(n, generator=g)).to(torch.bfloat16)   # noqa: E731

    def norm(name):
        out[name], out[name + ".b"] = vec(D, 1.0), vec(D)

    out["embed"] = (torch.randn(cfg["vocab"], D, generator=g) / D ** 0.5).to(torch.bfloat16)
    norm("final.norm")
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        for k in ("1", "2"):
            norm(p + "norm" + k)
            out[p + f"hc{k}.in"], out[p + f"hc{k}.out"] = vec(S, 1.0 / S), vec(S, 1.0)
            out[p + f"hc{k}.mix"] = (torch.eye(S) + 0.05 * torch.randn(S, S, generator=g)).to(torch.bfloat16)
        H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        for n, rows in (("q", H * dk), ("k", G * dk), ("v", G * dv)):
            out[p + "mix." + n], out[p + f"mix.{n}.b"] = lin(rows, D), vec(rows)
        buckets = next(s["attn"]["buckets"] for s in SIZES.values() if s["width"] == D)
        out[p + "mix.rel"] = vec(buckets * H).reshape(buckets, H)
        out[p + "mix.vmix"], out[p + "mix.o"] = torch.tensor(0.5, dtype=torch.bfloat16), lin(D, H * dv)
        mlp, q = L["mlp"], p + "mlp."
        if mlp["kind"] == "dense":
            out[q + "up"], out[q + "down"] = lin(mlp["ff"], D), lin(D, mlp["ff"])
        else:
            E, F = mlp["router"]["experts"], mlp["expert"]["ff"]
            out[q + "router"] = lin(E, D)
            for e in range(E):
                out[f"{q}e{e}.up"], out[f"{q}e{e}.down"] = lin(F, D), lin(D, F)
    return out


def kernel_table(size, prefill, batch, ctx, peaks):
    """Each kernel of the design alone at the prefill shape (one sequence of `prefill` tokens) and the decode shape
    (`batch` sequences at context `ctx`): ms, achieved and the fraction of the bound it should sit on."""
    s, dev = SIZES[size], "cuda"
    hbm, tc = float(peaks["hbm_gbs"]) * 1e9, float(peaks["bf16_tflops"]) * 1e12
    g = torch.Generator(device=dev).manual_seed(0)
    rnd = lambda *sh: torch.randn(*sh, generator=g, device=dev)          # noqa: E731
    i32 = lambda a: torch.tensor(a, dtype=torch.int32, device=dev)       # noqa: E731
    rows = []

    def add(name, phase, ms, flops=0.0, nbytes=0.0, bound="hbm", note=""):
        _say(f"{name} {phase}: {ms:.3f} ms")
        ach_f, ach_b = flops / (ms * 1e-3), nbytes / (ms * 1e-3)
        frac = {"hbm": ach_b / hbm, "tensor": ach_f / tc}[bound]
        rows.append(dict(kernel=name, phase=phase, ms=round(ms, 4), tflops=round(ach_f / 1e12, 3),
                         gbs=round(ach_b / 1e9, 1), bound=bound, frac=round(frac, 4), note=note))

    D, S = s["width"], s["streams"]
    for phase, B, q_len, cx_len in (("prefill", 1, prefill, prefill), ("decode", batch, 1, ctx)):
        T, nblk = B * q_len, (cx_len + 63) // 64
        cu, cl = i32((np.arange(B + 1) * q_len).tolist()), i32([cx_len] * B)
        bt = i32(np.arange(B * nblk).reshape(B, nblk).tolist())
        keys = sum(p + 1 for p in range(cx_len - q_len, cx_len)) * B            # full causal context
        a = s["attn"]
        H, G, dk = a["heads"], a["kv_heads"], a["dim"]
        kc = (rnd(B * nblk, 64, G, dk) * 0.3).to(torch.bfloat16)
        vc = (rnd(B * nblk, 64, G, dk) * 0.3).to(torch.bfloat16)
        q, gate, slopes = rnd(T, H, dk) * 0.3, rnd(T, H * dk), head_slopes(H).to(dev)
        table = distance_table(rnd(a["buckets"], H).cpu(), a["far"]).to(dev)
        for name, kw in (("attention (learned distance bias)", dict(gate=None, dist_bias=table)),
                         ("like: attention (linear distance bias, element gate)", dict(gate=gate, dist_slopes=slopes)),
                         ("like: attention (no bias)", dict(gate=None))):
            ms = _time(lambda: ops.window_attn(q, kc, vc, None, kw["gate"], cu, cl, bt, window=0, keep_first=0,
                                               scale=dk ** -0.5, dist_slopes=kw.get("dist_slopes"),
                                               dist_bias=kw.get("dist_bias")), 5)
            if phase == "decode":
                add(name, phase, ms, 4.0 * H * keys * dk, keys * G * dk * 4.0, "hbm",
                    "bytes = visible K and V rows, read once per key / value head")
            else:
                add(name, phase, ms, 4.0 * H * keys * dk, 0.0, "tensor", "mma.sync form")
        n_in = (H + 2 * G) * dk
        proj, bias, qn, kn, first = rnd(T, n_in), rnd(n_in), rnd(dk), rnd(dk), rnd(T, G * dk)
        pos = torch.arange(cx_len - q_len, cx_len, device=dev).repeat(B)
        slot = ((torch.arange(B, device=dev) * nblk).repeat_interleave(q_len) + pos // 64) * 64 + pos % 64
        nb = T * (n_in * 4.0 + H * dk * 4.0 + 2 * G * dk * 2.0)
        ms = _time(lambda: ops.window_attn_prep(proj, bias, None, None, None, pos, slot, kc, vc, heads=H, rot_dims=0,
                                                eps=1e-6, head_norm=2, v_mix=0.5, v_first=first), 10)
        add("attention prep (biases, weightless head norms, mixed values)", phase, ms, 0.0, nb + T * G * dk * 4.0)
        ms = _time(lambda: ops.window_attn_prep(proj, None, qn, kn, None, pos, slot, kc, vc, heads=H, rot_dims=0,
                                                eps=1e-6, head_norm=True), 10)
        add("like: attention prep (weighted head norms)", phase, ms, 0.0, nb)
        del kc, vc, q, proj, gate
        # hyper-connected streams
        x, y, w, b = rnd(S, T, D), rnd(T, D), rnd(D), rnd(D)
        kw = dict(mix=rnd(S, S), out_w=rnd(S), in_w=rnd(S), w=w, bias=b, dtype=torch.bfloat16)
        mo = s["moe"]
        E, top, F = mo["experts"], mo["top"], mo["ff"]
        ms = _time(lambda: ops.hyper_step(x, y=y, **kw), 10)
        add(f"hyper step ({S} streams: update, read, layer norm)", phase, ms, 0.0, T * D * ((2 * S + 1) * 4.0 + 2.0))
        xs, h1 = y.clone(), rnd(T, D)
        ms = _time(lambda: ops.resid_add_rmsnorm(xs, h1, w, 1e-6), 10)
        add("like: norm + residual sum of one stream", phase, ms, 0.0, T * D * 12.0)
        ms = _time(lambda: ops.stream_norm(xs, w, b, kind="rms", dtype=torch.bfloat16), 10)
        add("like: RMS norm of one stream", phase, ms, 0.0, T * D * 6.0)
        er, sl = rnd(T * top, D), torch.randperm(T * top, generator=g, device=dev).to(torch.int32)
        tw = torch.rand(T, top, generator=g, device=dev)
        ms = _time(lambda: ops.hyper_step(x, experts=(er, sl, tw), **kw), 10)
        add(f"hyper step ({S} streams, sum of {top} expert rows)", phase, ms, 0.0, T * D * ((2 * S + top) * 4.0 + 2.0))
        ms = _time(lambda: ops.hyper_step(y, equal_streams=S, in_w=kw["in_w"], w=w, bias=b, dtype=torch.bfloat16), 10)
        add("hyper step (first read: equal streams)", phase, ms, 0.0, T * D * 6.0)
        del x, y, er, xs, h1
        # router, experts, activation
        z = rnd(T, E)
        ms = _time(lambda: ops.moe_route_full(z, None, top, 1.0, mo["groups"], mo["keep"], score="sigmoid", group_top=2,
                                              renorm=True), 10)
        add("router (sigmoid, group sums, normalised weights)", phase, ms, 0.0, T * (E * 4.0 + top * 8.0))
        ms = _time(lambda: ops.moe_route_ex(z, None, top, 1.0, mo["groups"], mo["keep"]), 10)
        add("like: router (softmax, groups)", phase, ms, 0.0, T * (E * 4.0 + top * 8.0))
        h = (rnd(T, D) * 0.5).to(torch.bfloat16)
        up = (rnd(E, F, D) / D ** 0.5).to(torch.bfloat16)
        dn = (rnd(E, D, F) / F ** 0.5).to(torch.bfloat16)
        idx, wt = ops.moe_route_full(z, None, top, 1.0, mo["groups"], mo["keep"], score="sigmoid", group_top=2, renorm=True)
        hit, xo = int(torch.unique(idx).numel()), torch.zeros(T, D, device=dev)
        for name, fn in (("experts (squared ReLU, rows left unsummed)", lambda: ops.moe_experts_rows(h, idx, up, dn, act="relu2")),
                         ("like: experts (squared ReLU, summed)",
                          lambda: ops.moe_experts_ex(xo, h, idx, wt, up, dn, act="relu2", accumulate=False))):
            ms = _time(fn, 5)
            if phase == "decode":
                add(name, phase, ms, 4.0 * T * top * F * D, hit * 2.0 * F * D * 2, "hbm", "bytes = weights of the experts hit")
            else:
                add(name, phase, ms, 4.0 * T * top * F * D, 0.0, "tensor", "mma.sync grouped GEMM")
        del h, up, dn
        upf = rnd(T, s["ff"])
        for name, act in (("GELU", "gelu"), ("like: squared ReLU", "relu2")):
            ms = _time(lambda: ops.ff_act(upf, None, act, dtype=torch.bfloat16), 10)
            add(name, phase, ms, 0.0, T * s["ff"] * 6.0)
        del upf
        torch.cuda.empty_cache()
    return rows


def run(size="w2048", layers=4, prefill=4096, batch=32, ctx=2048, reps=5):
    import json
    from pathlib import Path

    from . import models
    pk = Path(__file__).resolve().parent.parent / "MEASURED_PEAKS.json"
    peaks = json.loads(pk.read_text()) if pk.exists() else {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0}
    s = SIZES[size]
    res = {"size": size, "layers": layers, "prefill_tokens": prefill, "decode_batch": batch, "decode_context": ctx}
    nblk = (max(prefill, ctx) + 63) // 64
    mp, md = _meta(1, prefill, prefill, nblk, s["vocab"]), _meta(batch, 1, ctx, nblk, s["vocab"])
    arms = (("zufulix", config(size, layers), random_tensors),
            ("gibevik", like_config(size, layers), bench_gibevik.random_tensors))
    for name, cfg, make in arms:
        r = models.build_runner(cfg, make(cfg), dtype=torch.bfloat16, device="cuda", num_blocks=batch * nblk,
                                max_blocks_per_seq=nblk, max_seqs=batch, max_tokens=max(prefill, batch),
                                num_state_slots=batch)
        for c in list(r.kv_cache.values()) + list(r.v_cache.values()):
            c.normal_(std=0.3)
        ms = _time(lambda: r.step(mp, [prefill - 1]), 1, warm=1)
        ms = _time(lambda: r.step(mp, [prefill - 1]), reps, warm=1)
        res[name] = {"prefill_ms": ms, "prefill_tok_s": prefill * 1e3 / ms, "launches": int(r.launches_per_step)}
        ms = _time(lambda: r.step(md, list(range(batch))), reps * 4, warm=3)
        res[name].update(decode_ms=ms, decode_tok_s=batch * 1e3 / ms)
        _say(f"{name}: {res[name]}")
        del r
        torch.cuda.empty_cache()
    res["kernels"] = kernel_table(size, prefill, batch, ctx, peaks)
    return res
