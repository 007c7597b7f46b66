"""Throughput of the Sonalix decoder at layer sizes that resemble a real model (random weights), next to the closest
existing models of the framework at equal width, depth and expert sizes: the Gibevik decoder (grouped-head attention,
latent attention, routed experts) and the Fidasun decoder (latent attention, recurrent mixers, routed gated experts), all on
the same runner: `python bench.py --config sonalix`.

Per size: prefill tokens/s (one prompt of `prefill` tokens in one step) and decode tokens/s (`batch` sequences at
context `ctx`, one token each) of the three models, CUDA events after warm-up, and a table of the new design's kernels
timed alone at the same shapes (as replays of a CUDA graph of several calls, so that small kernels are not timed at the
rate of Python's launches) with their algorithmic bytes / flops against the measured copy bandwidth and cuBLAS bf16 peak
(the token-serial scans against the nominal fp32 FMA rate).  Every row is followed by a `like` row: the same kernel at the
same shape with the new options off, or the closest kernel of the other models."""
from __future__ import annotations

import numpy as np
import torch

from . import bench_gibevik, bench_hybrid, ops
from .bench_hybrid import _meta, _say, _time
from .rotary import rotary_frequencies

SIZES = {
    "w2048": dict(width=2048, vocab=32000, ff=5632,
                  attn=dict(heads=16, kv_heads=4, dim=128, vdim=128, window=1024, softcap=50.0),
                  latent=dict(heads=16, dim=64, rot_dim=32, vdim=64, kv_rank=256, q_rank=512),
                  ret=dict(heads=16, dim=128, vdim=128), moe=dict(experts=16, top=4, ff=512, limit=7.0)),
    "w4096": dict(width=4096, vocab=32000, ff=11008,
                  attn=dict(heads=32, kv_heads=8, dim=128, vdim=128, window=2048, softcap=50.0),
                  latent=dict(heads=32, dim=64, rot_dim=32, vdim=64, kv_rank=512, q_rank=1024),
                  ret=dict(heads=32, dim=128, vdim=128), moe=dict(experts=32, top=4, ff=1024, limit=7.0)),
}
ORDER = [("latent_attention", "dense"), ("attention", "moe"), ("retention", "moe"), ("attention", "moe")]


def config(size, layers):
    s = SIZES[size]
    a, la, re_, mo = s["attn"], s["latent"], s["ret"], s["moe"]
    mix = {"attention": dict(heads=a["heads"], kv_heads=a["kv_heads"], dim=a["dim"], vdim=a["vdim"], scale=a["dim"] ** -0.5,
                             softcap=a["softcap"], mask={"size": a["window"]}, v_mix=True,
                             rot={"base": 10000.0, "dims": a["dim"]}),
           "latent_attention": dict(heads=la["heads"], dim=la["dim"], rot_dim=la["rot_dim"], vdim=la["vdim"],
                                    kv_rank=la["kv_rank"], q_rank=la["q_rank"], scale=(la["dim"] + la["rot_dim"]) ** -0.5,
                                    rot={"base": 10000.0, "dims": la["rot_dim"]}),
           "retention": dict(heads=re_["heads"], dim=re_["dim"], vdim=re_["vdim"], rot={"base": 10000.0, "dims": re_["dim"]},
                             decay=[1.0 - 2.0 ** (-5 - h % 6) for h in range(re_["heads"])])}
    mlp = {"dense": {"kind": "dense", "ff": s["ff"]},
           "moe": {"kind": "moe", "expert": {"ff": mo["ff"], "limit": mo["limit"]},
                   "router": {"experts": mo["experts"], "top": mo["top"]}}}
    return {"architecture": "Sonalix", "width": s["width"], "vocab": s["vocab"], "norm": {"eps": 1e-6}, "residual_mult": 0.5,
            "embedding": {"scale": 4.0},
            "layers": [{"type": ORDER[i % 4][0], "mixer": mix[ORDER[i % 4][0]], "mlp": mlp[ORDER[i % 4][1]]} for i in range(layers)]}


def random_tensors(cfg, seed=0):
    g = torch.Generator().manual_seed(seed)
    D, out = cfg["width"], {}
    lin = lambda n, k: (torch.randn(n, k, generator=g) / k ** 0.5).to(torch.bfloat16)         # noqa: E731
    vec = lambda n, m=0.0, s=0.1: (m + s * torch.randn(n, generator=g)).to(torch.bfloat16)   # noqa: E731

    def norm(name):
        out[name], out[name + ".b"], out[name + ".alpha"] = vec(D, 1.0), vec(D), torch.tensor(0.7).to(torch.bfloat16)

    out["embed"], out["head"] = torch.randn(cfg["vocab"], D, generator=g).to(torch.bfloat16), lin(cfg["vocab"], D)
    norm("final.norm")
    for i, L in enumerate(cfg["layers"]):
        p, q, m = f"l{i}.", f"l{i}.mix.", L["mixer"]
        norm(p + "norm1"), norm(p + "norm2")
        H, dk, dv = m["heads"], m["dim"], m["vdim"]
        if L["type"] == "attention":
            G = m["kv_heads"]
            out.update({q + "q": lin(H * dk, D), q + "k": lin(G * dk, D), q + "v": lin(G * dv, D), q + "q.norm": vec(dk, 1.0),
                        q + "k.norm": vec(dk, 1.0), q + "sink": vec(H), q + "vmix": torch.tensor(0.5).to(torch.bfloat16)})
        elif L["type"] == "retention":
            out.update({q + "q": lin(H * dk, D), q + "k": lin(H * dk, D), q + "v": lin(H * dv, D), q + "g": lin(H * dv, D)})
        else:
            R, Q, dr = m["kv_rank"], m["q_rank"], m["rot_dim"]
            out.update({q + "dq": lin(Q, D), q + "dq.norm": vec(Q, 1.0), q + "uq": lin(H * (dk + dr), Q),
                        q + "dkv": lin(R + dr, D), q + "dkv.norm": vec(R, 1.0), q + "uk": lin(H * dk, R),
                        q + "uv": lin(H * dv, R), q + "g": lin(H * dv, D)})
        out[q + "o"] = lin(D, H * dv)
        mlp, q = L["mlp"], p + "mlp."
        if mlp["kind"] == "dense":
            F = mlp["ff"]
            out.update({q + "gate": lin(F, D), q + "up": lin(F, D), q + "down": lin(D, F)})
        else:
            E, F = mlp["router"]["experts"], mlp["expert"]["ff"]
            out.update({q + "router": lin(E, D), q + "router.b": vec(E)})
            for e in range(E):
                out.update({f"{q}e{e}.gate": lin(F, D), f"{q}e{e}.up": lin(F, D), f"{q}e{e}.down": lin(D, F)})
    return out


def _time_graph(fn, calls=8, reps=5):
    """ms per call: a CUDA graph of `calls` calls, replayed."""
    st = torch.cuda.Stream()
    st.wait_stream(torch.cuda.current_stream())
    with torch.cuda.stream(st):
        for _ in range(3):
            fn()
    torch.cuda.current_stream().wait_stream(st)
    graph = torch.cuda.CUDAGraph()
    with torch.cuda.graph(graph, stream=st):
        for _ in range(calls):
            fn()
    ms = _time(graph.replay, reps) / calls
    del graph
    return ms


def kernel_table(size, prefill, batch, ctx, peaks):
    """Each kernel of the design alone at the prefill shape (one sequence of `prefill` tokens) and the decode shape
    (`batch` sequences at context `ctx`): ms, achieved and the fraction of the bound it should sit on."""
    s, dev = SIZES[size], "cuda"
    hbm, tc = float(peaks["hbm_gbs"]) * 1e9, float(peaks["bf16_tflops"]) * 1e12
    fma = 148 * 128 * 2 * 1.9e9                      # fp32 FMA peak of the CUDA cores (nominal clocks)
    g = torch.Generator(device=dev).manual_seed(0)
    rnd = lambda *sh: torch.randn(*sh, generator=g, device=dev)          # noqa: E731
    i32 = lambda a: torch.tensor(a, dtype=torch.int32, device=dev)       # noqa: E731
    rows, D = [], s["width"]
    bf = torch.bfloat16

    def add(name, phase, fn, flops=0.0, nbytes=0.0, bound="hbm", note=""):
        ms = _time_graph(fn, 8 if phase == "decode" else 2)
        _say(f"{name} {phase}: {ms:.4f} ms")
        ach_f, ach_b = flops / (ms * 1e-3), nbytes / (ms * 1e-3)
        frac = {"hbm": ach_b / hbm, "tensor": ach_f / tc, "fp32": ach_f / fma}[bound]
        rows.append(dict(kernel=name, phase=phase, ms=round(ms, 4), tflops=round(ach_f / 1e12, 3),
                         gbs=round(ach_b / 1e9, 1), bound=bound, frac=round(frac, 4), note=note))

    for phase, B, q_len, cx_len in (("prefill", 1, prefill, prefill), ("decode", batch, 1, ctx)):
        T, nblk, dec = B * q_len, (cx_len + 63) // 64, phase == "decode"
        cu, cl = i32((np.arange(B + 1) * q_len).tolist()), i32([cx_len] * B)
        bt = i32(np.arange(B * nblk).reshape(B, nblk).tolist())
        slots = i32(list(range(B)))
        pos = torch.arange(cx_len - q_len, cx_len, device=dev).repeat(B)
        slot = ((torch.arange(B, device=dev) * nblk).repeat_interleave(q_len) + pos // 64) * 64 + pos % 64
        causal = sum(p + 1 for p in range(cx_len - q_len, cx_len)) * B
        # ---- attention: window, cap and a learned sink against window and cap with a gate per head
        a = s["attn"]
        H, G, dk, dv, W = a["heads"], a["kv_heads"], a["dim"], a["vdim"], a["window"]
        kc, vc = (rnd(B * nblk, 64, G, dk) * 0.3).to(bf), (rnd(B * nblk, 64, G, dv) * 0.3).to(bf)
        q, gate_h, sink = rnd(T, H, dk) * 0.3, rnd(T, H), rnd(H)
        seen = sum(min(p + 1, W) for p in range(cx_len - q_len, cx_len)) * B
        for name, sk, gt in (("attention (window, cap, learned sink)", sink, None),
                             ("like: attention (window, cap, head gate)", None, gate_h)):
            add(name, phase, lambda: ops.window_attn(q, kc, vc, sk, gt, cu, cl, bt, window=W, keep_first=0, scale=dk ** -0.5,
                                                     softcap=a["softcap"]),
                2.0 * H * seen * (dk + dv), seen * G * (dk + dv) * 2.0, "hbm" if dec else "tensor",
                "bytes = visible K and V rows, read once per key / value head" if dec else "mma.sync form")
        freq = torch.from_numpy(rotary_frequencies(dk, 10000.0)[0]).to(dev)
        proj, qn, kn, first = rnd(T, H * dk + G * (dk + dv)), rnd(dk), rnd(dk), rnd(T, G * dv)
        io = T * ((H * dk + G * (dk + dv)) * 4.0 + H * dk * 4.0 + G * (dk + dv) * 2.0)
        for name, kw, more in (("attention prep (head norms, two-halves rotary, mixed values)", dict(rot_half=True, v_mix=0.5, v_first=first), T * G * dv * 4.0),
                               ("like: attention prep (head norms, interleaved rotary)", {}, 0.0)):
            add(name, phase, lambda: ops.window_attn_prep(proj, None, qn, kn, freq, pos, slot, kc, vc, heads=H, rot_dims=dk,
                                                          eps=1e-6, head_norm=True, **kw), 0.0, io + more)
        del kc, vc, q, proj
        # ---- latent attention
        la = s["latent"]
        H, dn, dr, dv, R, Q = la["heads"], la["dim"], la["rot_dim"], la["vdim"], la["kv_rank"], la["q_rank"]
        cache = (rnd(B * nblk, 64, R + dr) * 0.3).to(bf)
        ql, gh = rnd(T, H, R + dr) * 0.1, rnd(T, H)
        for name, gt in (("latent attention (gate per element follows)", None), ("like: latent attention (head gate)", gh)):
            add(name, phase, lambda: ops.latent_attn(ql, cache, None, cu, cl, bt, kv_rank=R, rot_dim=dr, window=0, scale=0.1,
                                                     gate=gt),
                2.0 * H * causal * (2 * R + dr), causal * (R + dr) * 2.0, "hbm" if dec else "tensor",
                "bytes = visible cache rows, read once for all heads" if dec else "mma.sync form")
        fl = torch.from_numpy(rotary_frequencies(dr, 10000.0)[0]).to(dev)
        qx, low, wn = rnd(T, H * (dn + dr)), rnd(T, R + dr), rnd(R)
        both = torch.cat([qx, low], 1).contiguous()
        io = T * ((H * (dn + dr) + R + dr) * 4.0 + H * dn * 2.0 + H * dr * 4.0 + (R + dr) * 2.0)
        kw = dict(heads=H, dim=dn, rot_dim=dr, rot_dims=dr, kv_rank=R, eps=1e-6)
        add("latent prep (queries of a latent, two-halves rotary)", phase,
            lambda: ops.latent_prep_ex(qx, low, cache, wn, fl, 1.0, pos, slot, **kw), 0.0, io, note="ops clears q_full too")
        add("like: latent prep (one row, interleaved rotary)", phase,
            lambda: ops.latent_prep(both, cache, wn, fl, 1.0, pos, slot, **kw), 0.0, io, note="ops clears q_full too")
        wide, wq = rnd(T, Q + R + dr + H * dv), rnd(Q)
        add("norm of the query latent (rows of a wider row)", phase, lambda: ops.rmsnorm_rows(wide, Q, wq, 1e-6), 0.0, T * Q * 6.0)
        xq = rnd(T, Q)
        add("like: RMS norm of rows", phase, lambda: ops.resid_rmsnorm(xq, wq, 1e-6), 0.0, T * Q * 6.0)
        val, ge = rnd(T, H * dv), wide[:, Q + R + dr:].contiguous()
        add("gate per element, rounding", phase, lambda: ops.gate_rows(val, ge), 0.0, T * H * dv * 10.0)
        add("like: squared ReLU, rounding", phase, lambda: ops.ff_act(val, None, "relu2", dtype=bf), 0.0, T * H * dv * 6.0)
        del cache, ql, qx, low, both, wide
        # ---- retention
        r = s["ret"]
        H, dk, dv = r["heads"], r["dim"], r["vdim"]
        qk, fr = rnd(T, 2 * H * dk), torch.from_numpy(rotary_frequencies(dk, 10000.0)[0]).to(dev)
        add("rotary rows (q and k of the recurrence, in place)", phase,
            lambda: ops.rotary_rows(qk, fr, pos, heads=2 * H, dim=dk), 0.0, 2.0 * T * 2 * H * dk * 4.0)
        qr, kr, vr = rnd(T, H, dk), rnd(T, H, dk), rnd(T, H, dv)
        hd = 1.0 - torch.rand(H, device=dev) * 0.03
        chan = hd[None, :, None].expand(T, H, dk).contiguous()
        state = torch.zeros(B, H, dk, dv, device=dev)
        for name, kw in (("retention scan (decay per head)", dict(head_decay=hd, k_scale=dk ** -0.5)),
                         ("like: decayed scan (decay per key channel)", dict(chan_decay=chan))):
            add(name, phase, lambda: ops.decay_attn(qr, kr, vr, state, slots, cu, cl, **kw), 4.0 * T * H * dk * dv,
                B * H * dk * dv * 8.0, "hbm" if dec else "fp32",
                "bytes = state read + write; ops packs the rows first" if dec else "token-serial scan; ops packs the rows first")
        y, gg = rnd(T, H * dv), rnd(T, H * dv)
        add("head norm + SiLU gate (no weight)", phase, lambda: ops.gated_group_norm(y, gg, None, dv, 1e-6, False), 0.0, T * H * dv * 10.0)
        wv = rnd(dv)
        add("like: head norm + SiLU gate (weight)", phase, lambda: ops.gated_group_norm(y, gg, wv, dv, 1e-6, False), 0.0, T * H * dv * 10.0)
        del qk, qr, kr, vr, chan, state, y, gg
        # ---- router, experts, the norm that sums them
        mo = s["moe"]
        E, top, F = mo["experts"], mo["top"], mo["ff"]
        z, bias = rnd(T, E), rnd(E) * 0.1
        nb = T * (E * 4.0 + top * 8.0)
        add("router (softmax over the chosen logits)", phase, lambda: ops.moe_route_full(z, bias, top, score="chosen"), 0.0, nb)
        add("like: router (softmax over all)", phase, lambda: ops.moe_route(z, top, 1.0), 0.0, nb)
        h = (rnd(T, D) * 0.5).to(bf)
        gu, dn_ = (rnd(E, 2 * F, D) / D ** 0.5).to(bf), (rnd(E, D, F) / F ** 0.5).to(bf)
        idx, w = ops.moe_route_full(z, bias, top, score="chosen")
        hit = int(torch.unique(idx).numel())
        flops, wb = 6.0 * T * top * F * D, hit * 3.0 * F * D * 2.0
        note = "bytes = weights of the experts hit" if dec else "mma.sync grouped GEMM"
        xo = torch.zeros(T, D, device=dev)
        add("experts (clamped gate, rows left unsummed)", phase,
            lambda: ops.moe_experts_rows(h, idx, gu, dn_, act="clamped", limit=mo["limit"], alpha=1.702, up_add=1.0), flops, wb,
            "hbm" if dec else "tensor", note)
        add("like: experts (SiLU gate, summed)", phase, lambda: ops.moe_experts(xo, h, idx, w, gu, dn_), flops, wb,
            "hbm" if dec else "tensor", note)
        x1, er, wn, bn = rnd(1, T, D), rnd(T * top, D), rnd(D), rnd(D)
        sl = torch.randperm(T * top, device=dev).to(torch.int32)
        add("dynamic-tanh norm + sum of the experts' rows", phase,
            lambda: ops.hyper_step(x1, experts=(er, sl, w), w=wn, bias=bn, kind="dyntanh", alpha=0.7, dtype=bf), 0.0,
            T * D * (top * 4.0 + 8.0 + 2.0))
        y1 = er[:T].contiguous()
        add("like: RMS norm + residual sum", phase, lambda: ops.resid_add_rmsnorm(x1[0], y1, wn, 1e-6), 0.0, T * D * 12.0)
        add("dynamic-tanh norm", phase, lambda: ops.stream_norm(x1[0], wn, bn, kind="dyntanh", alpha=0.7, dtype=bf), 0.0, T * D * 6.0)
        add("like: RMS norm of the stream", phase, lambda: ops.resid_rmsnorm(x1[0], wn, 1e-6), 0.0, T * D * 6.0)
        del h, gu, dn_, xo, x1, er
        torch.cuda.empty_cache()
    return rows


def run(size="w2048", layers=4, prefill=4096, batch=32, ctx=2048, reps=5):
    import json
    from pathlib import Path

    from . import models
    pk = Path(__file__).resolve().parent.parent / "MEASURED_PEAKS.json"
    peaks = json.loads(pk.read_text()) if pk.exists() else {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0}
    s = SIZES[size]
    res = {"size": size, "layers": layers, "order": [f"{m} + {f}" for m, f in ORDER[:layers]], "prefill_tokens": prefill,
           "decode_batch": batch, "decode_context": ctx}
    nblk = (max(prefill, ctx) + 63) // 64
    mp, md = _meta(1, prefill, prefill, nblk, s["vocab"]), _meta(batch, 1, ctx, nblk, s["vocab"])
    arms = (("sonalix", config(size, layers), random_tensors),
            ("gibevik", bench_gibevik.config(size, layers), bench_gibevik.random_tensors),
            ("fidasun", bench_hybrid.config(size, layers), bench_hybrid.random_tensors))
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
