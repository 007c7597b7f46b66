"""A plain, slow restatement of the Sonalix decoder in double precision, one function per mechanism.  It shares no code
with the product path (vllm_rs_b200/models/sonalix.py arranges weights for CUDA kernels; this file multiplies them out on
the CPU) and is what the GPU tests compare the framework with.

Notation: T tokens at positions 0 .. T-1, the stream X [T, D] starts as the scaled embedding rows, and every sublayer F
(mixer, then feed-forward) adds  c F(N(X))  with one factor c and a dynamic-tanh norm N(x) = tanh(a x) w + b.  The logits
are H N_f(X)."""
from __future__ import annotations

import math

import torch

D64 = torch.float64


def dynamic_tanh(x, W, name):
    return torch.tanh(W[name + ".alpha"] * x) * W[name] + W[name + ".b"]


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def turn(x, dims, base):
    """x [T, heads, d]: the first `dims` entries of every head turned by the row's position; entry i and entry
    i + dims / 2 are the two coordinates of a plane that turns by base^(-2 i / dims) per token."""
    if not dims:
        return x
    half = dims // 2
    pos = torch.arange(x.shape[0], dtype=D64)
    ang = pos[:, None] * torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=D64)
    c, s = torch.cos(ang)[:, None].to(x.dtype), torch.sin(ang)[:, None].to(x.dtype)
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], -1)


def softmax_seen(scores, window=0, sink=None):
    """scores [heads, T, T] -> weights over the keys j <= i (with a window: i - j < window).  sink [heads]: exp(sink)
    joins the denominator."""
    T = scores.shape[-1]
    d = torch.arange(T)[:, None] - torch.arange(T)[None]
    hidden = (d < 0) | ((d >= window) if window else torch.zeros_like(d, dtype=torch.bool))
    scores = scores.masked_fill(hidden, float("-inf"))
    top = scores.max(-1, keepdim=True).values
    if sink is not None:
        top = torch.maximum(top, sink[:, None, None])
    e = torch.exp(scores - top)
    total = e.sum(-1, keepdim=True)
    if sink is not None:
        total = total + torch.exp(sink[:, None, None] - top)
    return e / total


def cap(scores, limit):
    return limit * torch.tanh(scores / limit) if limit else scores


def mix_values(v, first, lam):
    return (1 - lam) * v + lam * first


def attention(h, W, p, m, eps, first=None):
    """Grouped softmax attention with head norms, rotation, capped scores, a window and a sink per head.  `first`: the
    values that this layer's own values are mixed with (None: no mixing).  Returns (output, the layer's own values)."""
    T = h.shape[0]
    H, G, dk, dv, rot = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m.get("rot") or {}
    q = unit_rms((h @ W[p + "q"].T).view(T, H, dk), eps) * W[p + "q.norm"]
    k = unit_rms((h @ W[p + "k"].T).view(T, G, dk), eps) * W[p + "k.norm"]
    q, k = (turn(z, rot.get("dims", 0), rot.get("base", 1.0)) for z in (q, k))
    own = (h @ W[p + "v"].T).view(T, G, dv)
    v = own if first is None else mix_values(own, first, W[p + "vmix"])
    k, v = k.repeat_interleave(H // G, 1), v.repeat_interleave(H // G, 1)
    s = cap(torch.einsum("ihd,jhd->hij", q, k) * m["scale"], m.get("softcap"))
    a = softmax_seen(s, (m.get("mask") or {}).get("size", 0), W.get(p + "sink"))
    return torch.einsum("hij,jhd->ihd", a, v).reshape(T, H * dv) @ W[p + "o"].T, own


def latent_attention(h, W, p, m, eps):
    T = h.shape[0]
    H, dn, dr, dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    rot = m.get("rot") or {}
    cq = unit_rms(h @ W[p + "dq"].T, eps) * W[p + "dq.norm"]
    q = (cq @ W[p + "uq"].T).view(T, H, dn + dr)
    low = h @ W[p + "dkv"].T
    c = unit_rms(low[:, :R], eps) * W[p + "dkv.norm"]
    q_rot = turn(q[..., dn:], rot.get("dims", 0), rot.get("base", 1.0))
    k_rot = turn(low[:, None, R:], rot.get("dims", 0), rot.get("base", 1.0))[:, 0]
    k = (c @ W[p + "uk"].T).view(T, H, dn)
    v = (c @ W[p + "uv"].T).view(T, H, dv)
    s = torch.einsum("ihd,jhd->hij", q[..., :dn], k) + torch.einsum("ihd,jd->hij", q_rot, k_rot)
    o = torch.einsum("hij,jhd->ihd", softmax_seen(s * m["scale"]), v).reshape(T, H * dv)
    return (o * torch.sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def retention_scan(q, k, v, decay):
    """q, k [T, H, dk], v [T, H, dv], decay [H]: S <- decay S + k v^T, o = S^T q, token by token."""
    S = torch.zeros(q.shape[1], q.shape[2], v.shape[2], dtype=q.dtype)
    out = []
    for t in range(q.shape[0]):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hkv,hk->hv", S, q[t]))
    return torch.stack(out)


def retention(h, W, p, m, eps):
    T = h.shape[0]
    H, dk, dv, rot = m["heads"], m["dim"], m["vdim"], m.get("rot") or {}
    q, k = (turn((h @ W[p + n].T).view(T, H, dk), rot.get("dims", 0), rot.get("base", 1.0)) for n in ("q", "k"))
    o = retention_scan(q, k / math.sqrt(dk), (h @ W[p + "v"].T).view(T, H, dv), torch.tensor(m["decay"], dtype=h.dtype))
    g = h @ W[p + "g"].T
    return (unit_rms(o, eps).reshape(T, H * dv) * g * torch.sigmoid(g)) @ W[p + "o"].T


def dense(h, W, p):
    g = h @ W[p + "gate"].T
    return (g * torch.sigmoid(g) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def clamped_act(g, u, limit):
    g, u = torch.clamp(g, max=limit), torch.clamp(u, -limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1)


def expert(h, W, q, limit):
    return clamped_act(h @ W[q + "gate"].T, h @ W[q + "up"].T, limit) @ W[q + "down"].T


def route(z, top):
    """z: one token's logits.  -> (chosen experts, best first, their weights: a softmax over the chosen logits only)."""
    chosen = sorted(range(len(z)), key=lambda e: (-z[e].item(), e))[:top]
    return chosen, torch.softmax(z[chosen], 0)


def mixture(h, W, p, mlp):
    z = h @ W[p + "router"].T + W[p + "router.b"]
    rows = []
    for t in range(h.shape[0]):
        idx, wt = route(z[t], mlp["router"]["top"])
        rows.append(sum(w * expert(h[t], W, f"{p}e{e}.", mlp["expert"]["limit"]) for e, w in zip(idx, wt)))
    return torch.stack(rows)


def forward(cfg, tensors, tokens, dtype=D64, layers_out=None):
    """Logits [T, vocab] of one sequence; layers_out (a list) receives the stream after every layer."""
    W = {k: v.to(dtype) for k, v in tensors.items()}
    eps, c = cfg["norm"]["eps"], cfg["residual_mult"]
    x = W["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
    first = None
    for i, L in enumerate(cfg["layers"]):
        n, m = f"l{i}.", L["mixer"]
        h = dynamic_tanh(x, W, n + "norm1")
        if L["type"] == "attention":
            y, own = attention(h, W, n + "mix.", m, eps, first if m.get("v_mix") else None)
            if m.get("v_mix") and first is None:
                first = own
        elif L["type"] == "retention":
            y = retention(h, W, n + "mix.", m, eps)
        elif L["type"] == "latent_attention":
            y = latent_attention(h, W, n + "mix.", m, eps)
        else:
            raise ValueError(L["type"])
        x = x + c * y
        if L.get("mlp"):
            h = dynamic_tanh(x, W, n + "norm2")
            y = dense(h, W, n + "mlp.") if L["mlp"]["kind"] == "dense" else mixture(h, W, n + "mlp.", L["mlp"])
            x = x + c * y
        if layers_out is not None:
            layers_out.append(x)
    return dynamic_tanh(x, W, "final.norm") @ W["head"].T
