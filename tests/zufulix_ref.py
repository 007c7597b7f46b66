"""A plain, slow restatement of the Zufulix decoder in double precision, one function per mechanism.  It shares no code
with the product path (vllm_rs_b200/models/zufulix.py arranges weights for CUDA kernels; this file multiplies them out on
the CPU) and is what the GPU tests compare the framework with.

Notation: T tokens at positions 0 .. T-1, S streams X_1 .. X_S, each [T, D], all equal to the scaled embedding rows at the
start.  Every sublayer F (mixer, then feed-forward) with its vectors a (S), b (S) and matrix M (S x S):
    y = F(N(sum_s a_s X_s));    X_t <- sum_s M_st X_s + b_t y      (all streams from the old ones)
and the logits are E N_f(sum_s X_s) with the embedding table E.  N is a layer norm with weight and bias."""
from __future__ import annotations

import math

import torch

D64 = torch.float64


def layer_norm(x, w, b, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w + b


def read_streams(streams, a):
    return sum(a[s] * streams[s] for s in range(len(streams)))


def update_streams(streams, mix, out, y):
    n = len(streams)
    return [sum(mix[s, t] * streams[s] for s in range(n)) + out[t] * y for t in range(n)]


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def distance_bucket(n, buckets, far):
    """Half of the buckets count single distances, the others grow geometrically up to `far`; the last one is open."""
    half = buckets // 2
    if n < half:
        return n
    if half == 0:
        return buckets - 1
    steps = math.log(n / half) / math.log(far / half) * (buckets - half)
    return min(buckets - 1, half + math.floor(steps + 1e-9))


def distance_bias_rows(rel, rows, n, far):
    """The bias of the query positions `rows` against the keys 0 .. n - 1, [heads, len(rows), n]: rel[bucket(i - j), head]
    (entries with j > i are zero)."""
    B = rel.shape[0]
    by_dist = torch.tensor([distance_bucket(d, B, far) for d in range(n)])
    out = torch.zeros(rel.shape[1], len(rows), n, dtype=rel.dtype)
    for r, i in enumerate(rows):
        out[:, r, :i + 1] = rel[by_dist[:i + 1].flip(0)].T
    return out


def softmax_causal(scores):
    T = scores.shape[-1]
    later = torch.ones(T, T, dtype=torch.bool).triu(1)
    scores = scores.masked_fill(later, float("-inf"))
    e = torch.exp(scores - scores.max(-1, keepdim=True).values)
    return e / e.sum(-1, keepdim=True)


def mix_values(v, first, lam):
    return (1 - lam) * v + lam * first


def attention(h, W, p, m, eps, first=None):
    """Grouped softmax attention, weightless RMS norm per q / k head, a learned bias per distance bucket.  `first`: the
    values that this layer's own values are mixed with (None: no mixing).  Returns (output, the layer's own values)."""
    T = h.shape[0]
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = unit_rms((h @ W[p + "q"].T + W[p + "q.b"]).view(T, H, dk), eps)
    k = unit_rms((h @ W[p + "k"].T + W[p + "k.b"]).view(T, G, dk), eps)
    own = (h @ W[p + "v"].T + W[p + "v.b"]).view(T, G, dv)
    v = own if first is None else mix_values(own, first, W[p + "vmix"])
    k, v = k.repeat_interleave(H // G, 1), v.repeat_interleave(H // G, 1)
    s = torch.einsum("ihd,jhd->hij", q, k) * m["scale"] + distance_bias_rows(W[p + "rel"], range(T), T, m["bias_max"])
    o = torch.einsum("hij,jhd->ihd", softmax_causal(s), v)
    return o.reshape(T, H * dv) @ W[p + "o"].T, own


def gelu(z):
    return 0.5 * z * (1 + torch.erf(z / math.sqrt(2.0)))


def dense(h, W, p):
    return gelu(h @ W[p + "up"].T) @ W[p + "down"].T


def route(z, top, count=0, keep=0):
    """z: one token's router logits (list or 1-d tensor).  -> (chosen experts, best first, their weights)."""
    s = 1 / (1 + torch.exp(-z))
    E = len(s)
    allowed = list(range(E))
    if count:
        per = E // count
        score = [sum(sorted(s[g * per:(g + 1) * per].tolist(), reverse=True)[:2]) for g in range(count)]
        best = sorted(range(count), key=lambda g: (-score[g], g))[:keep]
        allowed = [e for e in allowed if e // per in best]
    chosen = sorted(allowed, key=lambda e: (-s[e].item(), e))[:top]
    total = sum(s[e] for e in chosen) + 1e-20
    return chosen, [s[e] / total for e in chosen]


def expert(h, W, q):
    return torch.relu(h @ W[q + "up"].T) ** 2 @ W[q + "down"].T


def mixture(h, W, p, mlp):
    r = mlp["router"]
    g = r.get("groups") or {}
    z = h @ W[p + "router"].T
    rows = []
    for t in range(h.shape[0]):
        idx, wt = route(z[t], r["top"], g.get("count", 0), g.get("keep", 0))
        rows.append(sum(w * expert(h[t], W, f"{p}e{e}.") for e, w in zip(idx, wt)))
    return torch.stack(rows)


def forward(cfg, tensors, tokens, dtype=D64, layers_out=None):
    """Logits [T, vocab] of one sequence; layers_out (a list) receives the sum of the streams after every layer."""
    W = {k: v.to(dtype) for k, v in tensors.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
    streams = [x] * cfg["streams"]
    first = None
    for i, L in enumerate(cfg["layers"]):
        n, m = f"l{i}.", L["mixer"]
        if L["type"] != "attention":
            raise ValueError(L["type"])
        h = layer_norm(read_streams(streams, W[n + "hc1.in"]), W[n + "norm1"], W[n + "norm1.b"], eps)
        y, own = attention(h, W, n + "mix.", m, eps, first if m.get("v_mix") else None)
        if m.get("v_mix") and first is None:
            first = own
        streams = update_streams(streams, W[n + "hc1.mix"], W[n + "hc1.out"], y)
        if L.get("mlp"):
            h = layer_norm(read_streams(streams, W[n + "hc2.in"]), W[n + "norm2"], W[n + "norm2.b"], eps)
            y = dense(h, W, n + "mlp.") if L["mlp"]["kind"] == "dense" else mixture(h, W, n + "mlp.", L["mlp"])
            streams = update_streams(streams, W[n + "hc2.mix"], W[n + "hc2.out"], y)
        if layers_out is not None:
            layers_out.append(sum(streams))
    x = layer_norm(sum(streams), W["final.norm"], W["final.norm.b"], eps)
    return x @ W["embed"].T
