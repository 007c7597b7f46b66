"""Zufulix checkpoints -> hybrid.HybridRunner.

config.json: {"architecture": "Zufulix", "width", "vocab", "streams", "embedding": {"scale"}, "norm": {"eps"}, "layers":
[{"type": "attention", "mixer": {...}, "mlp": {...} | null}, ...]}; tensors are named "embed", "l<i>.norm1" (+ ".b"),
"l<i>.norm2", "l<i>.hc1.{in,mix,out}", "l<i>.hc2.*", "l<i>.mix.*", "l<i>.mlp.*", "final.norm"; linear weights [out, in].
The model keeps several residual streams joined by hyper-connections: a pre-norm sublayer (layer norm with bias) reads a
weighted sum of the streams and rewrites all of them from one matrix over the old streams and its own result; the model
ends with their sum, and the embedding table (scaled on the way in) is also the output matrix.
  attention    : softmax attention with grouped key / value heads and projection biases, weightless RMS norm per q / k
                 head, no rotation, a learned bias per head and bucket of the distance; values mixed with those of the
                 first layer that has `v_mix`
  feed-forward : `dense` (exact GELU) or `moe`: ungated squared-ReLU experts behind a sigmoid router whose expert groups
                 are ranked by their two best members, the chosen scores divided by their sum
This file only arranges weights for the launch plan (fused input projections, stacked experts, fp32 small parameters, the
bias per distance); the arithmetic is in the CUDA kernels."""
from __future__ import annotations

import math

import torch

from ..hybrid import LAYOUT_HYPER, MAX_STREAMS, MIXER_WINDOW_ATTN, NORM_LAYER, HybridRunner, LayerSpec
from . import register

_ZERO = dict(heads=0, kv_heads=0, dim=0, rot_dim=0, rot_dims=0, vdim=0, kv_rank=0, window=0, state=0, conv_taps=0,
             norm_groups=0, scale=0.0, rot_mag=1.0, experts=0, top=0, expert_ff=0, shared_ff=0, route_scale=1.0,
             layout=LAYOUT_HYPER, out_scale=1.0, gated=0, norm_kind=NORM_LAYER)


def distance_buckets(buckets: int, far: int) -> list[int]:
    """Bucket of every distance 0, 1, .. up to the first one in the last bucket (which holds for all further ones).  The
    first half of the buckets count single distances, the rest grow geometrically from buckets // 2 to `far`."""
    half = buckets // 2
    if half == 0:
        return [buckets - 1]
    if far <= half:
        raise ValueError("bias_max must exceed half the number of buckets")
    out = []
    while not out or out[-1] != buckets - 1:
        n = len(out)
        if n < half:
            out.append(n)
            continue
        # (a distance that lies on a bucket's edge belongs to that bucket: the quotient of the logarithms may fall short
        # of the whole number by a rounding)
        steps = math.log(n / half) / math.log(far / half) * (buckets - half)
        out.append(min(buckets - 1, half + math.floor(steps + 1e-9)))
    return out


def distance_table(rel: torch.Tensor, far: int) -> torch.Tensor:
    """rel [buckets, heads] -> fp32 [heads, distances]; the last column stands for every greater distance."""
    idx = torch.tensor(distance_buckets(rel.shape[0], far))
    return rel.to(torch.float32)[idx].t().contiguous()


@register("Zufulix")
def build(cfg, tensors, *, dtype=torch.bfloat16, device="cuda", num_blocks, max_blocks_per_seq, max_seqs, max_tokens,
          num_state_slots=None, layer_trace=False, **_):
    dtype = dtype or torch.bfloat16
    dev = torch.device(device)
    width, streams = int(cfg["width"]), int(cfg.get("streams", 1))
    if not 1 <= streams <= MAX_STREAMS:
        raise ValueError(f"streams must be 1 .. {MAX_STREAMS}")

    def mat(*names):                      # matrix-product operand(s), fused along the output rows
        ts = [tensors[n] for n in names]
        return (torch.cat(ts, 0) if len(ts) > 1 else ts[0]).to(dtype).contiguous().to(dev)

    def vec(*names):                      # small parameters stay fp32
        ts = [tensors[n].to(torch.float32).reshape(-1) for n in names]
        return (torch.cat(ts, 0) if len(ts) > 1 else ts[0]).contiguous().to(dev)

    specs = []
    first_values = None                   # (kv_heads, vdim) of the first layer that mixes values
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix.", layer["mixer"]
        if layer["type"] != "attention":
            raise ValueError(f"layer {i}: unknown mixer type {layer['type']!r}")
        H, G, dk, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
        d = dict(_ZERO, heads=H, kv_heads=G, dim=dk, vdim=dv, scale=float(m["scale"]), head_norm=2)
        table = distance_table(tensors[p + "rel"], m["bias_max"])
        d["dist_n"] = table.shape[1]
        t = dict(norm_w=vec(f"l{i}.norm1"), norm_b=vec(f"l{i}.norm1.b"), hc_in=vec(f"l{i}.hc1.in"),
                 hc_mix=vec(f"l{i}.hc1.mix"), hc_out=vec(f"l{i}.hc1.out"), w_in=mat(p + "q", p + "k", p + "v"),
                 in_bias=vec(p + "q.b", p + "k.b", p + "v.b"), w_o=mat(p + "o"), dist_bias=table.to(dev))
        if m.get("v_mix"):
            if first_values is None:
                first_values, d["v_mix_role"] = (G, dv), 1
            elif first_values != (G, dv):
                raise ValueError(f"layer {i}: mixed values need the kv_heads and vdim of the first layer that mixes")
            else:
                d.update(v_mix_role=2, v_mix=float(tensors[p + "vmix"].to(torch.float32)))
        mlp = layer.get("mlp")
        if mlp:
            q = f"l{i}.mlp."
            t.update(ff_norm_w=vec(f"l{i}.norm2"), ff_norm_b=vec(f"l{i}.norm2.b"), ff_hc_in=vec(f"l{i}.hc2.in"),
                     ff_hc_mix=vec(f"l{i}.hc2.mix"), ff_hc_out=vec(f"l{i}.hc2.out"))
            if mlp["kind"] == "dense":
                d.update(shared_ff=int(mlp["ff"]), shared_act=2)
                t.update(w_shared_gate_up=mat(q + "up"), w_shared_down=mat(q + "down"))
            elif mlp["kind"] == "moe":
                r = mlp["router"]
                E, groups = int(r["experts"]), r.get("groups") or {}
                d.update(experts=E, top=int(r["top"]), expert_ff=int(mlp["expert"]["ff"]), expert_act=1, route_score=1,
                         route_renorm=1, route_groups=int(groups.get("count", 0)), route_keep=int(groups.get("keep", 0)),
                         route_group_top=2)
                t.update(w_router=mat(q + "router"),
                         w_gate_up=torch.stack([mat(f"{q}e{e}.up") for e in range(E)]).contiguous(),
                         w_down=torch.stack([mat(f"{q}e{e}.down") for e in range(E)]).contiguous())
            else:
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
        specs.append(LayerSpec(MIXER_WINDOW_ATTN, d, t))
    embed = mat("embed")
    return HybridRunner(width=width, vocab=int(cfg["vocab"]), layers=specs, embed=embed, final_norm=vec("final.norm"),
                        lm_head=embed, norm_eps=float(cfg["norm"]["eps"]), norm_weight_offset=0.0,
                        embed_scale=float(cfg["embedding"]["scale"]), dtype=dtype, num_blocks=num_blocks,
                        max_blocks_per_seq=max_blocks_per_seq, max_seqs=max_seqs, max_tokens=max_tokens,
                        num_state_slots=num_state_slots or max_seqs, device=device, layer_trace=layer_trace,
                        final_norm_kind=NORM_LAYER, final_norm_bias=vec("final.norm.b"), streams=streams)
