"""Sonalix checkpoints -> hybrid.HybridRunner.

config.json: {"architecture": "Sonalix", "width", "vocab", "embedding": {"scale"}, "residual_mult", "norm": {"eps"},
"layers": [{"type", "mixer": {...}, "mlp": {...} | null}, ...]}; tensors are named "embed", "l<i>.norm1" (+ ".b",
".alpha"), "l<i>.norm2", "l<i>.mix.*", "l<i>.mlp.*", "final.norm", "head"; linear weights [out, in].  Every layer is
pre-norm with dynamic-tanh norms (tanh(alpha x) w + b), and both sublayers are added to the stream times residual_mult.
Mixer types (rotary positions in the two-halves layout throughout):
  attention        : softmax attention with grouped key / value heads, RMS norm per q / k head with one weight shared by
                     the heads, capped scores, a sliding window, a learned sink per head, and values mixed with those of
                     the first layer that has `v_mix`
  retention        : linear attention with one fixed decay per head, rotated queries and keys, RMS norm per head and a
                     SiLU gate
  latent_attention : latent (compressed key / value) attention whose queries go through a normed latent of their own, with
                     a rotated part beside the plain one and a sigmoid gate per output element
Feed-forward kinds: `dense` (SiLU-gated) and `moe`: clamped gated experts g sigmoid(1.702 g) (u + 1) behind a router that
picks the largest biased logits and weighs them by a softmax over the chosen ones.
This file only arranges weights for the launch plan (fused input projections, stacked experts, fp32 small parameters,
frequency tables); the arithmetic is in the CUDA kernels."""
from __future__ import annotations

import numpy as np
import torch

from ..hybrid import (EXPERT_CLAMPED, LAYOUT_PRENORM, MIXER_DECAY_ATTN, MIXER_LATENT_ATTN, MIXER_WINDOW_ATTN,
                      NORM_DYNTANH, HybridRunner, LayerSpec)
from ..rotary import rotary_frequencies
from . import register

EXPERT_ALPHA, EXPERT_UP_ADD = 1.702, 1.0      # the experts' activation: g sigmoid(alpha g) (u + up_add)
ROUTE_CHOSEN_LOGITS = 2                       # choice by logit + bias, softmax over the chosen logits

_ZERO = dict(heads=0, kv_heads=0, dim=0, rot_dim=0, rot_dims=0, vdim=0, kv_rank=0, window=0, state=0, conv_taps=0,
             norm_groups=0, scale=0.0, rot_mag=1.0, experts=0, top=0, expert_ff=0, shared_ff=0, route_scale=1.0,
             layout=LAYOUT_PRENORM, gated=0, norm_kind=NORM_DYNTANH, rot_half=1)


@register("Sonalix")
def build(cfg, tensors, *, dtype=torch.bfloat16, device="cuda", num_blocks, max_blocks_per_seq, max_seqs, max_tokens,
          num_state_slots=None, layer_trace=False, **_):
    dtype = dtype or torch.bfloat16
    dev = torch.device(device)
    width, mult = int(cfg["width"]), float(cfg.get("residual_mult", 1.0))

    def mat(*names):                      # matrix-product operand(s), fused along the output rows
        ts = [tensors[n] for n in names]
        return (torch.cat(ts, 0) if len(ts) > 1 else ts[0]).to(dtype).contiguous().to(dev)

    def vec(*names):                      # small parameters stay fp32
        ts = [tensors[n].to(torch.float32).reshape(-1) for n in names]
        return (torch.cat(ts, 0) if len(ts) > 1 else ts[0]).contiguous().to(dev)

    def norm(name, prefix):               # a dynamic-tanh norm: weight, bias, the scalar inside the tanh
        return {prefix + "_w": vec(name), prefix + "_b": vec(name + ".b") if name + ".b" in tensors else None}, \
            float(tensors[name + ".alpha"].to(torch.float32))

    specs = []
    first_values = None                   # (kv_heads, vdim) of the first layer that mixes values
    for i, layer in enumerate(cfg["layers"]):
        p, m, kind = f"l{i}.mix.", layer["mixer"], layer["type"]
        H, dk, dv, rot = int(m["heads"]), int(m["dim"]), int(m["vdim"]), m.get("rot") or {}
        d = dict(_ZERO, out_scale=mult, ff_scale=mult, heads=H, dim=dk, vdim=dv, rot_dims=int(rot.get("dims", 0)))
        t, d["norm_alpha"] = norm(f"l{i}.norm1", "norm")
        t["w_o"] = mat(p + "o")
        if d["rot_dims"]:
            freq, _mag = rotary_frequencies(d["rot_dims"], float(rot["base"]))
            t["rot_freq"] = torch.from_numpy(np.ascontiguousarray(freq, dtype=np.float64)).to(dev)
        if kind == "attention":
            mixer, G = MIXER_WINDOW_ATTN, int(m["kv_heads"])
            d.update(kv_heads=G, scale=float(m["scale"]), softcap=float(m.get("softcap") or 0.0), head_norm=1,
                     window=int((m.get("mask") or {}).get("size", 0)))
            t.update(w_in=mat(p + "q", p + "k", p + "v"), q_norm_w=vec(p + "q.norm"), k_norm_w=vec(p + "k.norm"),
                     sink=vec(p + "sink") if p + "sink" in tensors else None)
            if m.get("v_mix"):
                if first_values is None:
                    first_values, d["v_mix_role"] = (G, dv), 1
                elif first_values != (G, dv):
                    raise ValueError(f"layer {i}: mixed values need the kv_heads and vdim of the first layer that mixes")
                else:
                    d.update(v_mix_role=2, v_mix=float(tensors[p + "vmix"].to(torch.float32)))
        elif kind == "retention":
            mixer = MIXER_DECAY_ATTN
            if len(m["decay"]) != H:
                raise ValueError(f"layer {i}: one decay per head")
            d.update(norm_groups=H, q_scale=1.0, k_scale=dk ** -0.5)
            t.update(w_in=mat(p + "q", p + "k", p + "v", p + "g"),
                     head_decay=torch.tensor([float(x) for x in m["decay"]], dtype=torch.float32, device=dev))
        elif kind == "latent_attention":
            mixer, dr = MIXER_LATENT_ATTN, int(m["rot_dim"])
            d.update(rot_dim=dr, kv_rank=int(m["kv_rank"]), q_rank=int(m["q_rank"]), scale=float(m["scale"]), gated=2)
            t.update(w_in=mat(p + "dq", p + "dkv", p + "g"), q_norm_w=vec(p + "dq.norm"), w_uq=mat(p + "uq"),
                     latent_norm_w=vec(p + "dkv.norm"), w_uk=mat(p + "uk"), w_uv=mat(p + "uv"))
        else:
            raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
        mlp = layer.get("mlp")
        if mlp:
            q = f"l{i}.mlp."
            n2, d["ff_norm_alpha"] = norm(f"l{i}.norm2", "ff_norm")
            t.update(n2)
            if mlp["kind"] == "dense":
                d["shared_ff"] = int(mlp["ff"])
                t.update(w_shared_gate_up=mat(q + "gate", q + "up"), w_shared_down=mat(q + "down"))
            elif mlp["kind"] == "moe":
                r, e = mlp["router"], mlp["expert"]
                E = int(r["experts"])
                d.update(experts=E, top=int(r["top"]), expert_ff=int(e["ff"]), expert_act=EXPERT_CLAMPED,
                         expert_limit=float(e["limit"]), expert_alpha=EXPERT_ALPHA, expert_up_add=EXPERT_UP_ADD,
                         route_score=ROUTE_CHOSEN_LOGITS)
                t.update(w_router=mat(q + "router"), route_bias=vec(q + "router.b"),
                         w_gate_up=torch.stack([mat(f"{q}e{j}.gate", f"{q}e{j}.up") for j in range(E)]).contiguous(),
                         w_down=torch.stack([mat(f"{q}e{j}.down") for j in range(E)]).contiguous())
            else:
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
        specs.append(LayerSpec(mixer, d, t))
    fin, alpha = norm("final.norm", "f")
    return HybridRunner(width=width, vocab=int(cfg["vocab"]), layers=specs, embed=mat("embed"), final_norm=fin["f_w"],
                        lm_head=mat("head"), norm_eps=float(cfg["norm"]["eps"]), norm_weight_offset=0.0,
                        embed_scale=float(cfg["embedding"]["scale"]), dtype=dtype, num_blocks=num_blocks,
                        max_blocks_per_seq=max_blocks_per_seq, max_seqs=max_seqs, max_tokens=max_tokens,
                        num_state_slots=num_state_slots or max_seqs, device=device, layer_trace=layer_trace,
                        final_norm_kind=NORM_DYNTANH, final_norm_bias=fin["f_b"], final_norm_alpha=alpha)
