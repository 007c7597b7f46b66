"""Host-side pieces behind the Sonalix decoder: the model registry, the config reader's checks, and the plain
restatement's own invariants."""
import math

import numpy as np
import pytest
import torch

import sonalix_ref as R
from sonalix_util import dense_cfg, full_cfg, layer, make_cfg, moe_cfg, random_layers, random_tensors

D64 = torch.float64


def test_registry_knows_the_family():
    from vllm_rs_b200 import models
    assert "Sonalix" in models.registered() and "Sonalix" in models.HYBRID_ARCHITECTURES
    assert models.architecture_of({"architecture": "Sonalix"}) == "Sonalix"


def test_command_line_lists_the_architecture(capsys):
    from vllm_rs_b200.__main__ import main
    assert main(["models"]) == 0
    assert "Sonalix" in capsys.readouterr().out.split()


def test_config_reader_rejects_what_the_design_excludes():
    from vllm_rs_b200.models import build_runner
    kw = dict(dtype=torch.float32, device="cpu", num_blocks=2, max_blocks_per_seq=2, max_seqs=1, max_tokens=64)
    other = make_cfg([layer("attention"), layer("attention", vdim=24)])          # mixed values of different sizes
    with pytest.raises(ValueError):
        build_runner(other, random_tensors(other), **kw)
    unknown = make_cfg([layer("attention")])
    w = random_tensors(unknown)
    unknown["layers"][0]["type"] = "attention_2"
    with pytest.raises(ValueError):
        build_runner(unknown, w, **kw)
    kind = make_cfg([layer("retention", dense_cfg())])
    w = random_tensors(kind)
    kind["layers"][0]["mlp"]["kind"] = "gated"
    with pytest.raises(ValueError):
        build_runner(kind, w, **kw)
    short = make_cfg([layer("retention", decay=[0.5])])                          # one decay for four heads
    with pytest.raises(ValueError):
        build_runner(short, random_tensors(short), **kw)


def test_plain_model_invariants():
    """The restatement itself: causal; the sink, the cap, the gates, the router's bias and which layer's values are kept all
    matter; the kept layer's own mixing weight does not."""
    cfg = full_cfg()
    w = random_tensors(cfg, seed=1)
    t = np.random.default_rng(0).integers(0, cfg["vocab"], size=90).tolist()
    full = R.forward(cfg, w, t).numpy()
    part = R.forward(cfg, w, t[:47]).numpy()
    assert np.abs(full[:47] - part).max() < 1e-9
    for name in ("l0.mix.sink", "l1.mix.g", "l3.mix.g", "l1.mlp.router.b", "l4.mix.vmix", "l2.norm1.alpha", "final.norm.b"):
        w2 = dict(w)
        w2[name] = torch.zeros_like(w[name])
        assert np.abs(R.forward(cfg, w2, t).numpy() - full).max() > 1e-3, name
    w2 = dict(w)
    w2["l2.mix.vmix"] = torch.zeros_like(w["l2.mix.vmix"])            # the first mixing layer keeps its own values
    assert np.abs(R.forward(cfg, w2, t).numpy() - full).max() == 0.0


def test_plain_mechanisms():
    g = torch.Generator().manual_seed(2)
    x = torch.randn(6, 3, 10, generator=g, dtype=D64)
    y = R.turn(x, 6, 50.0)
    assert torch.equal(y[..., 6:], x[..., 6:]) and torch.equal(y[0], x[0])
    a = 2 * 50.0 ** (-2.0 / 6)                                        # position 2, second plane: entries 1 and 4
    assert torch.allclose(y[2, :, 1], x[2, :, 1] * math.cos(a) - x[2, :, 4] * math.sin(a))
    assert torch.allclose(y[2, :, 4], x[2, :, 4] * math.cos(a) + x[2, :, 1] * math.sin(a))
    s = torch.zeros(1, 5, 5, dtype=D64)
    p = R.softmax_seen(s, 2, torch.tensor([math.log(3.0)], dtype=D64))
    assert torch.allclose(p[0, 0], torch.tensor([0.25, 0, 0, 0, 0], dtype=D64))
    assert torch.allclose(p[0, 4], torch.tensor([0, 0, 0, 0.2, 0.2], dtype=D64))
    z = torch.tensor([1.0, 3.0, 2.0, 3.0], dtype=D64)
    idx, wt = R.route(z, 3)
    assert idx == [1, 3, 2] and torch.allclose(wt, torch.softmax(torch.tensor([3.0, 3.0, 2.0], dtype=D64), 0))
    g_, u = torch.tensor([9.0, -9.0, 0.3], dtype=D64), torch.tensor([-9.0, 9.0, 0.2], dtype=D64)
    c = R.clamped_act(g_, u, 2.0)
    sg = lambda v: 1 / (1 + math.exp(-1.702 * v))                     # noqa: E731
    want = [2 * sg(2) * -1, -9 * sg(-9) * 3, 0.3 * sg(0.3) * 1.2]     # the gate is clamped from above only
    assert torch.allclose(c, torch.tensor(want, dtype=D64))
    k, v = torch.randn(4, 1, 3, generator=g, dtype=D64), torch.randn(4, 1, 2, generator=g, dtype=D64)
    q = torch.randn(4, 1, 3, generator=g, dtype=D64)
    o = R.retention_scan(q, k, v, torch.tensor([0.5], dtype=D64))
    want = sum(0.5 ** (3 - j) * (q[3, 0] @ k[j, 0]) * v[j, 0] for j in range(4))
    assert torch.allclose(o[3, 0], want)


def test_random_layers_are_consistent():
    for seed in range(30):
        layers = random_layers(np.random.default_rng(seed), 6)
        mixing = {(L["mixer"]["kv_heads"], L["mixer"]["vdim"]) for L in layers if L["mixer"].get("v_mix")}
        assert len(mixing) <= 1
        for L in layers:
            m, mlp = L["mixer"], L["mlp"]
            assert m["heads"] % m.get("kv_heads", 1) == 0
            assert m["rot"]["dims"] <= (m["rot_dim"] if L["type"] == "latent_attention" else m["dim"])
            assert not mlp or mlp["kind"] == "dense" or mlp["router"]["top"] <= mlp["router"]["experts"]
    assert moe_cfg()["router"]["top"] == 3
