"""Host-side pieces behind the Zufulix decoder: the model registry, the table of the distance bias, the config reader's
checks, and the plain restatement's own invariants."""
import math

import numpy as np
import pytest
import torch

import zufulix_ref as R
from zufulix_util import dense_cfg, full_cfg, layer, make_cfg, moe_cfg, random_layers, random_tensors


def test_registry_knows_the_family():
    from vllm_rs_b200 import models
    assert "Zufulix" in models.registered() and "Zufulix" in models.HYBRID_ARCHITECTURES
    assert models.architecture_of({"architecture": "Zufulix"}) == "Zufulix"


def test_command_line_lists_the_architecture(capsys):
    from vllm_rs_b200.__main__ import main
    assert main(["models"]) == 0
    assert "Zufulix" in capsys.readouterr().out.split()


@pytest.mark.parametrize("buckets,far", [(32, 128), (32, 100), (8, 16), (2, 2), (2, 500), (7, 90), (1, 5), (24, 96), (40, 21)])
def test_distance_table_agrees_with_the_plain_buckets(buckets, far):
    from vllm_rs_b200.models.zufulix import distance_buckets, distance_table
    b = distance_buckets(buckets, far)
    assert b == [R.distance_bucket(n, buckets, far) for n in range(len(b))]
    assert b[-1] == buckets - 1 and (len(b) == 1 or b[-2] < buckets - 1) and b == sorted(b)
    assert all(R.distance_bucket(n, buckets, far) == buckets - 1 for n in (len(b), 2 * len(b), 100000))
    rel = torch.arange(buckets * 3, dtype=torch.float32).reshape(buckets, 3)
    t = distance_table(rel, far)
    assert t.shape == (3, len(b)) and torch.equal(t, rel[torch.tensor(b)].T)


def test_bucket_edges_that_are_whole_numbers():
    """far / half = 8 over 12 geometric buckets: every third edge doubles the distance; a distance on an edge belongs to
    the bucket that starts there, whatever the rounding of the logarithms."""
    from vllm_rs_b200.models.zufulix import distance_buckets
    b = distance_buckets(24, 96)
    for k in range(3):
        n = 12 * 2 ** k
        assert n >= len(b) or b[n] == 12 + 4 * k
        assert b[n - 1] == (11 if k == 0 else 12 + 4 * k - 1)
    for B, far in ((32, 16 * 2 ** 4), (20, 10 * 4), (6, 3 * 27)):
        half = B // 2
        ratio = far // half
        got = distance_buckets(B, far)
        for n in range(half, len(got)):
            k = got[n] - half                                         # half * ratio^(k / (B - half)) <= n < the next edge
            assert half ** (B - half) * ratio ** k <= n ** (B - half)
            assert got[n] == B - 1 or n ** (B - half) < half ** (B - half) * ratio ** (k + 1)


def test_bias_range_must_exceed_the_linear_half():
    from vllm_rs_b200.models.zufulix import distance_buckets
    for far in (16, 3):
        with pytest.raises(ValueError):
            distance_buckets(32, far)


def test_config_reader_rejects_what_the_design_excludes():
    from vllm_rs_b200.models import build_runner
    kw = dict(dtype=torch.float32, device="cpu", num_blocks=2, max_blocks_per_seq=2, max_seqs=1, max_tokens=64)
    other = make_cfg([layer(), layer(vdim=24)])                       # mixed values of different sizes
    with pytest.raises(ValueError):
        build_runner(other, random_tensors(other), **kw)
    unknown = make_cfg([layer()])
    unknown["layers"][0]["type"] = "attention_2"
    with pytest.raises(ValueError):
        build_runner(unknown, random_tensors(make_cfg([layer()])), **kw)
    kind = make_cfg([layer(dense_cfg())])
    w = random_tensors(kind)
    kind["layers"][0]["mlp"]["kind"] = "gated"
    with pytest.raises(ValueError):
        build_runner(kind, w, **kw)
    many = make_cfg([layer()], streams=17)
    with pytest.raises(ValueError):
        build_runner(many, random_tensors(many), **kw)


def test_plain_model_invariants():
    """The restatement itself: causal; equal tokens are told apart by the distance bias; the matrix of the connections is
    indexed from row to column; which layer's values are kept matters."""
    cfg = full_cfg()
    w = random_tensors(cfg, seed=1)
    t = np.random.default_rng(0).integers(0, cfg["vocab"], size=90).tolist()
    full = R.forward(cfg, w, t).numpy()
    part = R.forward(cfg, w, t[:47]).numpy()
    assert np.abs(full[:47] - part).max() < 1e-9
    for name in ("l1.hc2.mix", "l0.hc1.mix"):
        w2 = dict(w)
        w2[name] = w[name].T.contiguous()
        assert np.abs(R.forward(cfg, w2, t).numpy() - full).max() > 1e-3
    w2 = dict(w)
    w2["l2.mix.vmix"] = torch.zeros_like(w["l2.mix.vmix"])
    assert np.abs(R.forward(cfg, w2, t).numpy() - full).max() > 1e-3
    w2["l1.mix.vmix"] = torch.zeros_like(w["l1.mix.vmix"])          # the first mixing layer keeps its own values
    w3 = dict(w2)
    w3["l1.mix.vmix"] = w["l1.mix.vmix"]
    assert np.abs(R.forward(cfg, w2, t).numpy() - R.forward(cfg, w3, t).numpy()).max() == 0.0


def test_plain_mechanisms():
    g = torch.Generator().manual_seed(2)
    x = torch.randn(5, 9, generator=g, dtype=torch.float64) + 3.0
    n = R.layer_norm(x, torch.ones(9), torch.zeros(9), 0.0)
    assert torch.allclose(n.mean(-1), torch.zeros(5, dtype=torch.float64), atol=1e-12)
    assert torch.allclose((n * n).mean(-1), torch.ones(5, dtype=torch.float64))
    streams = [torch.randn(2, 3, generator=g, dtype=torch.float64) for _ in range(2)]
    mix = torch.tensor([[0.0, 1.0], [0.0, 0.0]], dtype=torch.float64)  # stream 0 goes to stream 1, nothing to stream 0
    new = R.update_streams(streams, mix, torch.tensor([2.0, 0.0], dtype=torch.float64), torch.ones(2, 3, dtype=torch.float64))
    assert torch.equal(new[0], torch.full((2, 3), 2.0, dtype=torch.float64)) and torch.equal(new[1], streams[0])
    # the group with the best single member loses to the one with the better pair
    z = torch.logit(torch.tensor([0.9, 0.05, 0.6, 0.5, 0.3, 0.2], dtype=torch.float64))
    idx, wt = R.route(z, 2, 3, 1)
    assert idx == [2, 3] and math.isclose(float(wt[0]), 0.6 / 1.1, rel_tol=1e-12)
    assert R.route(z, 2)[0] == [0, 2]
    assert [R.distance_bucket(n, 8, 16) for n in (0, 3, 4, 5, 6, 8, 11, 12, 16, 99)] == [0, 3, 4, 4, 5, 6, 6, 7, 7, 7]
    rel = torch.arange(8, dtype=torch.float64).reshape(8, 1)
    b = R.distance_bias_rows(rel, [3], 5, 16)
    assert b[0, 0].tolist() == [3.0, 2.0, 1.0, 0.0, 0.0]
    assert torch.allclose(R.gelu(torch.tensor([0.0, 10.0, -10.0, 1.0], dtype=torch.float64)),
                          torch.tensor([0.0, 10.0, 0.0, 0.8413447460685429], dtype=torch.float64), atol=1e-12)


def test_random_layers_are_consistent():
    for seed in range(30):
        layers = random_layers(np.random.default_rng(seed), 6)
        mixing = {(L["mixer"]["kv_heads"], L["mixer"]["vdim"]) for L in layers if L["mixer"]["v_mix"]}
        assert len(mixing) <= 1
        for L in layers:
            m, mlp = L["mixer"], L["mlp"]
            assert m["heads"] % m["kv_heads"] == 0 and m["bias_max"] > m["buckets"] // 2
            if mlp and mlp["kind"] == "moe":
                r, g = mlp["router"], mlp["router"].get("groups")
                assert not g or (r["experts"] % g["count"] == 0 and r["top"] <= r["experts"] // g["count"] * g["keep"])
    assert moe_cfg(groups=None)["router"].get("groups") is None
