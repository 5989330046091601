"""Host side of Latodra: configuration, layer runs, tensor names, rotary frequencies, states; the plain implementation on closed forms."""
import copy
import math

import pytest
import torch

import latent_cases as H


def test_registry_and_configuration():
    import model_registry as R
    from hybrid_model import HybridConfig, Latodra, tensor_shapes
    cfg = H.CONFIGS["loop_inside"]
    assert R.model_class(cfg) is Latodra
    assert R.check_dtype(cfg, "float32") == torch.float32
    c = HybridConfig.from_dict(cfg)
    assert c.runs() == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (1, 2), (2, None), (3, None)]
    s = tensor_shapes(cfg)
    assert s["loop.step"] == (3, 64) and "l2.norm2" not in s and "l2.ls2" not in s and "head" not in s and s["l0.norm1b"] == (64,)
    assert s["l1.mix.dkv"] == (72 + 16, 64) and s["l1.mix.uq"] == (3 * 40, 56) and s["l1.mix.sink"] == (3,) and "l1.mix.g" not in s
    assert s["l0.mix.dkv"] == (48, 64) and s["l0.mix.g"] == (80, 64) and "l0.mix.sink" not in s
    assert "loop.step" not in tensor_shapes(H.CONFIGS["no_loop"])
    for bad in ((0, 0, 2), (1, 5, 2), (1, 3, 0), (-1, 2, 2)):
        b = copy.deepcopy(cfg)
        b["loop"] = dict(zip(("start", "stop", "times"), bad))
        with pytest.raises(ValueError):
            HybridConfig.from_dict(b)
    b = copy.deepcopy(cfg)
    b["layers"][0]["mlp"]["kind"] = "other"
    with pytest.raises(ValueError, match="feed-forward"):
        HybridConfig.from_dict(b)


@pytest.mark.parametrize("name", list(H.CONFIGS))
def test_runs_are_the_oracles(name):
    import latodra_oracle as O
    from hybrid_model import HybridConfig
    assert HybridConfig.from_dict(H.CONFIGS[name]).runs() == O.layer_runs(H.CONFIGS[name])


@pytest.mark.parametrize("entry", [H.rot(64, 1e4, None), H.rot(64, 1e4, (8.0, 4096, 32.0, 1.0)), H.rot(16), H.rot(2, 7.0, (2.0, 9, 1.0, 1.0)), H.rot(128, 5e5, (1.0, 128, 30.0, 2.0)),
                                   H.rot(40, 50.0, (16.0, 4, 100.0, 1e-3)), H.rot(24, 1e6, (4.0, 100000, 1e-2, 1e-3))])
def test_rotary_frequencies(entry):
    import latodra_oracle as O
    import mixers
    got, want = mixers.rotary_frequencies(entry), O.yarn_frequencies(entry)
    assert got[1] == pytest.approx(want[1], rel=1e-14) and got[0] == pytest.approx(want[0], rel=1e-12)
    if "scaling" in entry:                       # between the plain frequency and the divided one
        fac = entry["scaling"]["factor"]
        for i, f in enumerate(got[0]):
            p = entry["base"] ** (-2 * i / entry["dims"])
            assert p / fac * (1 - 1e-12) <= f <= p * (1 + 1e-12)


def test_state_holds_the_latent_and_the_shared_key_part_only():
    import mixers
    mc = H.turned()["mixer"]
    m = mixers.LatentAttention.__new__(mixers.LatentAttention)
    m.R, m.dr = mc["kv_rank"], mc["rot_dim"]
    assert {k: s.shape for k, s in m.state_spec().items()} == {"c": ("T_max", 72), "kr": ("T_max", 16)}
    m.dr = 0
    assert list(m.state_spec()) == ["c"]


def test_oracle_against_closed_forms():
    import latodra_oracle as O
    d = torch.float64
    torch.manual_seed(0)
    # a turn keeps lengths (times the factor), position 0 only scales, and products depend on the difference of positions
    e = H.rot(8, 100.0)
    x, y = torch.randn(1, 8, dtype=d), torch.randn(1, 8, dtype=d)
    m = O.yarn_frequencies(e)[1]
    assert torch.allclose(O.rotate(x, [0], e), m * x)
    assert torch.allclose(O.rotate(x, [77], e).norm(), m * x.norm())
    assert torch.allclose((O.rotate(x, [12], e) * O.rotate(y, [5], e)).sum(), (O.rotate(x, [107], e) * O.rotate(y, [100], e)).sum())
    e = H.rot(4, 9.0, None)
    z = O.rotate(torch.tensor([[1.0, 0, 0, 0, 5.0]], dtype=d), [2], e)
    assert torch.allclose(z, torch.tensor([[math.cos(2), math.sin(2), 0, 0, 5.0]], dtype=d))
    # a sink as high as the one score takes half; a low one nothing; without it the rows sum to one
    s = torch.full((3, 3), 2.0, dtype=d)
    w = O.causal_softmax(s, torch.tensor(2.0, dtype=d))
    assert torch.allclose(w.sum(-1), torch.tensor([1 / 2, 2 / 3, 3 / 4], dtype=d)) and w[0, 1] == 0
    assert torch.allclose(O.causal_softmax(s, torch.tensor(-60.0, dtype=d)), O.causal_softmax(s))
    assert torch.allclose(O.gelu_tanh(torch.tensor([0.0, 10.0, -10.0], dtype=d)), torch.tensor([0.0, 10.0, 0.0], dtype=d))


def test_oracle_is_causal():
    cfg = H.CONFIGS["loop_inside"]
    W = H.weights(cfg, 3)
    t = H.tokens(cfg, 12)
    a = H.expected(cfg, W, t)
    t2 = t[:8] + [(x + 1) % cfg["vocab"] for x in t[8:]]
    b = H.expected(cfg, W, t2)
    assert torch.equal(a[:8], b[:8]) and (a[8:] - b[8:]).abs().min(-1).values.max() > 0
