"""Fakelorn's configuration, description and cache needs, and the plain implementation's mechanisms against facts that can be
worked out by hand, all without a GPU."""

import copy
import math

import numpy as np
import pytest
import torch

import plain_fakelorn as pf
from fakelorn_cases import CONFIGS, as_float64, random_weights, tensor_shapes

F64 = torch.float64


def _model(cfg, dtype=torch.float32):
    from rusty_llama_b200.models.model import Model
    from rusty_llama_b200.parts.base import Runtime
    from rusty_llama_b200.registry import describe_model

    return Model(describe_model(cfg), Runtime.create("cpu", dtype))


@pytest.mark.parametrize("name", list(CONFIGS))
def test_the_described_model_asks_for_the_checkpoints_tensors(name):
    cfg = CONFIGS[name]()
    want = tensor_shapes(cfg)
    for dtype in (torch.float32, torch.bfloat16):
        got = {k: tuple(v.shape) for k, v in _model(cfg, dtype).param_infos().items()}
        assert set(got) == set(want)
        for k, shape in want.items():
            assert got[k] == tuple(shape), (k, got[k], shape)


def test_cache_needs_follow_the_layers():
    from rusty_llama_b200.cache import Cache
    from rusty_llama_b200.parts.base import KVNeed, StateNeed

    model = _model(CONFIGS["a"]())
    needs = dict(model.cache_needs())
    assert needs[0] == (StateNeed((3, 24, 20), torch.float32), StateNeed((2, 3 * 20 + 2 * 24), torch.float32))
    assert needs[1] == KVNeed(1, 24 + 8, 0, values=False)
    assert needs[2] == KVNeed(2, 20, 33, value_dim=12)  # a kv head's two keys as one row, its value once
    assert needs[3] == KVNeed(1, 40 + 8, 0, values=False)
    assert 4 not in needs  # reads layer 1's latents
    assert needs[5] == KVNeed(2, 16, 0, value_dim=8)
    assert dict(_model(CONFIGS["b"]()).cache_needs())[2] == StateNeed((1, 40, 36), torch.float32)  # a convolution of one tap keeps no inputs
    cache = Cache(model.cache_needs(), 64 * 4, 2, torch.float32, "cpu")
    s = cache.open_sequence()
    cache.view(0)[0].state[s] += 1.0
    cache.view(0)[1].state[s] += 1.0
    cache.reserve([s], [100])
    cache.commit([s], [100])
    cache.check_consistent()
    cache.close_sequence(s)
    assert cache.open_sequence() == s  # the slot is used again, and its records read zero
    assert float(cache.view(0)[0].state[s].abs().sum()) == 0.0 and float(cache.view(0)[1].state[s].abs().sum()) == 0.0


def test_description_names_the_parts():
    from rusty_llama_b200.registry import describe_model

    spec = describe_model(CONFIGS["a"]())
    assert [e.cache_from for e in spec.schedule] == [None, None, None, None, 1, None]
    assert all(layer.block == "gated_prenorm" for layer in spec.layers)
    assert spec.layers[0].norms["mixer"].params["groups"] == 3 and spec.final_norm.params["groups"] == 3
    assert spec.head.params["tied_to"] == "embed" and spec.head.params["scale"] == 0.25 and spec.head.params["softcap"] == 5.0
    assert describe_model(CONFIGS["b"]()).head.params["softcap"] == 0.0


def test_configuration_errors_are_named():
    from rusty_llama_b200.errors import ConfigError
    from rusty_llama_b200.registry import describe_model

    def broken(change):
        cfg = copy.deepcopy(CONFIGS["a"]())
        change(cfg)
        with pytest.raises(ConfigError):
            describe_model(cfg)

    broken(lambda c: c["layers"][0].update(type="lightning"))
    broken(lambda c: c["layers"][0]["mixer"].update(groups=2))
    broken(lambda c: c["layers"][0]["mixer"].update(norm_groups=7))
    broken(lambda c: c["layers"][2]["mixer"].update(kv_heads=4))
    broken(lambda c: c["layers"][2]["mixer"].update(mask={"size": 0}))
    broken(lambda c: c["layers"][2]["mixer"].pop("diff"))
    broken(lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7))
    broken(lambda c: c["layers"][4]["mixer"].update(kv_from=3))  # another latent size
    broken(lambda c: c["layers"][4]["mixer"].update(kv_from=2))  # no latents there
    broken(lambda c: c["layers"][4]["mixer"].update(kv_from=5))  # runs later
    broken(lambda c: c["layers"][4]["mixer"]["rot"].update(base=501.0))
    broken(lambda c: c["layers"][1]["mlp"]["router"].update(top=6))
    broken(lambda c: c["layers"][0]["mlp"].update(kind="glu"))
    broken(lambda c: c["norm"].update(groups=5))
    broken(lambda c: c.update(logit_softcap=-1.0))
    broken(lambda c: c.pop("width"))


def test_norm_in_groups_divides_every_part_by_its_own_root_mean_square():
    x = torch.tensor([[3.0, 4.0, 30.0, 40.0]], dtype=F64)
    w = torch.tensor([1.0, 2.0, 1.0, -1.0], dtype=F64)
    r = math.sqrt(12.5)
    assert torch.allclose(pf.grouped_norm(x, w, 2, 0.0), torch.tensor([[3 / r, 8 / r, 3 / r, -4 / r]], dtype=F64))
    assert torch.allclose(pf.grouped_norm(x, torch.ones(4, dtype=F64), 1, 0.0), pf.rms(x, 0.0))
    assert pf.rms(torch.zeros(1, 2, dtype=F64), 1e-6).abs().sum() == 0.0  # eps inside the root


def test_rotation_pairs_halves():
    x = torch.arange(1.0, 7.0, dtype=F64).view(1, 1, 6).repeat(3, 1, 1)
    pos = torch.tensor([0, 1, 5])
    y = pf.rotate_halves(x, pos, 16.0, 4)
    assert torch.equal(y[0], x[0]) and torch.equal(y[..., 4:], x[..., 4:])
    f = [1.0, 16.0 ** -0.5]
    for i in (0, 1):
        c, s = math.cos(5 * f[i]), math.sin(5 * f[i])
        assert y[2, 0, i].item() == pytest.approx((1 + i) * c - (3 + i) * s) and y[2, 0, i + 2].item() == pytest.approx((3 + i) * c + (1 + i) * s)


def test_difference_of_two_maps_over_the_same_values():
    """Map 1 looks at key 0 only, map 2 at the last key only: the head is v_0 - lambda v_last, normed, times 1 - diff."""
    T = 4
    q = torch.zeros(T, 1, 2, 2, dtype=F64)
    k = torch.zeros(T, 1, 2, 2, dtype=F64)
    q[:, 0, 0, 0] = q[:, 0, 1, 1] = 100.0
    k[0, 0, 0, 0] = 1.0
    for t in range(T):
        k[t, 0, 1, 1] = float(t)
    v = torch.tensor([[1.0, 0.0], [0.0, 1.0], [2.0, 2.0], [0.0, -4.0]], dtype=F64).view(T, 1, 2)
    a1, a2 = pf.differential_maps(q, k, v, 1.0, 0)
    assert torch.allclose(a1[3, 0], v[0, 0]) and torch.allclose(a2[3, 0], v[3, 0])
    o = pf.combine_maps(a1, a2, 0.5, 0.2, 0.0)
    raw = torch.tensor([1.0, 2.0], dtype=F64)  # v_0 - v_3 / 2
    assert torch.allclose(o[3, 0], raw / math.sqrt(2.5) * 0.8)
    # a window of two hides key 0 from token 3: map 1 then spreads over what is left
    a1, _ = pf.differential_maps(q, k, v, 1.0, 2)
    assert torch.allclose(a1[3, 0], (v[2, 0] + v[3, 0]) / 2)
    W = {"lq1": torch.tensor([1.0, 0.0]), "lk1": torch.tensor([math.log(3.0), 5.0]), "lq2": torch.tensor([0.0, 1.0]), "lk2": torch.tensor([7.0, math.log(2.0)])}
    assert pf.lambda_of(W, "", 0.25).item() == pytest.approx(3.0 - 2.0 + 0.25)


def test_windows_edges():
    vis = pf.causal(6, 3)
    assert vis[5].tolist() == [False, False, False, True, True, True] and vis[1].tolist() == [True, True, False, False, False, False]


def test_state_space_recurrence_by_hand():
    one = torch.ones(3, 1, 1, dtype=F64)
    x = torch.tensor([1.0, 10.0, 100.0], dtype=F64).view(3, 1, 1)
    dt = torch.full((3, 1), 2.0, dtype=F64)
    rate = torch.tensor([math.log(math.log(2.0) / 2.0)], dtype=F64)  # exp(rate) dt = log 2: the state halves every token
    y = pf.ssm_recurrence(x, one, one, dt, rate, torch.tensor([0.5], dtype=F64))
    assert y.view(3).tolist() == pytest.approx([2 * 1 + 0.5, 2 * 10.5 + 5.0, 2 * 105.25 + 50.0])
    # heads of one group read the same B and C
    xs = torch.randn(5, 4, 3, dtype=F64)
    B, C = torch.randn(5, 2, 6, dtype=F64), torch.randn(5, 2, 6, dtype=F64)
    dts, r, D = torch.rand(5, 4, dtype=F64), torch.randn(4, dtype=F64), torch.randn(4, dtype=F64)
    y = pf.ssm_recurrence(xs, B, C, dts, r, D)
    alone = pf.ssm_recurrence(xs[:, 3:], B[:, 1:], C[:, 1:], dts[:, 3:], r[3:], D[3:])
    assert torch.allclose(y[:, 3:], alone)


def test_short_convolution_sees_the_past_only_and_the_gate_comes_before_the_norm():
    x = torch.tensor([[1.0], [10.0], [100.0], [1000.0]], dtype=F64)
    w = torch.tensor([[3.0, 2.0, 1.0]], dtype=F64)  # the last column is the current token's
    assert pf.short_convolution(x, w, torch.tensor([0.5], dtype=F64))[:, 0].tolist() == [1.5, 12.5, 123.5, 1230.5]
    y, z = torch.tensor([[1.0, 1.0]], dtype=F64), torch.tensor([[20.0, -20.0]], dtype=F64)
    o = pf.gate_then_norm(y, z, torch.ones(2, dtype=F64), 1, 0.0)
    assert o[0, 0].item() == pytest.approx(math.sqrt(2.0)) and abs(o[0, 1].item()) < 1e-6  # the norm sees the gated numbers


def test_router_weights_are_a_softmax_over_the_chosen_logits_only():
    h = torch.eye(3, dtype=F64)
    W = {"r.router": torch.tensor([[0.0, 2.0, -2.0], [1.0, 0.0, 0.0], [-1.0, 0.0, 3.0]], dtype=F64)}
    chosen, w = pf.route(h, W, "r.", 2)
    assert chosen.tolist() == [[1, 0], [0, 1], [2, 1]]
    assert w[0].tolist() == pytest.approx([math.e / (1 + math.e), 1 / (1 + math.e)])
    assert w.sum(dim=1).tolist() == pytest.approx([1.0, 1.0, 1.0])


def test_logits_are_scaled_before_they_are_capped():
    assert pf.cap_logits(torch.tensor([3.0], dtype=F64), 2.0, 5.0).item() == pytest.approx(5.0 * math.tanh(6.0 / 5.0))
    assert pf.cap_logits(torch.tensor([3.0], dtype=F64), 2.0, 0.0).item() == 6.0


def test_the_plain_model_runs_every_configuration():
    for i, (name, make) in enumerate(CONFIGS.items()):
        cfg = make()
        w = as_float64(random_weights(cfg, seed=5 + i))
        toks = np.random.default_rng(i).integers(0, cfg["vocab"], 40).tolist()
        logits, after = pf.plain_streams(cfg, w, toks)
        assert logits.shape == (40, cfg["vocab"]) and after.shape == (len(cfg["layers"]), 40, cfg["width"])
        assert torch.isfinite(logits).all()
        # causal: the first 25 positions do not change when the rest is replaced
        other = toks[:25] + np.random.default_rng(99).integers(0, cfg["vocab"], 15).tolist()
        assert torch.allclose(pf.plain_logits(cfg, w, other)[:25], logits[:25], rtol=0, atol=1e-9)
