"""Damadra's configuration, description and cache needs, and the plain implementation's mechanisms against facts that can be
worked out by hand, all without a GPU."""

import copy
import math

import numpy as np
import pytest
import torch

import plain_damadra as pd
from damadra_cases import CONFIGS, ROWS, as_float64, random_weights, tensor_shapes

F64 = torch.float64


def _model(cfg, dtype=torch.float32):
    from rusty_llama_b200.models.model import Model
    from rusty_llama_b200.parts.base import Runtime
    from rusty_llama_b200.registry import describe_model

    return Model(describe_model(cfg), Runtime.create("cpu", dtype))


@pytest.mark.parametrize("name", list(CONFIGS))
def test_the_described_model_asks_for_the_checkpoints_tensors(name):
    cfg = CONFIGS[name]()
    want = tensor_shapes(cfg, ROWS[name])
    for dtype in (torch.float32, torch.bfloat16):
        got = {k: tuple(v.shape) for k, v in _model(cfg, dtype).param_infos().items()}
        assert set(got) == set(want)
        for k, shape in want.items():
            if k.endswith(".rel"):  # (the number of buckets is the checkpoint's to say)
                assert got[k] == (-1, shape[1])
            else:
                assert got[k] == tuple(shape), (k, got[k], shape)


def test_cache_needs_follow_the_layers():
    from rusty_llama_b200.cache import Cache
    from rusty_llama_b200.parts.base import KVNeed

    model = _model(CONFIGS["a"]())
    needs = dict(model.cache_needs())
    assert needs[0] == KVNeed(1, 10, 0, value_dim=12)
    assert needs[1] == KVNeed(2, 12, 33)
    assert needs[2] == KVNeed(2, 20, 0, value_dim=6)
    assert 3 not in needs and 5 not in needs  # read layer 0's and layer 2's keys and values
    assert needs[4] == KVNeed(2, 8, 90)
    cache = Cache(model.cache_needs(), 64 * 8, 2, torch.float32, "cpu")
    s = cache.open_sequence()
    for n in (100, 1, 90, 64):
        cache.reserve([s], [n])
        cache.commit([s], [n])
        cache.check_consistent()
    held = [sum(p >= 0 for p in g.pages[s]) for g in cache.kv_groups]
    assert held == [4, 1, 4, 2]  # 255 positions; the groups with windows of 33 and 90 gave pages back
    assert cache.view(3 - 3).k_pages.shape[-1] == 10 and not cache.owns(3)
    cache.close_sequence(s)
    cache.check_consistent()


def test_description_names_the_parts():
    from rusty_llama_b200.registry import describe_model

    spec = describe_model(CONFIGS["a"]())
    assert [e.cache_from for e in spec.schedule] == [None, None, None, 0, None, 2]
    assert all(layer.block == "postnorm" for layer in spec.layers)
    assert spec.layers[0].norms["mixer_out"].params["factor"] == 0.7 and spec.final_norm.params["factor"] == 1.0
    assert "feed_forward_out" not in spec.layers[1].norms
    assert spec.embedding.params["scale"] == 3.0 and spec.head.params["tied_to"] is None
    assert spec.layers[1].mixer.params["position"].kind == "distance_bias" and spec.layers[1].mixer.params["position"].params["max_distance"] == 29
    assert spec.layers[0].mixer.params["q_temperature"] == (0.3, 7)
    assert spec.layers[3].feed_forward.params["identity"] == 2


def test_configuration_errors_are_named():
    from rusty_llama_b200.errors import ConfigError
    from rusty_llama_b200.registry import describe_model

    def broken(change):
        cfg = copy.deepcopy(CONFIGS["a"]())
        change(cfg)
        with pytest.raises(ConfigError):
            describe_model(cfg)

    broken(lambda c: c["layers"][0].update(type="lightning"))
    broken(lambda c: c["layers"][1]["mixer"].update(kv_heads=4))
    broken(lambda c: c["layers"][1]["mixer"].update(mask={"size": 0}))
    broken(lambda c: c["layers"][1]["mixer"].update(vdim=8))  # values that are keys have their size
    broken(lambda c: c["layers"][1]["mixer"].update(kv_from=0))
    broken(lambda c: c["layers"][0]["mixer"].pop("bias_max"))
    broken(lambda c: c["layers"][0]["mixer"].pop("scale"))
    broken(lambda c: c["layers"][0]["mixer"]["q_temp"].update(every=0))
    broken(lambda c: c["layers"][3]["mixer"].update(kv_from=2))  # another key size
    broken(lambda c: c["layers"][3]["mixer"].update(kv_from=1))  # a window: not every token is kept
    broken(lambda c: c["layers"][3]["mixer"].update(kv_from=4))  # runs later
    broken(lambda c: c["layers"][5]["mixer"].update(kv_from=3))  # has none of its own
    broken(lambda c: c["layers"][0]["mlp"]["router"].update(top=8))
    broken(lambda c: c["layers"][0]["mlp"]["router"].update(identity=-1))
    broken(lambda c: c["layers"][0]["mlp"].update(kind="glu"))
    broken(lambda c: c.pop("width"))
    broken(lambda c: c["norm"].pop("eps"))


# ------------------------------------------------------------------ buckets
def test_buckets_by_hand():
    # 8 rows up to a distance of 64: 0..3 alone, then borders at 4, 8, 16, 32
    want = [0, 1, 2, 3] + [4] * 4 + [5] * 8 + [6] * 16 + [7] * 100
    assert [pd.distance_bucket(n, 8, 64) for n in range(len(want))] == want
    assert [pd.distance_bucket(n, 2, 5) for n in range(4)] == [0, 1, 1, 1]


@pytest.mark.parametrize("rows,far", [(2, 5), (4, 9), (8, 64), (16, 128), (32, 128), (12, 29), (6, 21), (26, 90), (64, 1000), (7, 40), (20, 10.5), (30, 100000)])
def test_the_table_by_distance_has_every_border(rows, far):
    """Borders that are whole numbers among them, where a quotient of two logarithms may fall just below the whole number."""
    from rusty_llama_b200.parts.position import distance_buckets

    table = distance_buckets(rows, far)
    assert table[-1] == rows - 1 and (len(table) < 2 or table[-2] < rows - 1)  # no longer than it has to be
    step = max(1, len(table) // 400)
    for n in list(range(0, len(table), step)) + [i for i in range(1, len(table)) if table[i] != table[i - 1]]:
        assert table[n] == pd.distance_bucket(n, rows, far), n
        assert n == 0 or table[n - 1] == pd.distance_bucket(n - 1, rows, far), n - 1
    assert pd.distance_bucket(10 * len(table), rows, far) == rows - 1


def test_a_table_that_cannot_reach_its_distance_is_an_error():
    from rusty_llama_b200.errors import ConfigError
    from rusty_llama_b200.parts.position import distance_buckets

    for rows, far in ((16, 8), (1, 5), (10, 3)):
        with pytest.raises(ConfigError):
            distance_buckets(rows, far)


# ------------------------------------------------------------------ the plain mechanisms
def test_bias_is_added_after_the_scale_and_by_distance():
    rel = torch.tensor([[0.0], [10.0], [0.0], [0.0]], dtype=F64)  # distance 1 stands out
    bias = pd.bias_matrix(rel, 9, 5)
    q, k = torch.zeros(5, 1, 2, dtype=F64), torch.zeros(5, 1, 2, dtype=F64)
    v = torch.arange(5.0, dtype=F64).view(5, 1, 1)
    out = pd.softmax_attention(q, k, v, 0.001, bias, 0).view(5)
    assert out[0] == 0.0 and torch.allclose(out[1:], torch.arange(4.0, dtype=F64), atol=2e-3)


def test_windows_edges():
    vis = pd.causal(6, 3)
    assert vis[5].tolist() == [False, False, False, True, True, True] and vis[1].tolist() == [True, True, False, False, False, False]


def test_query_temperature_steps_at_multiples():
    t = pd.query_temperature(torch.arange(9), 0.5, 4)
    assert t[:3].tolist() == [1.0] * 3 and torch.allclose(t[3:7], torch.full((4,), 1 + 0.5 * math.log(2.0), dtype=F64))
    assert t[7].item() == pytest.approx(1 + 0.5 * math.log(3.0))


def test_norm_over_all_heads_and_values_before_it():
    m = {"heads": 2, "kv_heads": 1, "dim": 2}
    W = {"q": torch.eye(4, dtype=F64), "k": torch.eye(4, dtype=F64)[:2], "q.norm": torch.tensor([1.0, 1.0, 2.0, 1.0], dtype=F64), "k.norm": torch.tensor([1.0, -1.0], dtype=F64)}
    q, k, v = pd.windowed_queries_keys_values(torch.tensor([[3.0, 4.0, 0.0, 5.0]], dtype=F64), W, "", m, 0.0)
    r = math.sqrt(50 / 4)
    assert torch.allclose(q[0], torch.tensor([[3 / r, 4 / r], [0.0, 5 / r]], dtype=F64))
    assert torch.allclose(k[0, 0], torch.tensor([3.0, -4.0], dtype=F64) / math.sqrt(12.5)) and v[0, 0].tolist() == [3.0, 4.0]


def test_router_weights_are_scores_without_the_correction_and_not_renormalized():
    h = torch.eye(3, dtype=F64)
    W = {"r.router": torch.tensor([[0.0, 2.0, -2.0], [1.0, 0.0, 0.0], [-1.0, 0.0, 3.0]], dtype=F64), "r.correction": torch.tensor([0.0, -1.0, 0.0], dtype=F64)}
    chosen, w = pd.route(h, W, "r.", 2)
    assert chosen.tolist() == [[0, 2], [0, 2], [2, 0]]
    s0 = torch.softmax(torch.tensor([0.0, 1.0, -1.0], dtype=F64), 0)
    assert torch.allclose(w[0], s0[[0, 2]]) and float(w[0].sum()) < 0.5


def test_identity_choices_hand_the_input_on_and_experts_square_their_relu():
    h = torch.tensor([[2.0, -1.0]], dtype=F64)
    W = {"router": torch.tensor([[0.0, 0.0], [50.0, 0.0]], dtype=F64), "correction": torch.zeros(2, dtype=F64),
         "e0.up": torch.tensor([[1.0, 0.0], [0.0, 1.0]], dtype=F64), "e0.down": torch.tensor([[1.0, 1.0], [0.0, 3.0]], dtype=F64)}
    assert torch.allclose(pd.moe_ff(h, W, "", {"experts": 1, "identity": 1, "top": 1}), h)
    assert torch.allclose(pd.expert(h, W, "e0."), torch.tensor([[4.0, 0.0]], dtype=F64))
    W["router"] = -W["router"]
    assert torch.allclose(pd.moe_ff(h, W, "", {"experts": 1, "identity": 1, "top": 1}), torch.tensor([[4.0, 0.0]], dtype=F64))


def test_the_plain_model_runs_every_configuration():
    for i, (name, make) in enumerate(CONFIGS.items()):
        cfg = make()
        w = as_float64(random_weights(cfg, ROWS[name], seed=5 + i))
        toks = np.random.default_rng(i).integers(0, cfg["vocab"], 40).tolist()
        logits, after = pd.plain_streams(cfg, w, toks)
        assert logits.shape == (40, cfg["vocab"]) and after.shape == (len(cfg["layers"]), 40, cfg["width"])
        assert torch.isfinite(logits).all()
        # causal: the first 25 positions do not change when the rest is replaced
        other = toks[:25] + np.random.default_rng(99).integers(0, cfg["vocab"], 15).tolist()
        assert torch.allclose(pd.plain_logits(cfg, w, other)[:25], logits[:25], rtol=0, atol=1e-9)
