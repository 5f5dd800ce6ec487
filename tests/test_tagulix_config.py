"""Tagulix without a GPU: configuration keys and their errors, the tensors a checkpoint must hold, the parts and the schedule that a
configuration becomes, and the plain implementation's own mechanisms against hand-made cases."""

from __future__ import annotations

import copy
import math

import pytest
import torch

from research_2_b200 import models  # noqa: F401  (registers the architectures)
from research_2_b200.config.registry import ConfigError, architecture_of
from research_2_b200.config.tagulix import BiasedAttention, TagulixConfig, WindowAttention
from research_2_b200.models.tagulix import model_spec, random_weights, weight_spec
from research_2_b200.weights.loader import WeightError, check_and_select
from tests.plain import tagulix_plain as plain
from tests.tagulix_cases import CASES, moe, random_case

F64 = torch.float64


def test_every_case_parses_and_round_trips():
    for name, case in list(CASES.items()) + [(f"seed {s}", random_case(s)) for s in range(100, 140)]:
        arch = architecture_of(case["config"])
        cfg = arch.parse_config(case["config"])
        assert arch.name == "Tagulix" and isinstance(cfg, TagulixConfig)
        assert arch.parse_config(arch.config_to_json(cfg)) == cfg, name
        spec = model_spec(cfg)
        assert len(spec.schedule) == len(cfg.layers) and len(spec.layers) == sum(layer.weights_of is None for layer in cfg.layers)


def test_what_a_file_does_not_mention_is_not_there():
    cfg = TagulixConfig.from_json(CASES["c"]["config"])
    assert (cfg.streams, cfg.residual_mult) == (0, 1.0) and not any(".hc" in t.name for t in weight_spec(cfg).tensors)
    assert cfg.layers[0].mixer.left.temp_coef == 0.0 and cfg.layers[0].mlp.scale == 1.0 and cfg.layers[1].mlp is None
    assert model_spec(cfg).layers[0].block_weights == {}
    cfg = TagulixConfig.from_json(CASES["b"]["config"])
    e = cfg.layers[0].mlp
    assert (e.identity, e.groups, e.keep_groups, e.scale) == (0, 1, 1, 1.0) and cfg.layers[2].mixer.window == 0 and cfg.layers[4].mixer.rot is None
    assert not any(t.name.startswith("l3.") and ("norm2" in t.name or "hc2" in t.name) for t in weight_spec(cfg).tensors), "no feed-forward"
    mixer = WindowAttention.from_json({"heads": 6, "dim": 9, "scale": 0.1, "mask": None}, "")
    assert (mixer.kv_heads, mixer.vdim, mixer.window) == (6, 9, 0)
    assert BiasedAttention.from_json({"heads": 6, "dim": 9, "scale": 0.1, "bias_max": 7}, "").vdim == 9


@pytest.mark.parametrize("path, value, text", [
    (("vocab",), None, "vocab"), (("width",), 0, "width"), (("norm", "eps"), -1.0, "eps"), (("streams",), 0, "streams"), (("residual_mult",), "x", "residual_mult"),
    (("layers",), [], "layers"), (("layers", 1, "type"), "mamba", "type"), (("layers", 1, "mixer", "left", "heads"), 3, "multiple"),
    (("layers", 2, "mixer", "scale"), None, "scale"), (("layers", 2, "mixer", "rot", "dims"), 7, "dims"), (("layers", 2, "mixer", "rot", "base"), None, "base"),
    (("layers", 2, "mixer", "mask", "size"), 0, "size"), (("layers", 1, "mixer", "left", "bias_max"), None, "bias_max"), (("layers", 1, "mixer", "left_scale"), "x", "left_scale"),
    (("layers", 1, "mixer", "left", "q_temp", "every"), 0, "every"), (("layers", 1, "mixer", "left", "q_temp", "coef"), None, "coef"),
    (("layers", 1, "mixer", "right", "decay"), [0.5], "decay"), (("layers", 1, "mixer", "right", "decay"), [0.5, "x"], "decay"), (("layers", 1, "mixer", "right"), None, "right"),
    (("layers", 2, "mlp", "kind"), "dense", "kind"), (("layers", 2, "mlp", "expert", "ff"), None, "ff"), (("layers", 2, "mlp", "router", "top"), 5, "top"),
    (("layers", 2, "mlp", "router", "groups", "count"), 3, "groups"), (("layers", 2, "mlp", "router", "identity"), -1, "identity"), (("layers", 2, "mlp", "router", "experts"), None, "experts"),
    (("layers", 0, "weights_of"), 1, "another layer"), (("layers", 0, "weights_of"), 0, "weights_of"), (("layers", 2, "weights_of"), 0, "circle"),
])
def test_errors_name_the_key(path, value, text):
    data = copy.deepcopy(CASES["a"]["config"])
    at = data
    for key in path[:-1]:
        at = at[key]
    if value is None:
        del at[path[-1]]
    else:
        at[path[-1]] = value
    with pytest.raises(ConfigError, match=text):
        TagulixConfig.from_json(data)


def test_borrowed_layers_run_with_their_lenders_parts_and_memory_of_their_own():
    cfg = TagulixConfig.from_json(CASES["a"]["config"])
    assert [cfg.owner(i) for i in range(6)] == [2, 1, 2, 3, 1, 2], "a borrower of a borrower uses the owner's tensors"
    spec = model_spec(cfg)
    assert [e.layer for e in spec.schedule] == [1, 0, 1, 2, 0, 1] and [e.cache for e in spec.schedule] == list(range(6))
    assert [e.state for e in spec.schedule] == [None, 0, None, None, 1, None]
    names = {t.name.split(".")[0] for t in weight_spec(cfg).tensors}
    assert names == {"embed", "head", "final", "l1", "l2", "l3"}


def test_weights_fit_the_spec():
    for case in CASES.values():
        cfg = TagulixConfig.from_json(case["config"])
        w = random_weights(cfg, 1, bias_rows=case["bias_rows"])
        assert set(check_and_select(w, weight_spec(cfg))) == set(w)
        broken = {**w, "l0.norm9": torch.zeros(3)}
        del broken["head"]
        with pytest.raises(WeightError, match="(?s)head.*norm9"):
            check_and_select(broken, weight_spec(cfg))
    cfg = TagulixConfig.from_json(CASES["a"]["config"])
    w = random_weights(cfg, 1, bias_rows=10)
    assert w["l1.mix.left.rel"].shape == (10, 4) and w["l2.mlp.router"].shape == (8, 64) and w["l2.hc2.mix"].shape == (3, 3)
    with pytest.raises(WeightError, match="hc1.mix"):
        check_and_select({**w, "l1.hc1.mix": torch.zeros(3, 2)}, weight_spec(cfg))


def test_plain_temperature_buckets_and_rotation():
    assert plain.query_temperature(0, 0.5, 64) == 1.0 == plain.query_temperature(62, 0.5, 64)
    assert plain.query_temperature(63, 0.5, 64) == 1.0 + 0.5 * math.log(2) and plain.query_temperature(127, 2.0, 64) == 1.0 + 2.0 * math.log(3)
    assert [plain.distance_bucket(n, 8, 16) for n in range(18)] == [0, 1, 2, 3, 4, 4, 5, 5, 6, 6, 6, 6, 7, 7, 7, 7, 7, 7]
    x = torch.tensor([[[1.0, 0.0, 0.0, 2.0, 5.0]]], dtype=F64)
    out = plain.rotate_pairs(x, [3], 4, 100.0)[0, 0]
    want = [math.cos(3), math.sin(3), -2 * math.sin(0.3), 2 * math.cos(0.3), 5.0]     # (pairs (0, 1) and (2, 3), angles 3 and 3 / 10)
    assert torch.allclose(out, torch.tensor(want, dtype=F64))


def test_plain_window_bias_and_sink():
    """Equal keys and queries: the weights are the biases' and the sink's alone, inside the row's window."""
    T, window = 7, 3
    q, k, v = torch.zeros(T, 1, 2, dtype=F64), torch.zeros(T, 1, 2, dtype=F64), torch.eye(T, dtype=F64)[:, None, :]
    bias = torch.log(torch.tensor([[1.0, 2.0, 4.0] + [100.0] * 9], dtype=F64))
    out = plain.attend(q, k, v, 1.0, window=window, bias=bias, sink=torch.log(torch.tensor([3.0], dtype=F64)))[:, 0]
    for i in range(T):
        seen = {j: [1.0, 2.0, 4.0][i - j] for j in range(max(0, i - window + 1), i + 1)}
        want = torch.tensor([seen.get(j, 0.0) / (3.0 + sum(seen.values())) for j in range(T)], dtype=F64)
        assert torch.allclose(out[i], want), i


def test_plain_recurrence_and_streams_by_hand():
    one = torch.ones(3, 1, 1, dtype=F64)
    out, state = plain.decay_core(2.0 * one, one, torch.tensor([[[4.0]], [[10.0]], [[1.0]]], dtype=F64), torch.tensor([0.5], dtype=F64))
    assert out.flatten().tolist() == [8.0, 24.0, 14.0] and state.item() == 7.0     # S: 4, 2 + 10, 6 + 1
    w = {"in": torch.tensor([1.0, 2.0]), "out": torch.tensor([3.0, -1.0]), "mix": torch.tensor([[1.0, 10.0], [100.0, 1000.0]])}
    x = torch.tensor([[[1.0], [2.0]]], dtype=F64)
    new = plain.hyper(x, w, "", lambda u: 2.0 * u, 0.5)     # u = 5, y = 10: stream 0: 1 + 200 + 15, stream 1: 10 + 2000 - 5
    assert new.flatten().tolist() == [216.0, 2005.0]


def test_plain_router_by_hand():
    z = torch.log(torch.tensor([0.1, 0.2, 0.3, 0.4], dtype=F64))
    weights, gap = plain.route(z, torch.zeros(4, dtype=F64), 1, 2, 1, 2.0)
    assert weights.tolist() == [0, 0, 0, 2.0] and abs(gap - 0.1) < 1e-12
    # the correction decides who is chosen, the scores weigh
    weights, _ = plain.route(z, torch.tensor([-1.0, -1.0, -5.0, -9.0], dtype=F64), 2, 2, 1, 3.0)
    assert torch.allclose(weights, torch.tensor([1.0, 2.0, 0.0, 0.0], dtype=F64))
    # an identity output gives the row back
    h = torch.tensor([[1.0, -2.0]], dtype=F64)
    w = {"router": torch.zeros(2, 2), "correction": torch.tensor([0.0, 1.0]), "e0.up": torch.ones(3, 2), "e0.down": torch.ones(2, 3)}
    assert torch.allclose(plain.mixture(h, w, "", moe(1, 1, 1, 3, scale=1.5)), 1.5 * h)
