"""Lagelorn without a GPU: configuration keys and their errors, the tensors a checkpoint must hold (two sizes are its own), the
parts that a configuration becomes, the cache groups that they ask for, and the plain implementation's own mechanisms
against hand-made cases."""

from __future__ import annotations

import copy
import math

import pytest
import torch

from research_2_b200 import models  # noqa: F401  (registers the architectures)
from research_2_b200.cache.arena import MemberSpec, derive_groups
from research_2_b200.cache.manager import CacheManager, GroupSpec
from research_2_b200.config.lagelorn import ChunkAttention, DeltaMixer, LagelornConfig
from research_2_b200.config.registry import ConfigError, architecture_of
from research_2_b200.models.lagelorn import model_spec, random_weights, weight_spec
from research_2_b200.parts.attention import distance_buckets
from research_2_b200.weights.loader import TensorSpec, WeightError, WeightSpec, check_and_select
from tests.lagelorn_cases import CASES, random_case
from tests.plain import lagelorn_plain as plain

F64 = torch.float64


def test_every_case_parses_and_round_trips():
    for name, case in list(CASES.items()) + [(f"seed {s}", random_case(s)) for s in range(100, 140)]:
        arch = architecture_of(case["config"])
        cfg = arch.parse_config(case["config"])
        assert arch.name == "Lagelorn" and isinstance(cfg, LagelornConfig)
        assert arch.parse_config(arch.config_to_json(cfg)) == cfg, name
        spec = model_spec(cfg)
        assert spec.max_seq_len == cfg.max_positions and len(spec.layers) == len(cfg.layers)


def test_what_a_file_does_not_mention_is_not_there():
    cfg = LagelornConfig.from_json(CASES["c"]["config"])
    assert cfg.alpha == 1.0 and cfg.logit_softcap == 0.0 and cfg.side_dim == 24 and cfg.layers[0].mlp is None
    cfg = LagelornConfig.from_json(CASES["b"]["config"])
    assert cfg.side_dim == 0 and cfg.layers[3].mixer.left.chunk == 0
    spec = model_spec(cfg)
    assert all(layer.token_side is None for layer in spec.layers) and spec.logit_softcap == 7.0
    assert not any("side" in t.name for t in weight_spec(cfg).tensors)
    mixer = DeltaMixer.from_json({"heads": 6, "dim": 9, "conv": 3}, "")
    assert (mixer.kv_heads, mixer.vdim) == (6, 9)
    left = ChunkAttention.from_json({"heads": 6, "dim": 9, "scale": 0.1, "bias_max": 30, "mask": None}, "")
    assert (left.kv_heads, left.chunk) == (6, 0)


@pytest.mark.parametrize("path, value, text", [
    (("vocab",), None, "vocab"), (("width",), 0, "width"), (("max_positions",), None, "max_positions"), (("norm", "eps"), -1.0, "eps"),
    (("layers", 0, "type"), "mamba", "type"), (("layers", 0, "mixer", "left", "heads"), 3, "multiple"),
    (("layers", 0, "mixer", "left", "vdim"), 8, "vdim"), (("layers", 0, "mixer", "left", "scale"), None, "scale"),
    (("layers", 0, "mixer", "left", "bias_max"), None, "bias_max"), (("layers", 0, "mixer", "left_scale"), "x", "left_scale"),
    (("layers", 0, "mixer", "left", "mask"), 5, "mask"), (("layers", 0, "mixer", "right", "dim"), None, "dim"),
    (("layers", 0, "mixer", "right"), None, "right"), (("layers", 1, "mixer", "conv"), 0, "conv"), (("layers", 1, "mixer", "kv_heads"), 3, "multiple"),
    (("layers", 0, "mlp", "kind"), "moe", "kind"), (("layers", 0, "mlp", "ff"), None, "ff"), (("token_side", "dim"), 0, "dim"),
    (("logit_softcap",), -2.0, "logit_softcap"), (("layers",), [], "layers"),
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
        LagelornConfig.from_json(data)


def test_weights_fit_the_spec_and_the_checkpoint_has_its_own_sizes():
    for name, case in CASES.items():
        cfg = LagelornConfig.from_json(case["config"])
        w = random_weights(cfg, 1, bias_rows=case["bias_rows"], decay_rank=case["decay_rank"])
        picked = check_and_select(w, weight_spec(cfg))
        assert set(picked) == set(w)
        _, i = min((layer.type != "parallel", i) for i, layer in enumerate(cfg.layers))
        assert w[f"l{i}.mix.left.rel"].shape[0] == case["bias_rows"] and w[f"l{i}.mix.right.w1"].shape[0] == case["decay_rank"]
        # the two small matrices of one layer agree on the size that is theirs; another layer may have another
        broken = dict(w)
        broken[f"l{i}.mix.right.w2"] = torch.zeros(w[f"l{i}.mix.right.w2"].shape[0], case["decay_rank"] + 1)
        with pytest.raises(WeightError, match="right.w2"):
            check_and_select(broken, weight_spec(cfg))
        broken[f"l{i}.mix.right.w1"] = torch.zeros(case["decay_rank"] + 1, cfg.width)
        check_and_select(broken, weight_spec(cfg))
        broken["l0.norm9"] = torch.zeros(3)
        del broken["head"]
        with pytest.raises(WeightError, match="(?s)head.*norm9"):
            check_and_select(broken, weight_spec(cfg))


def test_named_sizes():
    spec = WeightSpec(tensors=(TensorSpec("a", ("n", 3)), TensorSpec("b", ("n", "n")), TensorSpec("c", ("m",))))
    t = torch.zeros
    check_and_select({"a": t(5, 3), "b": t(5, 5), "c": t(2)}, spec)
    for bad in ({"a": t(5, 3), "b": t(5, 4), "c": t(2)}, {"a": t(5, 4), "b": t(5, 5), "c": t(2)}, {"a": t(5, 3), "b": t(5), "c": t(2)}):
        with pytest.raises(WeightError):
            check_and_select(bad, spec)


def test_buckets_of_distances():
    """The first half of the rows are distances of their own, then equal steps of the logarithm up to bias_max."""
    for rows, bias_max in ((4, 9), (8, 20), (16, 128), (32, 128), (12, 50), (6, 4), (2, 5)):
        got = distance_buckets(3 * bias_max, rows, bias_max)
        half = rows // 2
        assert got == [plain.distance_bucket(n, rows, bias_max) for n in range(3 * bias_max)]
        assert got[:half] == list(range(half)) and got[bias_max:] == [rows - 1] * (2 * bias_max)
        assert all(a <= b for a, b in zip(got, got[1:]))
        for n in range(half, bias_max):   # (in whole numbers: row half + k begins where (n / half)^(rows - half) reaches (bias_max / half)^k)
            k = got[n] - half
            assert n ** (rows - half) * half ** k >= bias_max ** k * half ** (rows - half)
            if got[n] < rows - 1:
                assert n ** (rows - half) * half ** (k + 1) < bias_max ** (k + 1) * half ** (rows - half)
    assert distance_buckets(40, 8, 16)[:18] == [0, 1, 2, 3, 4, 4, 5, 5, 6, 6, 6, 6, 7, 7, 7, 7, 7, 7]
    for rows, bias_max in ((8, 4), (8, 3), (1, 9)):
        with pytest.raises(ValueError):
            distance_buckets(10, rows, bias_max)


def test_layers_share_cache_groups_by_their_chunks():
    members = [MemberSpec(2, 16, chunk=24), MemberSpec(2, 32, chunk=40), MemberSpec(1, 8, chunk=24), MemberSpec(1, 8), MemberSpec(1, 8, 24)]
    groups, index = derive_groups(members, 8, 30)
    assert index == [0, 1, 0, 2, 3] and [(g.window, g.chunk) for g in groups] == [(0, 24), (0, 40), (0, 0), (24, 0)]
    with pytest.raises(ValueError):
        CacheManager([GroupSpec(4, 6, 8, chunk=8)], 1, 64)
    with pytest.raises(ValueError):
        CacheManager([GroupSpec(4, 0, 8, chunk=-1)], 1, 64)


@pytest.mark.parametrize("page, chunk", [(4, 12), (4, 10), (8, 5), (4, 4), (16, 40)])
def test_a_chunk_group_gives_pages_back_when_a_chunk_is_left(page, chunk):
    for step in (1, 3, 7):
        cm = CacheManager([GroupSpec(page, 0, 64, chunk=chunk), GroupSpec(page, 0, 64)], 2, 200)
        cm.open(0)
        held = []
        for start in range(0, 100, step):
            cm.slide(0, start)
            end = min(start + step, 100)
            cm.reserve(0, start, end)
            table = cm.table(0, 0)
            first = start // chunk * chunk // page    # the page of the first key that the step's first row reads
            assert all(table[i] == 0 for i in range(first)), "a page of an earlier chunk is still held"
            assert all(table[i] != 0 for i in range(first, -(-end // page))), "a page that a row reads is missing"
            assert cm.pages_held(0, 1) == -(-end // page) and cm.check() == ""
            held.append(cm.pages_held(0, 0))
        if step == 1:
            assert max(held) <= cm.worst_pages(0, 100, 1) <= chunk // page + 2
        assert cm.worst_pages(0, 100, 16, page) <= (chunk + 16) // page + 2 and cm.worst_pages(1, 100, 16, page) == -(-100 // page)
        cm.close(0)
        assert cm.n_free(0) == 64 and cm.n_free(1) == 64


def test_plain_delta_rule_by_hand():
    """One head of one key and one value dimension: numbers that can be followed."""
    g, beta = torch.tensor([[0.5], [0.25]], dtype=F64), torch.tensor([[0.5], [1.0]], dtype=F64)
    one = torch.ones(2, 1, 1, dtype=F64)
    v = torch.tensor([[[4.0]], [[10.0]]], dtype=F64)
    out, state = plain.delta_core(3.0 * one, one, v, g, beta)
    # S: 0 -> 0 + 0.5 * 4 = 2, read 3 * 2; then 0.25 * 2 = 0.5, u = 1 * (10 - 0.5), S = 10, read 30
    assert out.flatten().tolist() == [6.0, 30.0] and state.item() == 10.0
    # in two portions
    first, s = plain.delta_core(3.0 * one[:1], one[:1], v[:1], g[:1], beta[:1])
    second, s = plain.delta_core(3.0 * one[1:], one[1:], v[1:], g[1:], beta[1:], s)
    assert torch.equal(torch.cat([first, second]), out) and torch.equal(s, state)
    # with g = 1, beta = 1 and orthonormal keys the state is a table that returns what was written
    eye = torch.eye(3, dtype=F64)[:, None, :]
    values = torch.randn(3, 1, 2, dtype=F64, generator=torch.Generator().manual_seed(1))
    ones = torch.ones(3, 1, dtype=F64)
    _, table = plain.delta_core(eye, eye, values, ones, ones)
    assert torch.allclose(table[0], values[:, 0])
    # writing a second time under the same key replaces the first value
    again, _ = plain.delta_core(eye[:1], eye[:1], values[1:2], ones[:1], ones[:1], table)
    assert torch.allclose(again[0, 0], values[1, 0])


def test_plain_time_mixing_by_hand():
    one = torch.ones(2, 1, 1, dtype=F64)
    r, k, v = 2.0 * one, torch.tensor([[[3.0]], [[1.0]]], dtype=F64), torch.tensor([[[5.0]], [[7.0]]], dtype=F64)
    w = torch.tensor([[[0.5]], [[0.1]]], dtype=F64)
    out, state = plain.time_mix_core(r, k, v, w, torch.tensor([[4.0]], dtype=F64))
    # row 0: nothing stored, the own write with bonus 4: 2 * 4 * 15; S = 15; row 1: 2 * (15 + 4 * 7); S = 0.1 * 15 + 7
    assert out.flatten().tolist() == [120.0, 86.0] and math.isclose(state.item(), 8.5)
    assert plain.shifted(torch.arange(6.0, dtype=F64).view(3, 2)).tolist() == [[0, 0], [0, 1], [2, 3]]


def test_plain_chunks_bias_and_sink():
    """Equal keys and queries: the weights are the biases' and the sink's alone, inside the row's own chunk."""
    T, chunk = 7, 3
    q, k, v = torch.zeros(T, 1, 2, dtype=F64), torch.zeros(T, 1, 2, dtype=F64), torch.eye(T, dtype=F64)[:, None, :]
    bias = torch.log(torch.tensor([[1.0, 2.0, 4.0] + [100.0] * 9], dtype=F64))
    out = plain.chunk_attention_core(q, k, v, 1.0, bias, torch.log(torch.tensor([3.0], dtype=F64)), chunk)[:, 0]
    for i in range(T):
        seen = {j: [1.0, 2.0, 4.0][i - j] for j in range(i // chunk * chunk, i + 1)}
        total = 3.0 + sum(seen.values())
        want = torch.tensor([seen.get(j, 0.0) / total for j in range(T)], dtype=F64)
        assert torch.allclose(out[i], want), i
    taps = torch.tensor([[1.0, 10.0, 100.0]])
    x = torch.tensor([[1.0], [2.0], [3.0]], dtype=F64)
    y = torch.tensor([[100.0], [210.0], [321.0]], dtype=F64)
    assert torch.allclose(plain.short_conv(x, taps), y / (1 + torch.exp(-y)))
