"""Tagulix on the GPU against the plain implementation (tests/plain/tagulix_plain.py): each mechanism alone, one key that stands
out just inside and just outside a window, at pages' borders, far back and at a sequence's first token, one token that only a carried state
can tell, then whole models through the step function and the cache manager in every cutting, then generation through the engine."""

from __future__ import annotations

import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

from tests import traces
from tests.plain import tagulix_plain as plain
from tests.tagulix_cases import CASES, assert_close_to_plain, attention, make_model_dir, model, movement, parallel, plain_logits, random_case, random_tokens

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent
DEV = "cuda:0"
F64 = torch.float64

LENGTHS = {"a": (70, 45, 128, 33, 2, 97), "b": (60, 9, 41, 3, 77, 50, 30), "c": (150, 66, 5, 90, 17, 2, 170, 64), "d": (90, 66, 5, 131, 40)}


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    return {name: make_model_dir(tmp_path_factory.mktemp(f"tg_{name}"), case) for name, case in CASES.items()}


def requests_for(name: str) -> dict[str, list[int]]:
    vocab = CASES[name]["config"]["vocab"]
    return {f"r{i}": random_tokens(300 + i, n, vocab) for i, n in enumerate(LENGTHS[name])}


def i32(values):
    return torch.tensor(values, dtype=torch.int32, device=DEV)


def close(got, want, tol, what=""):
    err = float((got.double().cpu() - want).abs().max())
    assert err <= tol * max(1.0, float(want.abs().max())), (what, err)


# ---------------------------------------------------------------------------------------------
# each mechanism alone


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("shape", [(1, 64), (2, 37), (3, 768), (4, 1600), (5, 42), (6, 3), (7, 2052), (8, 1024), (9, 100), (16, 33), (32, 264), (4, 9000), (2, 4100), (12, 1500)])
def test_streams_side_by_side(shape, dtype):
    """The join alone: every stream from the old ones, the next sublayer's input of the new ones, in place and from one row for all."""
    from research_2_b200.kernels import ops

    s, width = shape
    gen = torch.Generator().manual_seed(s * 10000 + width)
    rows, eps = 19, 1e-3
    x, y = torch.randn(rows, s, width, generator=gen), torch.randn(rows, width, generator=gen) * 3
    mix, join, read = torch.randn(s, s, generator=gen), torch.randn(s, generator=gen), torch.randn(s, generator=gen)
    gain = 1.0 + 0.3 * torch.randn(width, generator=gen)
    x[4], y[4] = 0.0, 0.0     # a row of zeros stays zero: eps stands inside the root
    weights = dict(mix=mix.to(DEV), join=join.to(DEV))
    tol = 1e-5 if dtype == torch.float32 else 8e-3

    def wanted(old):
        new = torch.einsum("ab,tad->tbd", mix.double(), old) + join.double()[None, :, None] * y.double()[:, None, :]
        return new, torch.einsum("a,tad->td", read.double(), new)

    new, u = wanted(x.double())
    dev = x.to(DEV)
    got, h = ops.stream_join(dev, read.to(DEV), gain.to(DEV), eps, dtype, y=y.to(DEV), **weights)
    assert got.data_ptr() == dev.data_ptr() and h.dtype == dtype
    close(got, new, 1e-5, shape)
    close(h, plain.rms_norm(u, gain, eps), tol, shape)
    assert float(h[4].abs().max()) == 0.0
    # one row that stands for every stream
    one = x[:, 0].contiguous()
    new, u = wanted(one.double()[:, None, :].repeat(1, s, 1))
    dev = one.to(DEV)
    got, h = ops.stream_join(dev, read.to(DEV), gain.to(DEV), eps, dtype, y=y.to(DEV), **weights)
    assert got.shape == (rows, s, width) and torch.equal(dev.cpu(), one)
    close(got, new, 1e-5, shape)
    close(h, plain.rms_norm(u, gain, eps), tol, shape)
    # the streams as they are: the first sublayer's input, and at the end the sum of the new ones alone
    same, h = ops.stream_join(dev, read.to(DEV), gain.to(DEV), eps, dtype)
    assert same is dev
    close(h, plain.rms_norm(read.double().sum() * one.double(), gain, eps), tol, shape)
    dev = x.to(DEV)
    _, h = ops.stream_join(dev, read.to(DEV), gain.to(DEV), eps, dtype)
    close(h, plain.rms_norm(torch.einsum("a,tad->td", read.double(), x.double()), gain, eps), tol, shape)
    none, total = ops.stream_join(dev, torch.ones(s, device=DEV), y=y.to(DEV), keep=False, **weights)
    assert none is None and total.dtype == torch.float32 and torch.equal(dev.cpu(), x)
    close(total, wanted(x.double())[0].sum(1), 1e-5, shape)


def test_what_streams_refuse():
    from research_2_b200.kernels import ops

    x, read = torch.zeros(2, 3, 8, device=DEV), torch.ones(3, device=DEV)
    for bad in (dict(read=torch.ones(2, device=DEV)), dict(gain=torch.ones(7, device=DEV)), dict(y=torch.zeros(2, 8, device=DEV), mix=torch.zeros(3, 2, device=DEV), join=read)):
        with pytest.raises(ops.KernelError):
            ops.stream_join(**{"x": x, "read": read, **bad})
    with pytest.raises(ops.KernelError):
        ops.stream_join(torch.zeros(2, 33, 8, device=DEV), torch.ones(33, device=DEV), torch.ones(8, device=DEV))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_router_with_corrections_and_identity_outputs(dtype):
    """Chosen by the corrected score inside the best groups, weighted by the score; the identity outputs' share of the row."""
    from research_2_b200.kernels import ops

    gen = torch.Generator().manual_seed(1)
    shapes = [  # rows, width, experts, identities, top, groups, kept groups, factor, size of the corrections, their offset
        (37, 40, 6, 2, 3, 4, 2, 1.5, 0.1, 0.0), (9, 64, 8, 0, 4, 4, 3, 1.0, 0.3, -5.0), (130, 96, 1, 2, 3, 1, 1, 0.5, 0.0, 0.0), (4, 200, 30, 3, 4, 11, 3, 2.5, 0.05, -0.2),
        (50, 24, 11, 1, 4, 2, 1, 1.0, 0.1, 0.0), (700, 132, 7, 3, 3, 2, 1, 1.5, 0.1, 0.0), (600, 50, 5, 3, 2, 1, 1, 0.8, 0.1, 0.0), (1030, 900, 61, 3, 6, 8, 3, 2.0, 0.01, -1.0), (21, 32, 1, 4, 2, 5, 3, 3.0, 0.2, -1.0), (64, 48, 40, 40, 8, 4, 4, 1.0, 0.02, 0.0), (17, 16, 1, 1, 1, 2, 1, 0.1, 0.1, 0.0),
    ]
    for rows, width, experts, identity, top, groups, keep, factor, spread, offset in shapes:
        n = experts + identity
        h = torch.randn(rows, width, generator=gen).to(dtype)
        w = (torch.randn(n, width, generator=gen) * 0.4).to(torch.bfloat16).float()
        correction = (torch.randn(n, generator=gen) * spread + offset).to(torch.bfloat16).float()
        base = torch.randn(rows, width, generator=gen)
        z = h.double() @ w.double().T
        for with_base in (False, True) if identity else (False,):
            dense, chosen, weight, gates, *carried = ops.route_scored(
                h.to(DEV), w.to(DEV), correction.to(DEV), top, groups, keep, scoring="softmax", group_mark="best", weight_scale=factor,
                n_identity=identity, base=base.to(DEV) if with_base else None)
            n_clear = 0
            for t in range(rows):
                want, gap = plain.route(z[t], correction.double(), top, groups, keep, factor)
                if gap < 1e-5:
                    continue
                n_clear += 1
                assert float((dense[t].double().cpu() - want).abs().max()) < 1e-5 * max(1.0, factor), (rows, t)
                assert sorted(chosen[t].cpu().tolist()) == torch.nonzero(want).flatten().tolist()
                assert abs(float(weight[t].sum()) - factor) < 1e-5 * max(1.0, factor)
                if identity:
                    share = want[experts:].sum() * h[t].double() + (base[t].double() if with_base else 0.0)
                    assert float((carried[0][t].double().cpu() - share).abs().max()) < 2e-5 * max(1.0, factor) * 5
            assert n_clear > rows // 2 and gates is None and len(carried) == int(identity > 0)
    # a row's weights are the same bits whatever the number of rows beside it (a warp a row, or a CTA a row)
    h, w = torch.randn(900, 260, generator=gen).to(dtype).to(DEV), torch.randn(12, 260, generator=gen).to(DEV) * 0.3
    whole = ops.route_scored(h, w, None, 4, 3, 2, scoring="softmax", group_mark="best", n_identity=2)
    for rows in (1, 40, 300):
        part = ops.route_scored(h[:rows].contiguous(), w, None, 4, 3, 2, scoring="softmax", group_mark="best", n_identity=2)
        assert all(torch.equal(a[:rows], b) for a, b in zip(whole, part) if a is not None), rows
    # choice scores may be negative: what is outside the kept groups counts as minus infinity, not as zero
    h = torch.zeros(2, 16, dtype=dtype, device=DEV)
    dense, chosen, _, _ = ops.route_scored(h, torch.zeros(6, 16, device=DEV), torch.tensor([-3.0, -2.0, -9.0, -4.0, -1.0, -5.0], device=DEV), 2, 3, 1,
                                           scoring="softmax", group_mark="best")
    assert [sorted(r) for r in chosen.cpu().tolist()] == [[4, 5]] * 2 and torch.allclose(dense[0, 4:].cpu(), torch.full((2,), 0.5))


@pytest.mark.parametrize("rows", [1, 7, 16, 33, 64, 65, 200, 1100])
def test_experts_without_gates(rows):
    """gelu (erf) of the stacked first product times the row's weight for the column's expert: inside the product's kernel for
    more than 64 rows and experts of 32 columns and more (whose borders lie anywhere in a tile), else in a kernel of its own."""
    from research_2_b200.kernels import ops

    gen = torch.Generator().manual_seed(rows)
    for experts, width, k, spare in ((4, 64, 96, 0), (3, 40, 72, 2), (5, 24, 64, 1), (2, 33, 50, 0), (7, 104, 128, 3), (3, 200, 64, 0), (16, 96, 192, 4)):
        route = torch.rand(rows, experts + spare, generator=gen) * 2
        route[torch.rand(route.shape, generator=gen) < 0.5] = 0.0
        a, w = torch.randn(rows, k, generator=gen), torch.randn(experts * width, k, generator=gen) * k ** -0.5 * 2
        for dtype, tol in ((torch.float32, 1e-5), (torch.bfloat16, 6e-3)):
            x, m = a.to(dtype), w.to(dtype)
            want = plain.gelu_erf(x.double() @ m.double().T) * route.double()[:, :experts].repeat_interleave(width, dim=1)
            launches = ops.launch_count()
            close(ops.routed_linear(x.to(DEV), m.to(DEV), "gelu", route.to(DEV), width), want, tol, (rows, experts, width, dtype))
            fused = dtype == torch.bfloat16 and width >= 32 and k % 8 == 0 and rows > 64
            assert ops.launch_count() == launches + (1 if fused else 2)
            close(ops.expert_unit((x @ m.T).to(DEV), "gelu", route.to(DEV), width), want, tol * 2, "the activation alone")
    old = ops.use_pair_gemm("always")
    try:
        route = torch.rand(300, 6, generator=gen)
        x, m = torch.randn(300, 128, generator=gen).to(torch.bfloat16), (torch.randn(6 * 72, 128, generator=gen) * 0.2).to(torch.bfloat16)
        want = plain.gelu_erf(x.double() @ m.double().T) * route.double().repeat_interleave(72, dim=1)
        close(ops.routed_linear(x.to(DEV), m.to(DEV), "gelu", route.to(DEV), 72), want, 6e-3, "pairs of CTAs")
    finally:
        ops.use_pair_gemm(old)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_the_whole_mixture(dtype):
    """Experts and identities, alone and onto a stream; also gated experts beside identities."""
    from research_2_b200.parts import Runtime
    from research_2_b200.parts.mlp import RoutedExperts

    gen = torch.Generator().manual_seed(3)
    rows, width, ff, experts, identity = 50, 48, 40, 5, 3
    r = {"experts": experts, "identity": identity, "top": 3, "groups": {"count": 2, "keep": 1}, "scale": 1.8}
    w = {"router": torch.randn(experts + identity, width, generator=gen) * 0.2, "correction": torch.randn(experts + identity, generator=gen) * 20}
    for e in range(experts):
        w[f"e{e}.up"], w[f"e{e}.down"] = torch.randn(ff, width, generator=gen) * 0.2, torch.randn(width, ff, generator=gen) * 0.2
    w = {n: t.to(torch.bfloat16) for n, t in w.items()}
    names = {"router": w["router"], "correction": w["correction"]}
    for e in range(experts):
        names.update({f"e{e}.w_up": w[f"e{e}.up"], f"e{e}.w_down": w[f"e{e}.down"]})
    params = {"n_experts": experts, "n_identity": identity, "top": 3, "scoring": "softmax", "n_groups": 2, "keep_groups": 1, "group_mark": "best",
              "route_scale": 1.8, "activation": "gelu", "gated": False}
    part = RoutedExperts(params, names, Runtime(torch.device(DEV), dtype))
    h, stream = torch.randn(rows, width, generator=gen).to(dtype), torch.randn(rows, width, generator=gen)
    want = plain.mixture(h.double(), w, "", {"router": r})
    tol = 2e-5 if dtype == torch.float32 else 1.5e-2
    close(part.mix(h.to(DEV), None), want, tol)
    close(part.forward(h.to(DEV), stream.to(DEV), None), want + stream.double(), tol)
    gates = {f"e{e}.w_gate": torch.randn(ff, width, generator=gen).to(torch.bfloat16) * 0.2 for e in range(experts)}
    part = RoutedExperts({**params, "activation": "silu", "gated": True}, {**names, **gates}, Runtime(torch.device(DEV), dtype))
    z = h.double() @ w["router"].double().T
    want = torch.zeros(rows, width, dtype=F64)
    for t in range(rows):
        weights, _ = plain.route(z[t], w["correction"].double(), 3, 2, 1, 1.8)
        want[t] = weights[experts:].sum() * h[t].double()
        for e in range(experts):
            inner = plain.silu(h[t].double() @ gates[f"e{e}.w_gate"].double().T) * (h[t].double() @ w[f"e{e}.up"].double().T)
            want[t] += weights[e] * (inner @ w[f"e{e}.down"].double().T)
    close(part.mix(h.to(DEV), None), want, tol, "gated")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("shape", [(4, 2, 16, 16, 8), (1, 1, 24, 8, 24), (6, 2, 64, 64, 64), (8, 1, 32, 12, 2), (3, 3, 7, 16, 6), (5, 1, 12, 12, 0), (2, 2, 130, 40, 64)])
def test_turned_then_normed_heads(dtype, shape):
    """Neighbouring pairs turn by the position, then every head is divided by its root mean square; the same launch puts keys and
    values into the cache."""
    from research_2_b200.kernels import ops

    heads, kv, dim, vdim, rot = shape
    gen = torch.Generator().manual_seed(sum(shape))
    page, n_pages, eps, base = 4, 20, 1e-3, 700.0
    positions = [0, 1, 2, 3, 17, 255, 1000, 4095, 9, 10, 11] + list(range(40, 70))
    rows = len(positions)
    width = (heads + kv) * dim + kv * vdim
    proj = (torch.randn(rows, width, generator=gen) * 2).to(dtype)
    proj[5, : (heads + kv) * dim] = 0.0
    qk = proj[:, : (heads + kv) * dim].double().view(rows, heads + kv, dim)
    want = plain.unit_rms(plain.rotate_pairs(qk, positions, rot, base) if rot else qk, eps).reshape(rows, -1)
    freqs = torch.tensor([base ** (-2.0 * i / max(rot, 1)) for i in range(rot // 2)], dtype=F64).float().to(DEV)
    ones = torch.ones(dim, device=DEV)
    how = dict(q_norm=ones, k_norm=ones, n_q_heads=heads, norm_eps=eps, interleaved=True)
    slots = (torch.randperm((n_pages - 1) * page, generator=gen)[:rows] + page).to(torch.int32).to(DEV)
    stride = kv * page * (dim + vdim)
    tol = 3e-4 if dtype == torch.float32 else 8e-3     # (float32: the angle of position 4,095 itself)
    results = []
    for cached in (False, True):
        dev = proj.to(DEV)
        pool = torch.full((n_pages * stride,), 7.0, dtype=dtype, device=DEV)
        scatter = ops.kv_scatter(slots, pool, pool[kv * page * dim:], stride, page, n_pages, (heads + kv) * dim, kv * vdim, vdim) if cached else None
        ops.rotate_half(dev, heads + kv, dim, rot, freqs, i32(positions), kv=scatter, n_kv_heads=kv, k_col=heads * dim, **how)
        close(dev[:, : (heads + kv) * dim], want, tol, shape)
        assert torch.equal(dev[:, (heads + kv) * dim:].cpu(), proj[:, (heads + kv) * dim:]), "values are not turned"
        results.append(dev)
        if cached:
            pages = pool.view(n_pages, stride)
            for t in range(rows):
                p, o = int(slots[t]) // page, int(slots[t]) % page
                k_at = pages[p, : kv * page * dim].view(kv, page, dim)[:, o].reshape(-1)
                v_at = pages[p, kv * page * dim:].view(kv, page, vdim)[:, o].reshape(-1)
                assert torch.equal(k_at, dev[t, heads * dim: (heads + kv) * dim]) and torch.equal(v_at, dev[t, (heads + kv) * dim:])
            assert float(pages[0].min()) == 7.0 == float(pages[0].max()), "the null page was written"
    assert torch.equal(*results)
    # rotation alone, without a norm
    if rot:
        dev = proj.to(DEV)
        ops.rotate_half(dev, heads + kv, dim, rot, freqs, i32(positions), interleaved=True)
        close(dev[:, : (heads + kv) * dim], plain.rotate_pairs(qk, positions, rot, base).reshape(rows, -1), 1e-3 if dtype == torch.float32 else 8e-3)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("dim", [7, 20, 24, 64, 80, 256, 514])
def test_head_norms_with_a_query_temperature(dim, dtype):
    """Positions just before, at and after the steps of the temperature; keys have none."""
    from research_2_b200.kernels import ops

    gen = torch.Generator().manual_seed(dim)
    heads, kv, eps = 3, 2, 1e-4
    for coef, every in ((0.5, 64), (-0.3, 1), (2.0, 7), (0.0, 5)):
        positions = [0, 1, 5, 6, 7, 62, 63, 64, 126, 127, 128, 4094, 4095, 100000, 12, 13]
        rows = len(positions)
        proj = (torch.randn(rows, (heads + 2 * kv) * dim, generator=gen) * 2).to(dtype)
        gq, gk = 1.0 + 0.3 * torch.randn(dim, generator=gen), 1.0 + 0.3 * torch.randn(dim, generator=gen)
        factor = torch.tensor([plain.query_temperature(p, coef, every) for p in positions], dtype=F64)[:, None, None]
        qk = proj[:, : (heads + kv) * dim].double().view(rows, heads + kv, dim)
        want = torch.cat([plain.rms_norm(qk[:, :heads], gq, eps) * factor, plain.rms_norm(qk[:, heads:], gk, eps)], dim=1).reshape(rows, -1)
        dev = proj.to(DEV)
        ops.head_norm(dev, heads, kv, dim, gq.to(DEV), gk.to(DEV), eps, temperature=(i32(positions), coef, every))
        close(dev[:, : (heads + kv) * dim], want, 3e-6 if dtype == torch.float32 else 8e-3, (dim, coef, every))
        assert torch.equal(dev[:, (heads + kv) * dim:].cpu(), proj[:, (heads + kv) * dim:])


ATTENTION_SHAPES = [(4, 2, 64, 16, 48), (3, 1, 80, 4, 33), (1, 1, 24, 8, 5), (8, 1, 128, 32, 100), (2, 2, 32, 64, 0), (6, 2, 64, 8, 1), (9, 1, 20, 8, 40)]


@pytest.mark.parametrize("cut", ["prompts", "decoded", "portions"])
@pytest.mark.parametrize("kind", ["window", "bias"])
@pytest.mark.parametrize("shape", ATTENTION_SHAPES)
def test_attention_kernels(shape, kind, cut):
    """A window and nothing else with exact weights; a bias by distance with sinks over every earlier key. Pages scattered in a pool full of
    large numbers; bfloat16 on the kernels that serve it and on the general one, float32 on the general one."""
    from research_2_b200.kernels import ops

    heads, kv, dim, page, window = shape
    window = window if kind == "window" else 0
    gen = torch.Generator().manual_seed(heads * 1000 + dim)
    lengths = [1, 2, 63, 64, 65, 130, 200, 101]
    scale, factor, reach = dim ** -0.5, (1.0 if kind == "window" else 0.7), 50
    k = [(torch.randn(n, kv, dim, generator=gen) * 1.5).to(torch.bfloat16) for n in lengths]
    v = [torch.randn(n, kv, dim, generator=gen).to(torch.bfloat16) for n in lengths]
    sinks, bias = torch.randn(heads, generator=gen) * 2, torch.randn(heads, reach, generator=gen) * 2
    width = max(-(-n // page) for n in lengths)
    n_pages = 1 + len(lengths) * width
    order = (torch.randperm(n_pages - 1, generator=gen) + 1).tolist()
    pool = torch.full((n_pages, 2, kv, page, dim), 300.0, dtype=torch.bfloat16)
    tables = torch.zeros(len(lengths), width, dtype=torch.int32)
    for e, n in enumerate(lengths):
        for b in range(-(-n // page)):
            tables[e, b] = order.pop()
            rows = min(page, n - b * page)
            pool[tables[e, b], 0, :, :rows] = k[e][b * page: b * page + rows].transpose(0, 1)
            pool[tables[e, b], 1, :, :rows] = v[e][b * page: b * page + rows].transpose(0, 1)
    spans = {"prompts": [(0, n) for n in lengths], "decoded": [(n - 1, n) for n in lengths], "portions": [(n // 3, n - n // 4) for n in lengths]}[cut]
    entry_rows = [b - a for a, b in spans]
    q_start = [sum(entry_rows[:i]) for i in range(len(lengths) + 1)]
    positions = [p for a, b in spans for p in range(a, b)]
    row_entry = [e for e, (a, b) in enumerate(spans) for _ in range(a, b)]
    q = (torch.randn(len(positions), heads * dim, generator=gen) * 1.5).to(torch.bfloat16)
    full_bias = torch.cat([bias, bias[:, -1:].expand(heads, 200)], dim=1).double()
    how = dict(window=window) if kind == "window" else dict(bias=full_bias, sink=sinks.double())
    want = torch.cat([plain.attend(q[q_start[e]: q_start[e + 1]].double().view(-1, heads, dim), k[e].double(), v[e].double(), scale, positions=list(range(*spans[e])), **how)
                      for e in range(len(lengths))]).reshape(len(positions), -1) * factor
    extras = {} if kind == "window" else dict(dist_bias=bias.to(DEV), sinks=sinks.to(DEV), out_scale=factor)
    where = (i32(row_entry), i32(positions), i32([b for _, b in spans]), heads, kv, dim, scale)

    def paged(dtype):
        flat = pool.to(dtype).to(DEV).view(-1)
        return ops.paged_attention(q.to(dtype).to(DEV), flat, flat[kv * page * dim:], 2 * kv * page * dim, page, n_pages, tables.to(DEV), *where, window,
                                   decode_only=cut == "decoded", max_context=max(lengths), q_start=i32(q_start), n_tiles=sum(-(-r // 64) for r in entry_rows),
                                   exact=True, **extras)

    before = dict(ops.kernel_uses())
    close(paged(torch.bfloat16), want, 1.2e-2, f"{shape} {cut}")
    used = [name for name, n in ops.kernel_uses().items() if n > before.get(name, 0)]
    fast = dim % 16 == 0 and dim <= 128
    assert used == (["attention_prefill_tc"] if fast and kind == "window" and dim == 64 else ["attention_prefill"] if fast else ["attention_simt"]), used
    close(paged(torch.float32), want, 2e-5, f"{shape} {cut} float32")
    if cut != "decoded" or dim % 16 or heads // kv > 8:
        return
    # the decode kernel takes the newest key and value from the projection and puts them into the cache itself
    flat = pool.clone().to(DEV).view(-1)
    slot = [int(tables[e, (b - 1) // page]) * page + (b - 1) % page for e, (_, b) in enumerate(spans)]
    cells = flat.view(n_pages, 2, kv, page, dim)
    for s in slot:
        cells[s // page, :, :, s % page] = 55.0
    new = torch.stack([torch.cat([k[e][b - 1].reshape(-1), v[e][b - 1].reshape(-1)]) for e, (_, b) in enumerate(spans)]).to(DEV)
    got = ops.decode_attention_fused(q.to(DEV), new[:, : kv * dim], new[:, kv * dim:], i32(slot), flat, flat[kv * page * dim:], 2 * kv * page * dim, page, n_pages,
                                     tables.to(DEV), *where, window, max(lengths), exact_weights=True, **extras)
    close(got, want, 1.2e-2, f"{shape} fused")
    assert torch.equal(flat.view(-1).cpu(), pool.view(-1)), "the new keys and values are in their places and nothing else changed"


DECAY_SHAPES = [((0.9, 0.99), 256, 72), ((0.97,), 256, 64), ((0.8, -0.5), 17, 70), ((0.5, 0.97), 16, 24), ((0.0, 1.0, 0.8), 5, 7), ((0.9,), 33, 12), ((0.99, 0.3), 64, 64), ((0.999, 0.6, 0.9, 0.2), 32, 64), ((1.0,), 128, 96), ((0.95, 0.5), 100, 40),
                ((0.7,), 200, 8), ((0.6065, 0.999), 96, 128), ((0.999, 1e-3), 64, 30)]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("shape", DECAY_SHAPES)
def test_decay_attention_alone(shape, dtype):
    """silu and the recurrence over sequences in portions of 1 to 150 rows, beside one another in one batch, in slots that others held
    before. In float32 the results do not depend on the cutting, to the bit; in bfloat16 batches of 64 rows and more run in chunks, the
    others row by row."""
    from research_2_b200.kernels import ops

    decay, dim, vdim = shape
    heads = len(decay)
    gen = torch.Generator().manual_seed(dim * 100 + vdim)
    n_qk, n_v = heads * dim, heads * vdim
    lengths = (150, 9, 70)
    seqs = [torch.randn(n, 2 * n_qk + n_v + 3, generator=gen).to(dtype) for n in lengths]     # (three more columns: rows start anywhere)
    rates = torch.tensor(decay, dtype=F64)
    want = []
    for x in seqs:
        q, k, v = (plain.silu(c.double()).reshape(x.shape[0], heads, -1) for c in (x[:, :n_qk], x[:, n_qk: 2 * n_qk], x[:, 2 * n_qk: 2 * n_qk + n_v]))
        want.append(plain.decay_core(q, k, v, rates)[0].reshape(x.shape[0], -1))
    floats = heads * dim * vdim

    def run(cuts, slots, spare=0):
        """cuts: per step, the (sequence, rows) of its entries; spare: chunks that the launch allows for and no entry has."""
        state = torch.full((5, floats), 1e4, device=DEV)     # what other requests left there
        at, outs = [0] * len(seqs), [[] for _ in seqs]
        for step in cuts:
            starts = [sum(n for _, n in step[:i]) for i in range(len(step) + 1)]
            x = torch.cat([seqs[s][at[s]: at[s] + n] for s, n in step]).to(DEV)
            positions = i32([at[s] + i for s, n in step for i in range(n)])
            o = ops.retention_scan(x[:, :n_qk], x[:, n_qk: 2 * n_qk], x[:, 2 * n_qk: 2 * n_qk + n_v], rates.float().to(DEV), 1.0, None, 0, positions, state,
                                   i32(starts), i32([slots[s] for s, _ in step]), i32([int(at[s] == 0) for s, _ in step]), heads, dim, vdim, silu=True,
                                   n_tiles=sum(-(-n // 64) for _, n in step) + spare).cpu()
            for i, (s, n) in enumerate(step):
                outs[s].append(o[starts[i]: starts[i + 1]])
                at[s] += n
        assert at == list(lengths) and float(state[[i for i in range(5) if i not in slots]].min()) == 1e4, "a slot of no entry changed"
        return [torch.cat(o) for o in outs]

    used = ops.kernel_uses().get("decay_chunks", 0)
    whole = run([[(0, 150), (1, 9), (2, 70)]], (3, 0, 2))
    assert ops.kernel_uses().get("decay_chunks", 0) - used == int(dtype == torch.bfloat16)
    portions = run([[(0, 2), (2, 33)], [(0, 1), (1, 1), (2, 1)], [(0, 1), (1, 1), (2, 1)], [(2, 35), (0, 100)], [(1, 7), (0, 46)]], (1, 4, 0), spare=3)
    single = run([[(0, 1), (1, 1), (2, 1)]] * 9 + [[(0, 1), (2, 1)]] * 61 + [[(0, 1)]] * 80, (0, 1, 2))
    for s in range(3):
        for what, got in (("whole", whole), ("portions", portions), ("single", single)):
            close(got[s], want[s], 2e-5 if dtype == torch.float32 or what == "single" else 5e-5, f"{shape} {dtype} sequence {s} {what}")
        if dtype == torch.float32:
            assert torch.equal(portions[s], whole[s]) and torch.equal(single[s], whole[s]), f"{shape}: sequence {s} depends on its cutting"


def test_decay_chunks_of_many_entries_beside_the_walk():
    """Eighty entries, some without rows, some of one row: the two ways give the same outputs and states, and touch no slot of an
    entry without rows."""
    from research_2_b200.kernels import ops

    gen = torch.Generator().manual_seed(6)
    heads, dim, vdim = 3, 48, 40
    lengths = [(0, 1, 63, 64, 65, 7, 130, 1)[i % 8] for i in range(80)]
    starts = [sum(lengths[:i]) for i in range(81)]
    x = torch.randn(starts[-1], heads * (2 * dim + vdim), generator=gen).to(torch.bfloat16).to(DEV)
    q, k, v = x.split([heads * dim, heads * dim, heads * vdim], dim=1)
    slots, fresh = torch.randperm(90, generator=gen)[:80].to(torch.int32), torch.randint(0, 2, (80,), generator=gen).to(torch.int32)
    first = torch.randn(90, heads * dim * vdim, generator=gen)
    decay = torch.tensor([0.9, 0.999, 0.2], device=DEV)
    results = []
    for chunks in (True, False):
        state = first.to(DEV).clone()
        old = ops.use_decay_chunks(chunks)
        try:
            out = ops.retention_scan(q, k, v, decay, 0.5, None, 0, i32([0] * starts[-1]), state, i32(starts), slots.to(DEV), fresh.to(DEV), heads, dim, vdim,
                                     silu=True, n_tiles=sum(-(-n // 64) for n in lengths))
        finally:
            ops.use_decay_chunks(old)
        results.append((out, state))
    for a, b in zip(*results):
        close(a, b.double().cpu(), 5e-5)
    idle = [i for i in range(90) if i not in set(slots.tolist()) or lengths[slots.tolist().index(i)] == 0]
    assert len(idle) == 20 and torch.equal(results[0][1][idle].cpu(), first[idle])

# ---------------------------------------------------------------------------------------------
# one key that stands out: in the window and out of it, at pages' borders, at the first token, far back in a cache and in a carried state


QUERY_TOKEN, KEY_TOKEN = 1, 2


def planted_model(folder: Path, kind: str, window: int = 0) -> Path:
    """One layer whose weights are made so that the token QUERY_TOKEN asks for exactly what the token KEY_TOKEN left: coordinate 0 of the
    stream drives head 0's query, coordinate 1 its key, along one direction that no rotation turns; every other token has coordinate 2,
    whose key lies across it. In attention the key's score is 40 above the others' wherever it is visible; in the recurrence nothing decays
    and no other token writes along that direction. What the other mixer of a pair makes is left out (its output matrix is zero)."""
    from research_2_b200 import models  # noqa: F401  (registers the architectures)
    from research_2_b200.config.registry import architecture_of
    from research_2_b200.weights.safetensors_io import write_file

    width, dim = 36, 16
    heads, kv = 4, 2
    one = attention(heads, kv, dim, dim, 2.5, window, (8, 400.0)) if kind == "window" else \
        parallel((heads, kv, dim, dim, 2.5, 30), ((1.0, 0.9), dim, 24), (1.5, 1.5), (0.1, 50))
    config = model(64, width, [one], eps=1e-5, streams=2, mult=4.0)
    arch = architecture_of(config)
    w = arch.random_weights(arch.parse_config(config), 17, std=0.08, bias_rows=8)
    gen = torch.Generator().manual_seed(18)
    w["embed"][:, :3] = 0.0
    w["embed"][:, 2] = 3.0
    for token, coordinate in ((QUERY_TOKEN, 0), (KEY_TOKEN, 1)):
        w["embed"][token, 2] = 0.0
        w["embed"][token, coordinate] = 6.0
    direction, across = torch.zeros(dim), torch.zeros(dim)
    direction[8:12], across[12:] = torch.randn(4, generator=gen).abs() + 0.5, torch.randn(4, generator=gen).abs() + 0.5
    p = "l0.mix."
    if kind == "state":
        for name, coordinate in (("q", 0), ("k", 1)):
            w[p + "right." + name][:dim] = 0.0
            w[p + "right." + name][:dim, coordinate] = direction
        w[p + "right.v"] *= 4.0
        w[p + "left.o"] *= 0.0
    else:
        prefix = p if kind == "window" else p + "left."
        for name, along in (("q", {0: direction}), ("k", {1: direction, 2: across, 0: across})):
            w[prefix + name][:dim] = 0.0
            for coordinate, vector in along.items():
                w[prefix + name][:dim, coordinate] = vector
            if kind == "window":
                w[prefix + name + ".b"][:dim] = 0.0
            else:
                w[prefix + name + ".norm"] = torch.ones(dim)
        if kind != "window":
            w[p + "right.o"] *= 0.0
    w["l0.norm1"] = torch.ones(width)
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(arch.config_to_json(arch.parse_config(config))))
    write_file(folder / "model.safetensors", {n: t.to(torch.bfloat16) for n, t in w.items()})
    return folder


def planted_sequence(n: int, ask_at: int, distance: int, seed: int = 0) -> list[int]:
    ids = [3 + t for t in random_tokens(seed, n, 61)]
    ids[ask_at] = QUERY_TOKEN
    if 0 <= ask_at - distance < ask_at:
        ids[ask_at - distance] = KEY_TOKEN
    return ids


# asking row, distance of the key (windows of 40 in pages of 16; borders of pages, of the prefill kernels' tiles of 64, the first token)
WINDOW_CASES = [(119, 39), (119, 40), (120, 38), (121, 1), (39, 39), (40, 40), (41, 40), (40, 39), (143, 15), (144, 16), (144, 24), (143, 39), (143, 40), (700, 39), (700, 40),
                (701, 41), (64, 39), (64, 40), (128, 39), (127, 40), (1, 1)]
OPEN_CASES = [(650, 600), (229, 229), (229, 1), (130, 2), (130, 3), (130, 30), (130, 31), (144, 16), (77, 77), (300, 172), (1, 1), (511, 448)]
STATE_CASES = [(650, 600), (229, 229), (77, 1), (130, 127), (66, 64), (128, 64), (127, 63), (1, 1)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("how", ["prompt", "decoded", "portion_between"])
@pytest.mark.parametrize("kind", ["window", "open", "state"])
def test_one_key_that_stands_out(tmp_path, dtype, how, kind):
    """The asking row in a prompt, decoded alone, or first in a portion that begins between the key and the row. Inside the window the
    logits are those with the key, outside those of a sequence without it."""
    cases = {"window": WINDOW_CASES, "open": OPEN_CASES}.get(kind, STATE_CASES)
    folder = planted_model(tmp_path / kind, kind, 40 if kind == "window" else 0)
    for ask_at, distance in cases:
        ids = planted_sequence(ask_at + 6, ask_at, distance, seed=ask_at)
        truth = plain_logits(folder, ids)[ask_at]
        without = plain_logits(folder, planted_sequence(ask_at + 6, ask_at, 0, seed=ask_at))[ask_at]
        gap, size = float(np.abs(truth - without).max()), float(np.abs(truth).max())
        if kind == "window" and distance >= 40:
            assert gap < 1e-9, (kind, ask_at, distance, gap)
        else:
            assert gap > 0.2 * size, (kind, ask_at, distance, gap, size)
        tb, n = traces.TraceBuilder(), len(ids)
        if how == "prompt":
            tb.step([("x", ids, list(range(n)))], end=["x"])
        elif how == "decoded":
            first = max(1, ask_at - 3)
            tb.step([("x", ids[:first], list(range(first)))])
            for t in range(first, n):
                tb.step([("x", ids[t: t + 1], [0])], end=["x"] if t == n - 1 else [])
        else:
            cut_at = max(1, ask_at - max(1, distance // 2))
            tb.step([("x", ids[:cut_at], list(range(cut_at)))])
            tb.step([("x", ids[cut_at: ask_at + 2], list(range(ask_at + 2 - cut_at)))])
            tb.step([("x", ids[ask_at + 2:], list(range(n - ask_at - 2)))], end=["x"])
        outputs, _, _ = run_trace(folder, tb, dtype, 16)
        got = compare(folder, {"x": ids}, tb, outputs, dtype, f"{kind} {how} row {ask_at} distance {distance}")["x"][ask_at]
        assert float(np.abs(got - truth).max()) < 0.1 * size, f"{kind} {how} row {ask_at} distance {distance}"


# ---------------------------------------------------------------------------------------------
# whole models in every cutting


def cut(requests, mode: str) -> traces.TraceBuilder:
    if mode == "whole":
        return traces.whole(requests)
    if mode == "decode":
        return traces.prefill_then_decode(requests, 48)
    if mode == "portions":
        return traces.portions(requests)
    if mode == "tiny_portions":
        return traces.portions(requests, sizes=(2, 3, 2, 5, 2, 2, 9))
    return traces.mixed(requests, max_live=4)


def run_trace(folder, tb, dtype, page_size, max_tokens=None, max_seq_len=0):
    """Replays the trace in a pool of the trace's own peak demand plus one page (or `max_tokens`), the cache and the state slots
    filled with loud values first. -> ({step: logits}, how many pages had two owners or more, the replay)."""
    from research_2_b200.engine.replay import Replay

    live, round_to = traces.max_live(tb), 64
    if max_tokens is None:
        max_tokens, round_to = (traces.peak_pages(tb, page_size) + 1) * page_size, page_size
    replay = Replay(str(folder), dtype, max_tokens, block_size=page_size, max_live=max(live, 1), round_to=round_to, max_seq_len=max_seq_len)
    replay.step_fn.arena.fill_(64.0)
    for t in replay.step_fn.state_tensors:
        t.fill_(50.0)
    owners: dict[tuple[int, int], set] = {}
    out = {}
    for record in tb.steps:
        logits = replay.step(record)
        if logits is not None:
            out[record["step"]] = logits
        for rid, per_group in replay.pages_of_last_step.items():
            for g, pages in enumerate(per_group):
                for page in pages:
                    owners.setdefault((g, page), set()).add(rid)
    assert replay.cache.check() == ""
    for g in range(len(replay.cache.groups)):
        assert replay.cache.n_free(g) == replay.cache.groups[g].num_pages, "pages were lost"
    return out, sum(len(v) >= 2 for v in owners.values()), replay


def compare(folder, requests, tb, outputs, dtype, what):
    assert sorted(outputs) == sorted(tb.rows)
    per_request: dict[str, dict[int, np.ndarray]] = {}
    for step, rows in tb.rows.items():
        for (rid, pos), logits in zip(rows, outputs[step]):
            assert pos not in per_request.setdefault(rid, {}), f"{what}: position {pos} of {rid} written twice"
            per_request[rid][pos] = logits
    for rid, ids in requests.items():
        assert sorted(per_request[rid]) == list(range(len(ids))), f"{what}: request {rid} misses positions"
        got = np.stack([per_request[rid][p] for p in range(len(ids))])
        assert_close_to_plain(got, folder, ids, dtype, what=f"{what} request {rid}")
    return per_request


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["a", "b", "c", "d"])
@pytest.mark.parametrize("mode", ["whole", "decode", "portions", "tiny_portions", "mixed"])
def test_cuttings(folders, name, dtype, mode):
    folder, requests = folders[name], requests_for(name)
    if mode == "tiny_portions":
        requests = dict(list(requests.items())[:3])
    tb = cut(requests, mode)
    outputs, reused, replay = run_trace(folder, tb, dtype, CASES[name]["page_size"])
    compare(folder, requests, tb, outputs, dtype, f"{name}/{dtype}/{mode}")
    windows = {layer["mixer"].get("mask", {}).get("size", 0) for layer in CASES[name]["config"]["layers"]}
    assert {g.window for g in replay.cache.groups} == windows, "one cache group per window"
    assert dtype == "float32" or name == "b" or all(np.isfinite(movement(str(folder), tuple(ids))).all() for ids in list(requests.values())[:2]), "no position is excused"
    if mode == "mixed":
        assert traces.max_live(tb) == 4 and len(requests) > 4, "request and state slots are used again"
        assert reused >= 2, f"only {reused} pages passed from one request to another"


def test_the_stream_after_every_layer(folders):
    """The sum of the streams after each layer (not only the logits), in float32: a layer that is wrong and then drowned by the next norm
    shows here."""
    from research_2_b200.engine.replay import Replay

    for name in ("a", "b", "c", "d"):
        folder = folders[name]
        ids = random_tokens(9, 50, CASES[name]["config"]["vocab"])
        cfg, w = plain.read_model(folder)
        want: list = []
        plain.forward(cfg, w, ids, layers_out=want)
        replay = Replay(str(folder), "float32", 64, block_size=CASES[name]["page_size"], max_live=1)
        got = []
        for b in replay.model.blocks:
            def tapped(*args, _original=b.forward, **kwargs):
                x = _original(*args, **kwargs)
                got.append((x.sum(1) if x.dim() == 3 else x).detach().double().cpu().clone())
                return x
            b.forward = tapped
        replay.step({"step": 0, "entries": [{"id": "x", "tokens": ids, "want": [len(ids) - 1]}], "end": ["x"]})
        assert len(got) == len(want)
        for i, (a, b) in enumerate(zip(got, want)):
            assert float((a[: len(ids)] - b).abs().max()) <= 3e-5 * float(b.abs().max()), (name, i)


def test_sequences_longer_than_their_pool(tmp_path):
    """Where every layer has a window, a sequence needs the pages of its window alone: 300 tokens in a pool of 96."""
    case = {"config": model(61, 48, [attention(2, 1, 16, 16, 0.3, 20, (8, 100.0)), attention(4, 2, 8, 12, 0.3, 32), attention(2, 1, 16, 16, 0.3, 20, (8, 100.0), weights_of=0)],
                            streams=2, mult=1.5), "seed": 4, "std": 0.08, "bias_rows": 8, "correction_std": 1.0}
    folder = make_model_dir(tmp_path / "model", case)
    ids = random_tokens(2, 300, 61)
    for dtype in ("float32", "bfloat16"):
        tb = traces.portions({"x": ids}, sizes=(30, 1, 17, 2, 1, 1, 24))
        outputs, _, replay = run_trace(folder, tb, dtype, 8, max_tokens=96, max_seq_len=320)
        compare(folder, {"x": ids}, tb, outputs, dtype, f"short pool {dtype}")
        assert all(g.num_pages * 8 < 200 for g in replay.cache.groups)


def test_which_kernels_serve_bfloat16(folders):
    """Case d has the shapes that the fast kernels are written for: its windows run on the tcgen05 kernel (heads of 64) or the mma.sync
    one, its biased attention on the mma.sync one, all decode steps on the fused decode kernel, which writes the new key itself."""
    from research_2_b200.kernels import ops

    folder, name = folders["d"], "d"
    ids = random_tokens(3, 150, CASES[name]["config"]["vocab"])
    tb = traces.prefill_then_decode({"x": ids}, n_decode=4)
    before = dict(ops.kernel_uses())
    outputs, _, _ = run_trace(folder, tb, "bfloat16", CASES[name]["page_size"])
    compare(folder, {"x": ids}, tb, outputs, "bfloat16", "kernels of case d")
    used = {k: v - before.get(k, 0) for k, v in ops.kernel_uses().items()}
    assert used.get("attention_decode_fused", 0) == 20 and used.get("attention_prefill", 0) == 3 and used.get("attention_prefill_tc", 0) == 2, used
    assert used.get("attention_simt", 0) == 0, used


@pytest.mark.parametrize("seed", range(100, 112))
def test_configurations_drawn_at_random(seed, tmp_path):
    """Layers in any order and sizes of any kind: float32 within its floor in three cuttings, bfloat16 within its own (a router's
    close calls excused)."""
    case = random_case(seed)
    folder = make_model_dir(tmp_path / "model", case)
    ids = random_tokens(seed, case["length"], case["config"]["vocab"])
    requests = {"x": ids, "y": ids[: max(3, len(ids) // 3)], "z": ids[5:]}
    for dtype, modes in (("float32", ("whole", "portions", "mixed")), ("bfloat16", ("mixed",))):
        for mode in modes:
            tb = cut(requests, mode) if mode != "mixed" else traces.mixed(requests, max_live=2)
            outputs, _, _ = run_trace(folder, tb, dtype, case["page_size"])
            compare(folder, requests, tb, outputs, dtype, f"seed {seed} {dtype} {mode}")


def test_float32_logits_do_not_depend_on_the_cutting_at_all(folders):
    for name in ("a", "b", "c"):
        folder, requests = folders[name], requests_for(name)
        results = {}
        for mode in ("whole", "decode", "portions", "mixed"):
            tb = cut(requests, mode)
            results[mode] = compare(folder, requests, tb, run_trace(folder, tb, "float32", CASES[name]["page_size"])[0], "float32", f"{name}/{mode}")
        for mode in ("decode", "portions", "mixed"):
            for rid, rows in results["whole"].items():
                for pos, logits in rows.items():
                    assert np.array_equal(logits, results[mode][rid][pos]), f"{name}: {mode} differs from whole at {rid}[{pos}]"


def test_batches_against_each_request_alone_in_bfloat16(folders):
    """What else is in the batch moves a request's logits by no more than rounding does."""
    for name in ("a", "d"):
        folder, requests = folders[name], requests_for(name)
        tb = cut(requests, "mixed")
        together = compare(folder, requests, tb, run_trace(folder, tb, "bfloat16", CASES[name]["page_size"])[0], "bfloat16", f"{name} together")
        for rid, ids in list(requests.items())[:3]:
            tb = traces.portions({rid: ids})
            alone = compare(folder, {rid: ids}, tb, run_trace(folder, tb, "bfloat16", CASES[name]["page_size"])[0], "bfloat16", f"{name} {rid} alone")
            a, b = (np.stack([x[rid][p] for p in range(len(ids))]) for x in (together, alone))
            assert float(np.abs(a - b).max()) <= 6e-2 * float(np.abs(b).max()), (name, rid)


def test_long_decoding(folders):
    """400 tokens, 390 of them decoded one by one: through many windows, with states carried all the way."""
    for name in ("a", "d"):
        folder, page = folders[name], CASES[name]["page_size"]
        ids = random_tokens(21, 400, CASES[name]["config"]["vocab"])
        tb = traces.prefill_then_decode({"x": ids}, n_decode=390)
        for dtype in ("float32", "bfloat16"):
            outputs, _, _ = run_trace(folder, tb, dtype, page, max_tokens=448)
            compare(folder, {"x": ids}, tb, outputs, dtype, f"long decoding {name} {dtype}")


def test_first_tokens(folders):
    for name in ("a", "b", "c", "d"):
        folder = folders[name]
        ids = random_tokens(7, 5, CASES[name]["config"]["vocab"])
        tb = traces.TraceBuilder()
        tb.step([("x", ids[:1], [0])])
        tb.step([("x", ids[1:2], [0])])
        tb.step([("x", ids[2:4], [0, 1])])
        tb.step([("x", ids[4:5], [0])], end=["x"])
        for dtype in ("float32", "bfloat16"):
            compare(folder, {"x": ids}, tb, run_trace(folder, tb, dtype, CASES[name]["page_size"], max_tokens=64)[0], dtype, f"first tokens {name} {dtype}")


def test_trace_run_program(folders, tmp_path):
    folder, name = folders["a"], "a"
    requests = {k: v for k, v in list(requests_for(name).items())[:3]}
    tb = traces.mixed(requests, max_live=3)
    out = tmp_path / "out"
    text = "".join(json.dumps(s) + "\n" for s in tb.steps)
    proc = subprocess.run(
        [sys.executable, str(ROOT / "bin" / "trace_run"), "--model", str(folder), "--dtype", "bfloat16",
         "--out", str(out), "--max-tokens", str(sum(-(-len(v) // 64) * 64 for v in requests.values()))],
        input=text, capture_output=True, text=True, timeout=900)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [line for line in proc.stdout.splitlines() if line.startswith("done ")] == [f"done {i}" for i in range(len(tb.steps))]
    vocab = CASES[name]["config"]["vocab"]
    outputs = {int(p.stem): np.fromfile(p, dtype="<f4").reshape(-1, vocab) for p in out.glob("*.f32")}
    compare(folder, requests, tb, outputs, "bfloat16", "trace_run program")


# ---------------------------------------------------------------------------------------------
# generation through the entry point and the scheduler


def test_greedy_generation_through_the_engine(folders):
    """Prompts of unequal length through `generate` (scheduler, portions under a small token budget, CUDA graphs): float32
    tokens equal the plain implementation's; bfloat16 tokens are (nearly) the best by the plain logits of the sequence so
    far."""
    import research_2_b200

    for name in ("a", "d"):
        folder, vocab = folders[name], CASES[name]["config"]["vocab"]
        prompts = [random_tokens(40 + i, n, vocab) for i, n in enumerate((5, 61, 18, 33))]
        cfg, w = plain.read_model(folder)
        want = [plain.generate(cfg, w, p, 10) for p in prompts]
        got = research_2_b200.generate(folder, prompts, max_new_tokens=10, dtype="float32", device=DEV, block_size=8,
                                       max_batch_tokens=32, max_requests=3, max_seq_len=128)
        assert got == want, (name, got, want)
        got16 = research_2_b200.generate(folder, prompts, max_new_tokens=10, dtype="bfloat16", device=DEV, block_size=16,
                                         max_batch_tokens=48, max_requests=4, max_seq_len=128)
        for prompt, tokens in zip(prompts, got16):
            assert len(tokens) == 10
            logits = plain_logits(folder, (prompt + tokens)[:-1])
            slack = 2 * 3e-2 * float(np.abs(logits).max())
            near_best = [float(logits[len(prompt) - 1 + i][tok]) >= float(logits[len(prompt) - 1 + i].max()) - slack
                         for i, tok in enumerate(tokens)]
            assert all(0 <= tok < vocab for tok in tokens) and sum(near_best) >= 8, (name, tokens, near_best)


def test_generation_in_a_pool_that_forces_preemption(folders):
    """A preempted request is computed again from its first token, in pages and a state slot that others held meanwhile."""
    import research_2_b200

    name = "b"
    folder, vocab = folders[name], CASES[name]["config"]["vocab"]
    prompts = [random_tokens(60 + i, n, vocab) for i, n in enumerate((30, 44, 25))]
    cfg, w = plain.read_model(folder)
    want = [plain.generate(cfg, w, p, 10) for p in prompts]
    got = research_2_b200.generate(folder, prompts, max_new_tokens=10, dtype="float32", device=DEV, block_size=4,
                                   max_batch_tokens=16, max_requests=3, max_seq_len=64, num_slabs=30)
    assert got == want, (got, want)


def test_command_line(folders):
    folder = folders["b"]
    proc = subprocess.run([sys.executable, "-m", "research_2_b200", "generate", "--model", str(folder), "--prompt-tokens", "5,17,3",
                           "--max-new-tokens", "4", "--dtype", "float32", "--max-seq-len", "64"],
                          capture_output=True, text=True, timeout=900, cwd=str(ROOT))
    assert proc.returncode == 0, proc.stderr[-2000:]
    tokens = json.loads(proc.stdout.strip().splitlines()[-1])["tokens"]
    cfg, w = plain.read_model(folder)
    assert tokens == plain.generate(cfg, w, [5, 17, 3], 4)
