"""Lagelorn on the GPU against the plain implementation (tests/plain/lagelorn_plain.py): each mechanism alone, one key that
stands out just inside and just outside a chunk, at pages' borders and at a sequence's first token, one token that only a carried
state can tell, then whole models through the step function and the cache manager in every cutting, then generation through
the engine."""

from __future__ import annotations

import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

from tests import traces
from tests.lagelorn_cases import CASES, assert_close_to_plain, delta, make_model_dir, model, parallel, plain_logits, random_case, random_tokens
from tests.plain import lagelorn_plain as plain

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent
DEV = "cuda:0"
F64 = torch.float64

LENGTHS = {"a": (70, 45, 128, 33, 2, 97), "b": (60, 9, 41, 3, 77, 50, 30), "c": (150, 66, 5, 90, 17, 2, 170, 64), "d": (90, 66, 5, 131, 40)}


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    return {name: make_model_dir(tmp_path_factory.mktemp(f"lg_{name}"), case) for name, case in CASES.items()}


def requests_for(name: str) -> dict[str, list[int]]:
    vocab = CASES[name]["config"]["vocab"]
    return {f"r{i}": random_tokens(300 + i, n, vocab) for i, n in enumerate(LENGTHS[name])}


def i32(values):
    return torch.tensor(values, dtype=torch.int32, device=DEV)


def close(got, want, tol, what=""):
    err = float((got.double().cpu() - want).abs().max())
    assert err <= tol * max(1.0, float(want.abs().max())), (what, err)


class Entries:
    """A batch of entries of `lengths` rows over state slots: the arrays that the kernels read."""

    def __init__(self, lengths, slots, fresh):
        self.starts = [sum(lengths[:i]) for i in range(len(lengths) + 1)]
        self.rows = self.starts[-1]
        self.arrays = (i32(self.starts), i32(slots), i32([int(f) for f in fresh]))
        self.row_entry = i32([e for e, n in enumerate(lengths) for _ in range(n)])

    def of(self, e):
        return slice(self.starts[e], self.starts[e + 1])


# ---------------------------------------------------------------------------------------------
# each mechanism alone


DELTA_SHAPES = [(4, 2, 16, 24, 4), (3, 1, 10, 6, 1), (1, 1, 7, 33, 7), (2, 2, 64, 64, 4), (6, 3, 33, 12, 2), (2, 1, 128, 40, 3), (1, 1, 130, 16, 4), (2, 1, 300, 8, 2),
                (1, 1, 600, 5, 3), (5, 5, 3, 100, 5)]


def delta_reference(raw, h, taps, w_gates, step_bias, log_rate, heads, groups, dim, vdim):
    """The mechanism for one sequence, from the projections on (raw [T, channels], h [T, D], float64)."""
    T, per = raw.shape[0], heads // groups
    y = plain.short_conv(raw, taps)
    q = plain.unit(y[:, : groups * dim].view(T, groups, dim)) * dim ** -0.5
    k = plain.unit(y[:, groups * dim: 2 * groups * dim].view(T, groups, dim))
    v = y[:, 2 * groups * dim:].view(T, heads, vdim)
    gates = h @ w_gates.double().T
    g = torch.exp(-torch.exp(log_rate.double()) * torch.nn.functional.softplus(gates[:, heads:] + step_bias.double()))
    return plain.delta_core(q.repeat_interleave(per, dim=1), k.repeat_interleave(per, dim=1), v, g, torch.sigmoid(gates[:, :heads]))[0].reshape(T, -1)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("shape", DELTA_SHAPES)
def test_the_delta_rule_alone(shape, dtype):
    """Convolutions, unit vectors, decays, strengths and the recurrence over sequences in portions of 1 to 61 rows, beside one
    another in one batch, in slots that others held before; a portion of one row runs on the decode kernel in a batch of such
    rows alone. The results do not depend on the cutting, to the bit."""
    from research_2_b200.kernels import ops

    heads, groups, dim, vdim, n_taps = shape
    gen = torch.Generator().manual_seed(dim * 100 + vdim)
    width, channels = 37, 2 * groups * dim + heads * vdim
    taps = torch.randn(channels, n_taps, generator=gen) * 0.5
    w_gates = (torch.randn(2 * heads, width, generator=gen) * 0.3).to(dtype)
    step_bias, log_rate = torch.randn(heads, generator=gen), torch.randn(heads, generator=gen) - 0.5
    lengths = (61, 9, 40)
    seqs = [((torch.randn(n, channels, generator=gen)).to(dtype), torch.randn(n, width, generator=gen).to(dtype)) for n in lengths]
    want = [delta_reference(raw.double(), h.double(), taps, w_gates.double(), step_bias, log_rate, heads, groups, dim, vdim) for raw, h in seqs]
    off = heads * ops.scan_state_floats(dim, vdim)
    floats = -(-(off + (n_taps - 1) * channels) // 4) * 4
    weights = (taps.to(DEV), w_gates.to(DEV), step_bias.to(DEV), log_rate.to(DEV))

    def run(cuts, slots):
        """cuts: per step, the (sequence, rows) of its entries."""
        state = torch.full((5, floats), 1e4, device=DEV)     # what other requests left there
        at, outs = [0] * len(seqs), [[] for _ in seqs]
        for step in cuts:
            e = Entries([n for _, n in step], [slots[s] for s, _ in step], [at[s] == 0 for s, _ in step])
            raw = torch.cat([seqs[s][0][at[s]: at[s] + n] for s, n in step]).to(DEV)
            h = torch.cat([seqs[s][1][at[s]: at[s] + n] for s, n in step]).to(DEV)
            qk, v, numbers = ops.delta_prepare(raw, h, *weights, dim ** -0.5, 1e-6, heads, groups, dim, vdim, state, off, e.row_entry, *e.arrays)
            o = ops.delta_scan(qk, v, numbers, dim, state, *e.arrays, conv_in=raw, conv_taps=n_taps, conv_state_off=off).cpu()
            for i, (s, n) in enumerate(step):
                outs[s].append(o[e.of(i)])
                at[s] += n
        assert at == list(lengths) and float(state[[i for i in range(5) if i not in slots]].min()) == 1e4, "a slot of no entry changed"
        return [torch.cat(o) for o in outs]

    whole = run([[(0, 61), (1, 9), (2, 40)]], (3, 0, 2))
    for s, got in enumerate(whole):
        close(got, want[s], 2e-5, f"{shape} {dtype} sequence {s}")
    portions = run([[(0, 2), (2, 33)], [(0, 1), (1, 1), (2, 1)], [(0, 1), (1, 1), (2, 1)], [(2, 5), (0, 40)], [(1, 7), (0, 17)]], (1, 4, 0))
    single = run([[(0, 1), (1, 1), (2, 1)]] * 9 + [[(0, 1), (2, 1)]] * 31 + [[(0, 1)]] * 21, (0, 1, 2))
    for s in range(3):
        assert torch.equal(portions[s], whole[s]) and torch.equal(single[s], whole[s]), f"{shape}: sequence {s} depends on its cutting"


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("shape", [(2, 16, 64, 5), (3, 14, 42, 1), (1, 128, 96, 16), (4, 8, 30, 9), (2, 64, 128, 33), (5, 3, 17, 2), (1, 200, 40, 4), (2, 32, 64, 12)])
def test_time_mixing_alone(shape, dtype):
    """The mixes with the row before, the decays, and the recurrence, in the cuttings of the delta rule's test."""
    from research_2_b200.kernels import ops

    heads, dim, width, rank = shape
    gen = torch.Generator().manual_seed(dim * 100 + width)
    n = heads * dim
    mu = torch.rand(3, width, generator=gen)
    w1 = (torch.randn(rank, width, generator=gen) * width ** -0.5).to(dtype)
    w2 = (torch.randn(n, rank, generator=gen) * rank ** -0.5).to(dtype)
    w0, bonus = torch.randn(n, generator=gen) - 1.0, torch.randn(n, generator=gen)
    lengths = (61, 9, 40)
    seqs = [tuple(torch.randn(t, c, generator=gen).to(dtype) for c in (width, 3 * n)) for t in lengths]
    off = heads * ops.scan_state_floats(dim, dim)
    floats = -(-(off + width) // 4) * 4
    want_mix, want_decay, want = [], [], []
    for h, rkv in seqs:
        h = h.double()
        step = plain.shifted(h) - h
        want_mix.append(torch.stack([h + step * mu[s].double() for s in range(2)], dim=1))
        mix_w = h + step * mu[2].double()
        decay = torch.exp(-torch.exp(torch.tanh(mix_w @ w1.double().T) @ w2.double().T + w0.double()))
        want_decay.append(decay)
        r, k, v = (x.reshape(-1, heads, dim) for x in rkv.double().split(n, dim=1))
        want.append(plain.time_mix_core(r, k, v, decay.view(-1, heads, dim), bonus.double().view(heads, dim))[0].reshape(-1, n))
    weights = (mu.to(DEV), w1.to(DEV), w2.T.contiguous().to(DEV), w0.to(DEV))

    def run(cuts, slots):
        state = torch.full((5, floats), 1e4, device=DEV)
        at, outs = [0] * len(seqs), [[] for _ in seqs]
        for step in cuts:
            e = Entries([t for _, t in step], [slots[s] for s, _ in step], [at[s] == 0 for s, _ in step])
            h = torch.cat([seqs[s][0][at[s]: at[s] + t] for s, t in step]).to(DEV)
            rkv = torch.cat([seqs[s][1][at[s]: at[s] + t] for s, t in step]).to(DEV)
            mixes, decay = ops.time_mix_prepare(h, *weights, state, off, e.row_entry, *e.arrays)
            o = ops.time_mix_scan(rkv[:, :n], rkv[:, n: 2 * n], rkv[:, 2 * n:], decay, bonus.to(DEV), state, *e.arrays, heads, dim, row_in=h, row_state_off=off)
            for i, (s, t) in enumerate(step):
                outs[s].append((mixes[e.of(i)].cpu(), decay[e.of(i)].cpu(), o[e.of(i)].cpu()))
                at[s] += t
        assert at == list(lengths) and float(state[[i for i in range(5) if i not in slots]].min()) == 1e4, "a slot of no entry changed"
        return [tuple(torch.cat(parts) for parts in zip(*o)) for o in outs]

    whole = run([[(0, 61), (1, 9), (2, 40)]], (3, 0, 2))
    for s, (mixes, decay, o) in enumerate(whole):
        close(mixes, want_mix[s], 1e-6 if dtype == torch.float32 else 1e-2, f"{shape} mixes")
        close(decay, want_decay[s], 2e-6, f"{shape} decays")
        close(o, want[s], 2e-5, f"{shape} {dtype} sequence {s}")
    portions = run([[(0, 2), (2, 33)], [(0, 1), (1, 1), (2, 1)], [(0, 1), (1, 1), (2, 1)], [(2, 5), (0, 40)], [(1, 7), (0, 17)]], (1, 4, 0))
    single = run([[(0, 1), (1, 1), (2, 1)]] * 9 + [[(0, 1), (2, 1)]] * 31 + [[(0, 1)]] * 21, (0, 1, 2))
    for other in (portions, single):
        for s in range(3):
            assert all(torch.equal(a, b) for a, b in zip(other[s], whole[s])), f"{shape}: sequence {s} depends on its cutting"


def test_many_rows_at_once_give_the_same_bits():
    """Batches that the preparing kernels take one, four and eight rows a CTA at a time, with pad rows of no entry between them."""
    from research_2_b200.kernels import ops

    gen = torch.Generator().manual_seed(4)
    heads, groups, dim, vdim, taps_n, width, rank = 4, 2, 24, 16, 4, 50, 7
    channels, n = 2 * groups * dim + heads * vdim, 1400
    raw, h = torch.randn(n, channels, generator=gen).to(DEV), torch.randn(n, width, generator=gen).to(DEV)
    d_weights = (torch.randn(channels, taps_n, generator=gen).to(DEV), torch.randn(2 * heads, width, generator=gen).to(DEV), torch.randn(heads, generator=gen).to(DEV),
                 torch.randn(heads, generator=gen).to(DEV))
    t_weights = (torch.rand(5, width, generator=gen).to(DEV), torch.randn(rank, width, generator=gen).to(DEV), torch.randn(rank, 40, generator=gen).to(DEV),
                 torch.randn(40, generator=gen).to(DEV))
    state = torch.randn(3, 4096, generator=gen).to(DEV)

    def both(rows, start, fresh):
        e = Entries([rows], [1], [fresh])
        a = ops.delta_prepare(raw[start: start + rows], h[start: start + rows], *d_weights, 0.2, 1e-6, heads, groups, dim, vdim, state, 8, e.row_entry, *e.arrays)
        b = ops.time_mix_prepare(h[start: start + rows], *t_weights, state, 16, e.row_entry, *e.arrays)
        return a + b

    whole = both(n, 0, False)
    for rows in (100, 500):
        for x, y in zip(both(rows, 0, False), whole):
            assert torch.equal(x, y[:rows]), rows
    # an entry's rows beside others: 5 rows, 7 pad rows, 900 rows; the second entry starts fresh
    lengths = (5, 900)
    row_entry = i32([0] * 5 + [1] * 900 + [-1] * 7)
    q_start, slots, fresh = i32([0, 5, 905]), i32([2, 0]), i32([0, 1])
    rows = sum(lengths) + 7
    a = ops.delta_prepare(raw[:rows], h[:rows], *d_weights, 0.2, 1e-6, heads, groups, dim, vdim, state, 8, row_entry, q_start, slots, fresh)
    b = ops.time_mix_prepare(h[:rows], *t_weights, state, 16, row_entry, q_start, slots, fresh)
    alone = both(900, 5, True)
    for x, y in zip(a + b, alone):
        assert torch.equal(x[5: 905], y)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("shape", [(4, 2, 16), (1, 1, 20), (6, 2, 64), (3, 3, 7), (40, 8, 80), (12, 3, 64)])
def test_norms_over_whole_query_and_key_rows(shape, dtype):
    """One root mean square over all heads; the normed keys to columns of their own or to the cache only; the values in the cache
    are the keys as projected."""
    from research_2_b200.kernels import ops

    heads, kv_heads, dim = shape
    gen = torch.Generator().manual_seed(sum(shape))
    rows, page, eps, n_pages = 61, 4, 1e-3, 20
    q_w, k_w = heads * dim, kv_heads * dim
    gq, gk = 1.0 + 0.3 * torch.randn(q_w, generator=gen), 1.0 + 0.3 * torch.randn(k_w, generator=gen)
    proj = (torch.randn(rows, q_w + 2 * k_w, generator=gen) * 2).to(dtype)
    proj[5, : q_w + k_w] = 0.0   # eps stands inside the root
    want_q = plain.rms_norm(proj[:, :q_w].double(), gq, eps)
    want_k = plain.rms_norm(proj[:, q_w: q_w + k_w].double(), gk, eps)
    tol = 2e-6 if dtype == torch.float32 else 8e-3
    dev = proj.to(DEV)
    ops.row_norm(dev, q_w, k_w, gq.to(DEV), gk.to(DEV), eps, k_out_col=q_w + k_w)
    close(dev[:, :q_w], want_q, tol)
    close(dev[:, q_w + k_w:], want_k, tol)
    assert torch.equal(dev[:, q_w: q_w + k_w].cpu(), proj[:, q_w: q_w + k_w]), "the keys as projected changed"
    slots = (torch.randperm((n_pages - 1) * page, generator=gen)[:rows] + page).to(torch.int32).to(DEV)
    stride = 2 * kv_heads * page * dim
    pool = torch.full((n_pages * stride,), 7.0, dtype=dtype, device=DEV)
    cached = proj.to(DEV)
    scatter = ops.kv_scatter(slots, pool, pool[kv_heads * page * dim:], stride, page, n_pages, q_w, k_w, dim)
    ops.row_norm(cached, q_w, k_w, gq.to(DEV), gk.to(DEV), eps, kv=scatter, head_dim=dim)
    assert torch.equal(cached[:, :q_w], dev[:, :q_w]) and torch.equal(cached[:, q_w:].cpu(), proj[:, q_w:])
    pages = pool.view(n_pages, 2, kv_heads, page, dim)
    for t in range(rows):
        p, o = int(slots[t]) // page, int(slots[t]) % page
        assert torch.equal(pages[p, 0, :, o].reshape(-1), dev[t, q_w + k_w:]) and torch.equal(pages[p, 1, :, o].reshape(-1), dev[t, q_w: q_w + k_w])
    assert float(pages[0].min()) == 7.0 == float(pages[0].max()), "the null page was written"


ATTENTION_SHAPES = [(4, 2, 64, 16, 48), (3, 1, 80, 4, 33), (1, 1, 24, 8, 5), (8, 1, 128, 32, 100), (2, 2, 32, 64, 0), (6, 2, 16, 16, 64), (9, 1, 20, 8, 40), (2, 1, 144, 16, 7)]


@pytest.mark.parametrize("cut", ["prompts", "decoded", "portions"])
@pytest.mark.parametrize("shape", ATTENTION_SHAPES)
def test_attention_by_chunks_with_a_bias_by_distance(shape, cut):
    """The kernels alone: chunks, biases (a table that ends inside the chunk, and at its last distance a value of its own), learned
    sinks, a factor on the output, pages scattered in a pool full of large numbers. bfloat16 on the fast kernels and on the
    general one, float32 on the general one."""
    from research_2_b200.kernels import ops

    heads, kv, dim, page, chunk = shape
    gen = torch.Generator().manual_seed(heads * 1000 + dim)
    lengths = [1, 2, 63, 64, 65, 130, 200, 101]
    scale, factor, reach = dim ** -0.5, 1.7, 50
    sinks, bias = torch.randn(heads, generator=gen) * 2, torch.randn(heads, reach, generator=gen) * 2
    sinks[0] = 12.0
    bias[:, -1] = 3.0
    k = [(torch.randn(n, kv, dim, generator=gen) * 1.5).to(torch.bfloat16) for n in lengths]
    v = [torch.randn(n, kv, dim, generator=gen).to(torch.bfloat16) for n in lengths]
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
    if cut == "decoded" and chunk:   # pages of earlier chunks are gone: their places in the table name the null page
        for e, (a, _) in enumerate(spans):
            tables[e, : a // chunk * chunk // page] = 0
    entry_rows = [b - a for a, b in spans]
    q_start = [sum(entry_rows[:i]) for i in range(len(lengths) + 1)]
    positions = [p for a, b in spans for p in range(a, b)]
    row_entry = [e for e, (a, b) in enumerate(spans) for _ in range(a, b)]
    q = (torch.randn(len(positions), heads * dim, generator=gen) * 1.5).to(torch.bfloat16)
    full_bias = torch.cat([bias, bias[:, -1:].expand(heads, 200)], dim=1).double()
    want = torch.cat([plain.chunk_attention_core(q[q_start[e]: q_start[e + 1]].double().view(-1, heads, dim), k[e].double(), v[e].double(), scale, full_bias,
                                                 sinks.double(), chunk, positions=list(range(*spans[e]))) for e in range(len(lengths))]).reshape(len(positions), -1) * factor
    extras = dict(chunk=chunk, dist_bias=bias.to(DEV), sinks=sinks.to(DEV), out_scale=factor)
    where = (i32(row_entry), i32(positions), i32([b for _, b in spans]), heads, kv, dim, scale)

    def paged(dtype):
        flat = pool.to(dtype).to(DEV).view(-1)
        return ops.paged_attention(q.to(dtype).to(DEV), flat, flat[kv * page * dim:], 2 * kv * page * dim, page, n_pages, tables.to(DEV), *where,
                                   decode_only=cut == "decoded", max_context=max(lengths), q_start=i32(q_start), n_tiles=sum(-(-r // 64) for r in entry_rows), **extras)

    before = dict(ops.kernel_uses())
    close(paged(torch.bfloat16), want, 1.2e-2, f"{shape} {cut}")
    used = [name for name, n in ops.kernel_uses().items() if n > before.get(name, 0)]
    assert used == (["attention_prefill"] if dim % 16 == 0 and dim <= 128 else ["attention_simt"]), used
    close(paged(torch.float32), want, 2e-5, f"{shape} {cut} float32")
    old = ops.use_fast_attention(False)
    try:
        close(paged(torch.bfloat16), want, 1.2e-2, f"{shape} {cut} on the general kernel")
    finally:
        ops.use_fast_attention(old)
    if cut != "decoded":
        return
    # the decode kernel takes the newest key and value from the projection and puts them into the cache itself
    flat = pool.clone().to(DEV).view(-1)
    slot = [int(tables[e, (b - 1) // page]) * page + (b - 1) % page for e, (_, b) in enumerate(spans)]
    cells = flat.view(n_pages, 2, kv, page, dim)
    for s in slot:
        cells[s // page, :, :, s % page] = 55.0
    new = torch.stack([torch.cat([k[e][b - 1].reshape(-1), v[e][b - 1].reshape(-1)]) for e, (_, b) in enumerate(spans)]).to(DEV)
    got = ops.decode_attention_fused(q.to(DEV), new[:, : kv * dim], new[:, kv * dim:], i32(slot), flat, flat[kv * page * dim:], 2 * kv * page * dim, page, n_pages,
                                     tables.to(DEV), *where, 0, max(lengths), exact_weights=True, **extras)
    if dim % 16 or heads // kv > 8:
        assert got is None
        return
    close(got, want, 1.2e-2, f"{shape} fused")
    assert torch.equal(flat.view(-1).cpu(), pool.view(-1)), "the new keys and values are in their places and nothing else changed"


@pytest.mark.parametrize("rows", [1, 8, 50, 64, 65, 200, 1500])
def test_products_side_by_side(rows):
    """Several inputs, each times a matrix of its own, in one launch where groups are multiples of a tile."""
    from research_2_b200.kernels import ops

    gen = torch.Generator().manual_seed(rows)
    for groups, k, n in ((4, 96, 128), (3, 72, 256), (4, 64, 80), (2, 200, 384), (1, 64, 128)):
        a = torch.randn(rows, groups, k, generator=gen)
        w = torch.randn(groups * n, k, generator=gen) * 0.2
        for dtype, tol in ((torch.float32, 1e-5), (torch.bfloat16, 6e-3)):
            x, m = a.to(dtype), w.to(dtype)
            want = torch.cat([x[:, s].double() @ m[s * n: (s + 1) * n].double().T for s in range(groups)], dim=1)
            launches = ops.launch_count()
            got = ops.grouped_linear(x.to(DEV), m.to(DEV))
            close(got, want, tol, (rows, groups, k, n, dtype))
            if dtype == torch.bfloat16 and n % 128 == 0:
                assert ops.launch_count() == launches + 1
    old = ops.use_pair_gemm("always")
    try:
        a, w = torch.randn(300, 4, 128, generator=gen).to(torch.bfloat16), (torch.randn(4 * 256, 128, generator=gen) * 0.2).to(torch.bfloat16)
        want = torch.cat([a[:, s].double() @ w[s * 256: (s + 1) * 256].double().T for s in range(4)], dim=1)
        close(ops.grouped_linear(a.to(DEV), w.to(DEV)), want, 6e-3, "pairs of CTAs")
    finally:
        ops.use_pair_gemm(old)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_the_tokens_own_rows_and_the_capped_logits(dtype):
    from research_2_b200.kernels import ops
    from research_2_b200.parts import Runtime, registry

    gen = torch.Generator().manual_seed(5)
    vocab, eps = 40, 1e-3
    for rows, width, dim, layers, i in ((9, 48, 8, 3, 1), (70, 100, 5, 2, 0), (200, 64, 32, 4, 3)):
        table = torch.randn(vocab, layers * dim, generator=gen).to(dtype)
        gate, proj = (torch.randn(dim, width, generator=gen) * 0.2).to(dtype), (torch.randn(width, dim, generator=gen) * 0.4).to(dtype)
        gain = 1.0 + 0.3 * torch.randn(width, generator=gen)
        part = registry("token_side")["gated_rows"]({"column": i * dim, "dim": dim, "eps": eps}, {"table": table, "gate": gate, "proj": proj, "norm": gain},
                                                    Runtime(torch.device(DEV), dtype))
        x = torch.randn(rows, width, generator=gen)
        ids = torch.randint(0, vocab, (rows,), generator=gen)
        w = {"gate": gate.double(), "proj": proj.double(), "norm": gain}
        h = x.to(dtype)
        want = x.double() + plain.side_input(h.double(), table[ids, i * dim: (i + 1) * dim].double(), w, "", eps)

        class Ctx:
            input_ids = ids.to(torch.int32).to(DEV)

        new, rounded = part.join(x.to(DEV), h.to(DEV), Ctx, dtype if dtype != torch.float32 else None)
        close(new, want, 1e-5 if dtype == torch.float32 else 1e-2)
        assert rounded is None if dtype == torch.float32 else torch.equal(rounded, new.to(dtype))
    x = torch.linspace(-300, 300, 997)
    close(ops.soft_cap(x.to(DEV).clone(), 12.5), 12.5 * torch.tanh(x.double() / 12.5), 1e-6)
    # the gated unit with biases
    from research_2_b200.parts.mlp import GatedMLP
    gate, up, down = (torch.randn(s, generator=gen).to(dtype) * 0.2 for s in ((50, 40), (50, 40), (40, 50)))
    bias = {n: torch.randn(k, generator=gen) for n, k in (("b_gate", 50), ("b_up", 50), ("b_down", 40))}
    mlp = GatedMLP({"activation": "gelu_tanh"}, {"w_gate": gate, "w_up": up, "w_down": down, **bias}, Runtime(torch.device(DEV), dtype))
    h = torch.randn(33, 40, generator=gen).to(dtype)
    w = {"gate": gate.double(), "gate.b": bias["b_gate"], "up": up.double(), "up.b": bias["b_up"], "down": down.double(), "down.b": bias["b_down"]}
    close(mlp.mix(h.to(DEV), None), plain.feed_forward(h.double(), w, ""), 2e-5 if dtype == torch.float32 else 1.5e-2)


# ---------------------------------------------------------------------------------------------
# one key that stands out: in the chunk and out of it, at pages' borders, at the first token, far back in a carried state


QUERY_TOKEN, KEY_TOKEN = 1, 2


def planted_model(folder: Path, kind: str, chunk: int = 0) -> Path:
    """One layer whose weights are made so that the token QUERY_TOKEN asks for exactly what the token KEY_TOKEN left: coordinate 0 of the
    stream drives the query, coordinate 1 the key, both along one direction of head 0. In attention such a key's score is about 25
    above the others wherever it is visible; in a recurrence nothing decays and no other token writes along that direction, so the
    state returns what was written there. What the other mixer of a pair makes is left out (its output matrix is zero)."""
    from research_2_b200 import models  # noqa: F401  (registers the architectures)
    from research_2_b200.config.registry import architecture_of
    from research_2_b200.weights.safetensors_io import write_file

    width, dim = 36, 16
    heads, kv = 4, 2
    one = delta(2, 1, dim, 24, 3) if kind == "delta" else parallel(heads, kv, dim, 25.0 / (dim * (heads * kv) ** 0.5), chunk, 30, 2, dim, (1.5, 1.5))
    config = model(64, width, [one], eps=1e-5, alpha=0.1, max_positions=800)
    arch = architecture_of(config)
    w = arch.random_weights(arch.parse_config(config), 17, std=0.08, bias_rows=8, decay_rank=4)
    gen = torch.Generator().manual_seed(18)
    w["pos"] *= 0.1
    w["pos"][:, :2] = 0.0
    w["embed"][:, :2] = 0.0
    for token, coordinate in ((QUERY_TOKEN, 0), (KEY_TOKEN, 1)):
        w["embed"][token] *= 0.1
        w["embed"][token, coordinate] = 6.0
    direction = torch.randn(dim, generator=gen)
    p = "l0.mix."
    if kind == "attention":
        for name, coordinate in (("left.q", 0), ("left.k", 1)):
            w[p + name][:, coordinate] = 0.0
            w[p + name][:dim, coordinate] = direction
            w[p + name + ".norm"] = torch.ones_like(w[p + name + ".norm"])
            w[p + name + ".b"] *= 0.1
        w[p + "left.sink"] = torch.tensor([0.5, -0.5, 1.0, 0.0])
        w[p + "right.o"] *= 0.0
    else:
        half = dim // 2
        prefix, query, key = (p, "q", "k") if kind == "delta" else (p + "right.", "r", "k")
        for name, coordinate in ((query, 0), (key, 1)):
            w[prefix + name][:half] = 0.0
            w[prefix + name][:, coordinate] = 0.0
            w[prefix + name][:half, coordinate] = direction[:half]
        if kind == "delta":
            w[p + "A_log"] = torch.full_like(w[p + "A_log"], -14.0)
            for name in "qkv":
                w[p + name + ".conv"][:, :-1] = 0.0
                w[p + name + ".conv"][:, -1] = 1.0
        else:
            w[p + "right.w0"] = torch.full_like(w[p + "right.w0"], -14.0)
            w[p + "right.w2"] *= 0.0
            for s in "rkv":
                w[p + f"right.mu.{s}"] *= 0.0
            w[p + "left.o"] *= 0.0
            w[p + "right.v"] *= 5.0
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


# asking row, distance of the key (chunks of 40 in pages of 16: chunks begin inside pages)
CHUNK_CASES = [(119, 39), (119, 40), (120, 1), (121, 1), (121, 2), (119, 1), (159, 39), (159, 40), (39, 39), (40, 40), (41, 1), (143, 15), (144, 16), (144, 24),
               (144, 25), (700, 20), (700, 21), (719, 39), (719, 40), (130, 3)]
OPEN_CASES = [(650, 600), (229, 229), (229, 1), (130, 2), (130, 3), (130, 18), (130, 19), (144, 16), (77, 77), (300, 172)]
STATE_CASES = [(650, 600), (229, 229), (77, 1), (130, 127), (66, 64)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("how", ["prompt", "decoded", "portion_between"])
@pytest.mark.parametrize("kind", ["chunk", "open", "delta", "time_mix"])
def test_one_key_that_stands_out(tmp_path, dtype, how, kind):
    """The asking row in a prompt, decoded alone, or first in a portion that begins between the key and the row (for chunks also
    where the portion begins in the middle of the chunk). Inside the chunk the logits are those with the key, outside those of a
    sequence without it."""
    cases = {"chunk": CHUNK_CASES, "open": OPEN_CASES}.get(kind, STATE_CASES)
    folder = planted_model(tmp_path / kind, "attention" if kind in ("chunk", "open") else kind, 40 if kind == "chunk" else 0)
    for ask_at, distance in cases:
        ids = planted_sequence(ask_at + 6, ask_at, distance, seed=ask_at)
        truth = plain_logits(folder, ids)[ask_at]
        without = plain_logits(folder, planted_sequence(ask_at + 6, ask_at, 0, seed=ask_at))[ask_at]
        gap, size = float(np.abs(truth - without).max()), float(np.abs(truth).max())
        if kind == "chunk" and (ask_at - distance) // 40 != ask_at // 40:
            assert gap < 1e-9, (kind, ask_at, distance, gap)
        else:
            assert gap > 0.25 * size, (kind, ask_at, distance, gap, size)
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
        assert float(np.abs(got - truth).max()) < 0.15 * size, f"{kind} {how} row {ask_at} distance {distance}"


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
    chunks = {layer["mixer"]["left"].get("mask", {}).get("size", 0) for layer in CASES[name]["config"]["layers"] if layer["type"] == "parallel"}
    assert {g.chunk for g in replay.cache.groups} == chunks, "one cache group per chunk size"
    if mode == "mixed":
        assert traces.max_live(tb) == 4 and len(requests) > 4, "request and state slots are used again"
        assert reused >= 2, f"only {reused} pages passed from one request to another"


def test_the_stream_after_every_layer(folders):
    """The stream after each layer (not only the logits), in float32: a layer that is wrong and then drowned by the next
    norm shows here."""
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
                got.append(x.detach().double().cpu().clone())
                return x
            b.forward = tapped
        replay.step({"step": 0, "entries": [{"id": "x", "tokens": ids, "want": [len(ids) - 1]}], "end": ["x"]})
        assert len(got) == len(want)
        for i, (a, b) in enumerate(zip(got, want)):
            assert float((a[: len(ids)] - b).abs().max()) <= 3e-5 * float(b.abs().max()), (name, i)


def test_sequences_longer_than_their_pool(tmp_path):
    """Where every layer has chunks, a sequence needs the pages of its chunk alone: 300 tokens in a pool of 96."""
    case = {"config": model(61, 48, [parallel(2, 1, 16, 0.3, 20, 30, 2, 8, ff=40), parallel(4, 2, 8, 0.3, 32, 30, 1, 16), delta(2, 1, 8, 8, 4)], alpha=1.5, side=6),
            "seed": 4, "std": 0.08, "bias_rows": 8, "decay_rank": 3}
    folder = make_model_dir(tmp_path / "model", case)
    ids = random_tokens(2, 300, 61)
    for dtype in ("float32", "bfloat16"):
        tb = traces.portions({"x": ids}, sizes=(30, 1, 17, 2, 1, 1, 24))
        outputs, _, replay = run_trace(folder, tb, dtype, 8, max_tokens=96, max_seq_len=320)
        compare(folder, {"x": ids}, tb, outputs, dtype, f"short pool {dtype}")
        assert all(g.num_pages * 8 < 200 for g in replay.cache.groups)


def test_which_kernels_serve_bfloat16(folders):
    """Case d has the shapes that the fast kernels are written for: its attention runs on the tensor-core prefill kernel and the
    fused decode kernel, which writes the new key itself."""
    from research_2_b200.kernels import ops

    folder, name = folders["d"], "d"
    ids = random_tokens(3, 150, CASES[name]["config"]["vocab"])
    tb = traces.prefill_then_decode({"x": ids}, n_decode=4)
    before = dict(ops.kernel_uses())
    outputs, _, _ = run_trace(folder, tb, "bfloat16", CASES[name]["page_size"])
    compare(folder, {"x": ids}, tb, outputs, "bfloat16", "kernels of case d")
    used = {k: v - before.get(k, 0) for k, v in ops.kernel_uses().items()}
    assert used.get("attention_decode_fused", 0) == 8 and used.get("attention_prefill", 0) == 2 and used.get("attention_simt", 0) == 0, used


@pytest.mark.parametrize("seed", range(100, 112))
def test_configurations_drawn_at_random(seed, tmp_path):
    """Layers in any order and sizes of any kind: float32 within its floor in three cuttings, bfloat16 within its own."""
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
    """400 tokens, 390 of them decoded one by one: through many chunks, with states carried all the way."""
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
