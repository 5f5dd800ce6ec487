"""Small Tagulix configurations for the tests, model folders with random weights, and the plain implementation's logits with
an error budget.

The configurations differ from one another in every size and constant, and between them cover the values that one model may happen to make
equal or trivial: layers in every order, of one kind only, that run with an earlier or a later layer's tensors (one of them by way of another
borrower), one head and several, as many key/value heads as heads, one for all and groups of three, value sizes that differ from the
keys' either way, sizes that are no multiple of 16, 8 or 4, windows smaller than a page, of one token, of many pages and none, rotations of
all dimensions, of two and none, bias tables of four rows and of more, queries with and without a temperature, decays of zero, one and
between, one stream, several and the plain residual sum, routers with one group and several, with and without identity outputs, that choose
one and that choose all, layers without a feed-forward, factors of one and of other sizes. Where a case has large corrections they
decide alone which experts are chosen (no choice is close, so bfloat16 can be compared everywhere); where they are small the scores do.
"""

from __future__ import annotations

import functools
from pathlib import Path

import numpy as np
import torch

from tests.plain import tagulix_plain


def moe(experts, identity, top, ff, groups=None, scale=None):
    router = {"experts": experts, "top": top}
    if identity:
        router["identity"] = identity
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    if scale is not None:
        router["scale"] = scale
    return {"kind": "moe", "expert": {"ff": ff}, "router": router}


def attention(heads, kv_heads, dim, vdim, scale, window=None, rot=None, mlp=None, weights_of=None):
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if window:
        mixer["mask"] = {"size": window}
    if rot:
        mixer["rot"] = {"dims": rot[0], "base": rot[1]}
    out = {"type": "attention", "mixer": mixer, "mlp": mlp}
    return out if weights_of is None else {**out, "weights_of": weights_of}


def parallel(left, right, scales=(1.0, 1.0), temp=None, mlp=None, weights_of=None):
    """left: (heads, kv_heads, dim, vdim, scale, bias_max); right: (decay, dim, vdim); temp: (coef, every)."""
    side = dict(zip(("heads", "kv_heads", "dim", "vdim", "scale", "bias_max"), left))
    if temp:
        side["q_temp"] = {"coef": temp[0], "every": temp[1]}
    mixer = {"left": side, "left_scale": scales[0], "right": {"heads": len(right[0]), "decay": list(right[0]), "dim": right[1], "vdim": right[2]},
             "right_scale": scales[1]}
    out = {"type": "parallel", "mixer": mixer, "mlp": mlp}
    return out if weights_of is None else {**out, "weights_of": weights_of}


def model(vocab, width, layers, eps=1e-6, streams=None, mult=None):
    out = {"architecture": "Tagulix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if streams is not None:
        out["streams"] = streams
    if mult is not None:
        out["residual_mult"] = mult
    return out


_A_MOE, _A_MOE2 = moe(6, 2, 3, 40, (4, 2), 1.7), moe(5, 1, 2, 24, (3, 1), 0.6)
_A_ATT = dict(heads=4, kv_heads=2, dim=16, vdim=16, scale=0.4, window=24, rot=(8, 1000.0), mlp=_A_MOE)
_A_PAR = dict(left=(4, 2, 16, 16, 0.3, 20), right=((0.5, 0.97), 16, 16), scales=(0.8, 1.4), temp=(0.7, 10), mlp=_A_MOE2)
_B_PAR = dict(left=(3, 1, 10, 6, 0.4, 9), right=((0.0, 1.0, 0.8), 5, 7), scales=(1.0, 2.0), mlp=moe(3, 0, 3, 30))
_D_ATT = dict(heads=4, kv_heads=2, dim=64, vdim=64, scale=0.3, window=48, rot=(64, 500.0), mlp=moe(6, 2, 4, 64, (2, 1), 1.2))
CASES = {
    # both mixers, borrowers before and after their lender, three streams; windows of 24 in pages of 16
    "a": {"config": model(211, 64, [
        attention(**_A_ATT, weights_of=2), parallel(**_A_PAR), attention(**_A_ATT), attention(4, 4, 24, 32, 0.2, 40, None),
        parallel(**_A_PAR, weights_of=1), attention(**_A_ATT, weights_of=0),
    ], eps=1e-6, streams=3, mult=0.8), "seed": 3, "std": 0.08, "page_size": 16, "bias_rows": 8, "correction_std": 30.0},
    # sizes that are no multiple of 4 or 8, one head, one stream, no groups or identities, every expert chosen, windows of 5 and 1 in pages of 8
    "b": {"config": model(97, 42, [
        parallel(**_B_PAR), attention(3, 1, 10, 6, 0.5, 5, (10, 50.0), mlp=moe(4, 3, 1, 26, (7, 2), 2.5)), attention(1, 1, 7, 33, 0.4, None, (2, 7.0)),
        parallel((1, 1, 20, 20, 0.5, 40), ((0.9,), 33, 12), (0.7, 1.0), (-0.3, 1)), attention(2, 1, 12, 5, 0.3, 1),
    ], eps=2e-5, streams=1, mult=1.3), "seed": 5, "std": 0.1, "page_size": 8, "bias_rows": 4, "correction_std": 0.2},
    # side by side only, the plain residual sum, heads in groups of three and of eight, pages of 32
    "c": {"config": model(300, 96, [
        parallel((6, 2, 16, 16, 0.25, 64), ((0.99, 0.6, 0.3), 32, 32), mlp=moe(2, 2, 2, 70, (2, 2))), parallel((3, 3, 40, 24, 0.15, 50), ((0.7, 0.9), 16, 40), temp=(1.2, 33)),
        parallel((8, 1, 32, 32, 0.2, 30), ((0.95, 1.0), 48, 16), (0.5, 0.5), (0.5, 7), mlp=moe(8, 0, 2, 128, (4, 2), 1.4)),
    ], eps=1e-5), "seed": 8, "std": 0.05, "page_size": 32, "bias_rows": 12, "correction_std": 30.0},
    # heads of 64 and more and experts of 64 columns (the tensor-core kernels' shapes), four streams, pages of 8
    "d": {"config": model(128, 128, [
        attention(**_D_ATT), parallel((4, 2, 64, 64, 0.125, 90), ((0.5, 0.999), 64, 64), (1.3, 0.9), (0.4, 20), mlp=moe(6, 2, 4, 64, (2, 1), 1.2)),
        attention(2, 1, 128, 128, 0.1, 48), attention(**_D_ATT, weights_of=0), parallel((2, 1, 80, 80, 0.1, 90), ((0.99,), 128, 96), (1.0, 1.1)),
    ], eps=1e-5, streams=4, mult=0.6), "seed": 13, "std": 0.06, "page_size": 8, "bias_rows": 32, "correction_std": 30.0},
}


def random_case(seed: int) -> dict:
    """A configuration drawn from a seed: one to five layers of either kind in any order, some with another's tensors, sizes that are and
    are not multiples of 16, every optional mechanism there or not."""
    import random

    rng = random.Random(seed)
    layers = []
    bias_rows = rng.choice([4, 6, 16, 32])

    def mlp():
        if rng.random() < 0.25:
            return None
        groups, per = rng.choice([1, 1, 2, 3]), rng.randint(2, 4)
        keep, total = rng.randint(1, groups), groups * per
        identity = rng.randint(0, total - 1)
        return moe(total - identity, identity, rng.randint(1, keep * per), rng.choice([8, 24, 33, 64, 96]), (groups, keep) if groups > 1 else None,
                   rng.choice([None, 0.7, 2.0]))

    for _ in range(rng.randint(1, 5)):
        kv, per, dim = rng.randint(1, 3), rng.choice([1, 2, 3, 4, 9]), rng.choice([6, 8, 16, 24, 32, 48, 64, 80, 128, 144])
        vdim = rng.choice([dim, dim, 10, 32, 64])
        if rng.random() < 0.5:
            layers.append(attention(kv * per, kv, dim, vdim, rng.choice([dim ** -0.5, 0.1, 0.3]), rng.choice([None, 1, 3, 16, 31, 64, 100]),
                                    rng.choice([None, (dim // 2 * 2, 10000.0), (dim // 4 * 2, 33.0)]), mlp=mlp()))
        else:
            decay = tuple(rng.choice([0.0, 0.5, 0.9, 0.999, 1.0]) for _ in range(rng.randint(1, 4)))
            layers.append(parallel((kv * per, kv, dim, vdim, rng.choice([dim ** -0.5, 0.1, 0.3]), rng.choice([bias_rows // 2 + 1, 24, 77, 300])),
                                   (decay, rng.choice([3, 8, 16, 20, 32, 64, 96]), rng.choice([5, 8, 16, 36, 64, 128])),
                                   (rng.choice([1.0, 0.3, 1.7]), rng.choice([1.0, 0.6, 2.2])), rng.choice([None, (0.5, 16), (1.5, 3), (0.2, 100)]), mlp=mlp()))
    for i in range(len(layers)):
        if rng.random() < 0.3:
            layers.append({**{k: v for k, v in layers[i].items() if k != "weights_of"}, "weights_of": i})
    config = model(rng.choice([50, 97, 256, 1000]), rng.choice([24, 40, 64, 72, 101, 128, 200, 320]), layers, eps=rng.choice([1e-6, 1e-5]),
                   streams=rng.choice([None, 1, 2, 3, 4, 5, 8, 9]), mult=rng.choice([None, 0.5, 1.0, 1.4]))
    return {"config": config, "seed": seed, "std": 0.06, "page_size": rng.choice([4, 8, 16, 32]), "length": rng.choice([40, 150, 300]), "bias_rows": bias_rows,
            "correction_std": 30.0 if seed % 2 else 0.2}


def make_model_dir(folder: Path, case: dict, store_dtype: str = "bfloat16") -> Path:
    from research_2_b200 import models  # noqa: F401  (registers the architectures)
    from research_2_b200.config.registry import architecture_of
    from research_2_b200.weights import write_model_folder

    arch = architecture_of(case["config"])
    return write_model_folder(folder, arch, arch.parse_config(case["config"]), case["seed"], store_dtype, std=case["std"],
                              bias_rows=case["bias_rows"], correction_std=case["correction_std"])


def random_tokens(seed: int, n: int, vocab: int) -> list[int]:
    gen = torch.Generator().manual_seed(seed)
    return torch.randint(0, vocab, (n,), generator=gen).tolist()


@functools.lru_cache(maxsize=64)
def _plain_cached(folder: str, ids: tuple) -> np.ndarray:
    cfg, w = tagulix_plain.read_model(folder)
    return tagulix_plain.forward(cfg, w, list(ids)).numpy()


def plain_logits(folder, ids) -> np.ndarray:
    return _plain_cached(str(folder), tuple(int(i) for i in ids))


@functools.lru_cache(maxsize=64)
def movement(folder: str, ids: tuple) -> np.ndarray:
    """Per position, how far the plain logits move when the rows that enter every sublayer are disturbed by relative noise of
    2^-9 (about bfloat16's rounding, which the engine applies in more places), the most over four draws. A position at which a router's
    choice (of a group or of an expert) hangs on a score gap below 0.01 is excused altogether (infinity), and so is every later one
    of the sequence."""
    cfg, w = tagulix_plain.read_model(folder)
    worst = np.zeros(len(ids))
    tagulix_plain.MARGINS = []
    try:
        truth = tagulix_plain.forward(cfg, w, list(ids)).numpy()
        for margin in tagulix_plain.MARGINS:
            worst[np.array(margin) < 0.01] = np.inf
        worst = np.maximum.accumulate(worst)
    finally:
        tagulix_plain.MARGINS = None
    for seed in range(4):
        gen = torch.Generator().manual_seed(1000 + seed)
        tagulix_plain.DISTURB = lambda x: x * (1 + 2.0 ** -9 * torch.randn(x.shape, generator=gen, dtype=torch.float64))
        try:
            moved = tagulix_plain.forward(cfg, w, list(ids)).numpy()
        finally:
            tagulix_plain.DISTURB = None
        worst = np.maximum(worst, np.abs(moved - truth).max(axis=1))
    return worst


FLOORS = {"float32": 1e-4, "bfloat16": 3e-2}


def assert_close_to_plain(got: np.ndarray, folder, ids, dtype_name: str, what: str = "") -> None:
    """|logit - truth| <= floor * max |truth| with truth in float64; floors 1e-4 (float32) and 3e-2 (bfloat16). In
    bfloat16 a position may also be off by three times what disturbances of the size of its rounding do to the plain logits
    there; positions from a router's first close call on are excused, and only those."""
    truth = plain_logits(folder, ids)
    allowed = np.full(len(truth), FLOORS[dtype_name] * float(np.abs(truth).max()))
    assert got.shape == truth.shape, (got.shape, truth.shape, what)
    err = np.abs(got.astype(np.float64) - truth).max(axis=1)
    if dtype_name == "bfloat16" and not bool((err <= allowed).all()):
        allowed = np.maximum(allowed, 3.0 * movement(str(folder), tuple(int(i) for i in ids)))
    if not bool((err <= allowed).all()):
        pos = int(np.argmax(~(err <= allowed)))
        raise AssertionError(f"{what}: |logit - truth| = {float(err[pos]):.3e} > allowed {float(allowed[pos]):.3e} at "
                             f"position {pos}, the first of {int((~(err <= allowed)).sum())} positions over their limit")
