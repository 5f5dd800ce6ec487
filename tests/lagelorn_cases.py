"""Small Lagelorn configurations for the tests, model folders with random weights, and the plain implementation's
logits with an error budget.

The configurations differ from one another in every size and constant, and between them cover the values that one model
may happen to make equal or trivial: layers in every order (the delta rule only, two mixers side by side only), one head and
several, as many key/value heads as heads, one for all and groups of three, key and value sizes of the delta rule that differ
either way, sizes that are no multiple of 16, 8 or 4, one tap and up to seven, chunks smaller than a page, larger than a page
and no multiple of one, no chunks at all, bias tables of four rows and of more, distances beyond the table's reach, a decay of
rank one, layers with and without a feed-forward for either mixer, factors of one and of other sizes on the two mixers and
on the stream, models without side input and without capped logits.
"""

from __future__ import annotations

import functools
from pathlib import Path

import numpy as np
import torch

from tests.plain import lagelorn_plain


def delta(heads, kv_heads, dim, vdim, conv, ff=None):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def parallel(heads, kv_heads, dim, scale, chunk, bias_max, mix_heads, mix_dim, scales=(1.0, 1.0), ff=None):
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale, "bias_max": bias_max}
    if chunk:
        left["mask"] = {"size": chunk}
    return {"type": "parallel", "mixer": {"left": left, "left_scale": scales[0], "right": {"heads": mix_heads, "dim": mix_dim}, "right_scale": scales[1]},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def model(vocab, width, layers, eps=1e-6, alpha=None, side=None, softcap=None, max_positions=1024):
    out = {"architecture": "Lagelorn", "vocab": vocab, "width": width, "max_positions": max_positions, "norm": {"eps": eps}, "layers": layers}
    if alpha is not None:
        out["postln_alpha"] = alpha
    if side is not None:
        out["token_side"] = {"dim": side}
    if softcap is not None:
        out["logit_softcap"] = softcap
    return out


CASES = {
    # both mixers, with and without feed-forwards; chunks of 24 in pages of 16
    "a": {"config": model(211, 64, [
        parallel(4, 2, 16, 0.3, 24, 20, 2, 16, (0.8, 1.4), ff=96), delta(4, 2, 16, 24, 4), delta(2, 2, 24, 8, 2, ff=40),
        parallel(2, 2, 32, 0.2, 40, 100, 4, 8, (1.5, 0.5)),
    ], eps=1e-6, alpha=2.0, side=8, softcap=20.0), "seed": 3, "std": 0.08, "page_size": 16, "bias_rows": 8, "decay_rank": 5},
    # sizes that are no multiple of 4 or 8, one head, one tap, a decay of rank one, chunks of 5 in pages of 8, no side input
    "b": {"config": model(97, 42, [
        delta(3, 1, 10, 6, 1, ff=30), parallel(3, 1, 12, 0.4, 5, 9, 1, 14, (1.0, 2.0)), delta(1, 1, 7, 33, 7),
        parallel(1, 1, 20, 0.5, 0, 40, 3, 5, (0.7, 1.0), ff=26),
    ], eps=2e-5, alpha=0.5, softcap=7.0), "seed": 5, "std": 0.1, "page_size": 8, "bias_rows": 4, "decay_rank": 1},
    # side by side in every layer, factors of one, plain logits, groups of three and of one, chunks of 33 and of 150 in pages of 32
    "c": {"config": model(300, 96, [
        parallel(6, 2, 16, 0.25, 33, 64, 3, 32), parallel(3, 3, 40, 0.15, 150, 50, 6, 16, ff=70), parallel(8, 1, 32, 0.2, 33, 30, 2, 48, (0.5, 0.5), ff=128),
    ], eps=1e-5, side=24), "seed": 8, "std": 0.05, "page_size": 32, "bias_rows": 12, "decay_rank": 20},
    # heads of 64 and more (the tensor-core kernels' shapes), groups of 128 features in the products side by side, pages of 4
    "d": {"config": model(128, 128, [
        delta(4, 2, 64, 32, 4, ff=96), parallel(4, 2, 64, 0.125, 48, 90, 2, 64, (1.3, 0.9), ff=120), delta(2, 1, 128, 64, 3),
        parallel(2, 1, 80, 0.1, 48, 90, 1, 128, (1.0, 1.1)),
    ], eps=1e-5, alpha=3.5, side=16, softcap=15.0), "seed": 13, "std": 0.06, "page_size": 4, "bias_rows": 32, "decay_rank": 16},
}


def random_case(seed: int) -> dict:
    """A configuration drawn from a seed: one to five layers of either kind in any order, sizes that are and are not
    multiples of 16, every optional mechanism there or not."""
    import random

    rng = random.Random(seed)
    layers = []
    bias_rows = rng.choice([4, 6, 16, 32])
    for _ in range(rng.randint(1, 5)):
        ff = rng.choice([None, 24, 50, 64, 144])
        if rng.random() < 0.5:
            groups = rng.randint(1, 3)
            layers.append(delta(groups * rng.choice([1, 2, 3]), groups, rng.choice([4, 8, 18, 32, 48, 64, 100, 128]), rng.choice([4, 9, 16, 32, 64, 72, 128]),
                                rng.randint(1, 6), ff=ff))
        else:
            groups, dim = rng.randint(1, 3), rng.choice([6, 8, 16, 24, 32, 48, 64, 80, 128, 144])
            layers.append(parallel(groups * rng.choice([1, 2, 3, 4, 9]), groups, dim, rng.choice([dim ** -0.5, 0.1, 0.3]), rng.choice([None, 3, 16, 31, 64, 100]),
                                   rng.choice([bias_rows // 2 + 1, 24, 77, 300]), rng.randint(1, 4), rng.choice([3, 8, 16, 20, 32, 64, 96]),
                                   (rng.choice([1.0, 0.3, 1.7]), rng.choice([1.0, 0.6, 2.2])), ff=ff))
    config = model(rng.choice([50, 97, 256, 1000]), rng.choice([24, 40, 64, 72, 101, 128, 200, 320]), layers, eps=rng.choice([1e-6, 1e-5]),
                   alpha=rng.choice([None, 1.0, 2.0, 4.0]), side=rng.choice([None, 4, 10, 32]), softcap=rng.choice([None, 10.0, 50.0]))
    return {"config": config, "seed": seed, "std": 0.06, "page_size": rng.choice([4, 8, 16, 32]), "length": rng.choice([40, 150, 300]),
            "bias_rows": bias_rows, "decay_rank": rng.choice([1, 4, 7, 16, 33])}


def make_model_dir(folder: Path, case: dict, store_dtype: str = "bfloat16") -> Path:
    from research_2_b200 import models  # noqa: F401  (registers the architectures)
    from research_2_b200.config.registry import architecture_of
    from research_2_b200.weights import write_model_folder

    arch = architecture_of(case["config"])
    return write_model_folder(folder, arch, arch.parse_config(case["config"]), case["seed"], store_dtype, std=case["std"],
                              bias_rows=case["bias_rows"], decay_rank=case["decay_rank"])


def random_tokens(seed: int, n: int, vocab: int) -> list[int]:
    gen = torch.Generator().manual_seed(seed)
    return torch.randint(0, vocab, (n,), generator=gen).tolist()


@functools.lru_cache(maxsize=64)
def _plain_cached(folder: str, ids: tuple) -> np.ndarray:
    cfg, w = lagelorn_plain.read_model(folder)
    return lagelorn_plain.forward(cfg, w, list(ids)).numpy()


def plain_logits(folder, ids) -> np.ndarray:
    return _plain_cached(str(folder), tuple(int(i) for i in ids))


@functools.lru_cache(maxsize=64)
def _movement_cached(folder: str, ids: tuple) -> np.ndarray:
    """Per position, how far the plain logits move when the rows that enter every sublayer are disturbed by relative
    noise of 2^-9 (about bfloat16's rounding, which the engine applies in more places), the most over four draws."""
    cfg, w = lagelorn_plain.read_model(folder)
    truth = _plain_cached(folder, ids)
    worst = np.zeros(len(ids))
    for seed in range(4):
        gen = torch.Generator().manual_seed(1000 + seed)
        lagelorn_plain.DISTURB = lambda x: x * (1 + 2.0 ** -9 * torch.randn(x.shape, generator=gen, dtype=torch.float64))
        try:
            moved = lagelorn_plain.forward(cfg, w, list(ids)).numpy()
        finally:
            lagelorn_plain.DISTURB = None
        worst = np.maximum(worst, np.abs(moved - truth).max(axis=1))
    return worst


FLOORS = {"float32": 1e-4, "bfloat16": 3e-2}


def assert_close_to_plain(got: np.ndarray, folder, ids, dtype_name: str, what: str = "") -> None:
    """|logit - truth| <= floor * max |truth| with truth in float64; floors 1e-4 (float32) and 3e-2 (bfloat16). In
    bfloat16 a position may also be off by three times what disturbances of the size of its rounding do to the plain logits
    there."""
    truth = plain_logits(folder, ids)
    allowed = np.full(len(truth), FLOORS[dtype_name] * float(np.abs(truth).max()))
    assert got.shape == truth.shape, (got.shape, truth.shape, what)
    err = np.abs(got.astype(np.float64) - truth).max(axis=1)
    if dtype_name == "bfloat16" and not bool((err <= allowed).all()):
        allowed = np.maximum(allowed, 3.0 * _movement_cached(str(folder), tuple(int(i) for i in ids)))
    if not bool((err <= allowed).all()):
        pos = int(np.argmax(~(err <= allowed)))
        raise AssertionError(f"{what}: |logit - truth| = {float(err[pos]):.3e} > allowed {float(allowed[pos]):.3e} at "
                             f"position {pos}, the first of {int((~(err <= allowed)).sum())} positions over their limit")
