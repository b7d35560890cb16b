"""Shared by the Paditar tests: tiny model folders, engines on them, the plain logits with what rounding alone does to them."""
import functools
import os

import numpy as np

import model_helpers as mh
import plain_paditar as plain
import tiny_paditar



@functools.lru_cache(maxsize=None)
def model_folder(name: str) -> str:
    from rust_deeplearning_b200 import write_random_model
    cfg, seed = tiny_paditar.config(name)
    folder = os.path.join(mh.tmp_root(), f"tiny_{name}")
    write_random_model(folder, cfg, seed, "bfloat16")
    return folder


@functools.lru_cache(maxsize=None)
def plain_model(name: str):
    return plain.load_folder(model_folder(name))


@functools.lru_cache(maxsize=None)
def loaded_model(name: str, dtype: str):
    from rust_deeplearning_b200 import load_model
    return load_model(model_folder(name), dtype, "cuda:0")


def engine(name: str, dtype: str, **kw):
    from rust_deeplearning_b200 import Engine
    kw.setdefault("max_tokens", 4096)
    return Engine(loaded_model(name, dtype), **kw)


def vocab(name):
    return tiny_paditar.config(name)[0]["vocab"]


def prompt(name: str, seed: int, n: int):
    return mh.prompt(seed, n, vocab(name))


class Want:
    """Plain logits and, per dtype, how far an implementation's may lie from them at each position: the usual share of the largest
    logit, or four times the most that noise of the dtype's rounding (three samples; in bfloat16 also the rounding itself) moves the
    plain logits there, whichever is larger (a difference of two maps or a memory's read-out may nearly cancel before it is divided by its root mean square)."""

    def __init__(self, logits, limits):
        self.logits, self.limits = logits, limits

    def __getitem__(self, rows):
        return Want(self.logits[rows], {k: v[rows] for k, v in self.limits.items()})


def cat(parts):
    return Want(np.concatenate([p.logits for p in parts]), {k: np.concatenate([p.limits[k] for p in parts]) for k in parts[0].limits})


NOISE = {"float32": 2.0 ** -23, "bfloat16": 2.0 ** -9}


def plain_want(cfg, w, ids) -> Want:
    logits = plain.forward(cfg, w, list(ids))
    limits = {}
    for dtype, size in NOISE.items():
        samples = [plain.noise(size, seed) for seed in range(3)] + ([plain.to_bfloat16] if dtype == "bfloat16" else [])
        moved = np.max([np.abs(plain.forward(cfg, w, list(ids), r=r) - logits).max(axis=1) for r in samples], axis=0)
        limits[dtype] = np.maximum(mh.tolerance(dtype, logits), 4.0 * moved)
    return Want(logits, limits)


_WANT = {}


def plain_logits(name: str, ids) -> Want:
    key = (name, tuple(ids))
    if key not in _WANT:
        _WANT[key] = plain_want(*plain_model(name), ids)
    return _WANT[key]


def assert_logits(got, want: Want, dtype: str, what=""):
    got = got.detach().float().cpu().double().numpy()
    assert got.shape == want.logits.shape, (what, got.shape, want.logits.shape)
    assert np.isfinite(got).all(), f"{what}: non-finite logits"
    err = np.abs(got - want.logits).max(axis=1)
    over = err > want.limits[dtype]
    assert not over.any(), f"{what}: {int(over.sum())} of {len(over)} positions over their limit, the first is {int(over.argmax())}: {err[over.argmax()]:.3e} > {want.limits[dtype][over.argmax()]:.3e}"
