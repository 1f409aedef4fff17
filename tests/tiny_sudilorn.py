"""Tiny configurations of the Sudilorn design for the tests, and the helper that writes them as model folders with
random weights.

The five differ in every size and option: widths and vocabularies (multiples of 8 and not), the order of the layers,
query heads per key/value head from one to ten, windows shorter than a page, longer than every prompt and none, kept first
tokens fewer than a page, more than a page, more than the window and none, rotations of part of a head, of all of it, with
and without scaling and none, convolutions of one to five taps, memories of sizes that the tensor-core kernels are built
for and of sizes that they are not, heads that share queries and keys, branch constants of 0 and 1 and others, experts in
one to eight groups, layers without a feed-forward.

The engine's random weights (N(0, 0.02) matrices) are made larger here, so that a fault shows: attention is peaked, the two
maps of a head differ and weigh alike, memories forget within a few tokens in some heads and keep hundreds in others, keys of
a memory repeat, write strengths cover (0, 1), and what sublayers add is as large as what they add to.
"""

from __future__ import annotations

import os

import numpy as np

ARCH = "Sudilorn"


def _mask(size, keep=None):
    return None if size is None else {"size": size} if keep is None else {"size": size, "keep_first": keep}


def _rot(dims, base, scaling=None):
    if not dims:
        return None
    r = {"dims": dims, "base": base}
    if scaling:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return r


def _without_none(d):
    return {k: v for k, v in d.items() if v is not None}


def _diff(heads, kv, dim, vdim, conv, diff, scale, window, rot, mlp):
    return {"type": "attention", "mixer": _without_none(dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, conv=conv, diff=diff, scale=scale, mask=_mask(window), rot=rot)),
            "mlp": mlp}


def _left(heads, kv, dim, vdim, scale, window, keep, rot):
    return _without_none(dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=scale, mask=_mask(window, keep), rot=rot))


def _right(heads, kv, dim, vdim, conv):
    return _without_none(dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, conv=conv))


def _par(left, right, left_scale, right_scale, mlp):
    return {"type": "parallel", "mixer": dict(left=left, right=right, left_scale=left_scale, right_scale=right_scale), "mlp": mlp}


def _moe(experts, top, ff, count=None, keep=None):
    router = {"experts": experts, "top": top}
    if count:
        router["groups"] = {"count": count, "keep": keep}
    return {"kind": "moe", "expert": {"ff": ff}, "router": router}


def _config(vocab, width, eps, mult, layers):
    return {"architecture": ARCH, "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult, "layers": layers}


# width 96: sizes the general kernels take; a window of 9 beside 3 kept tokens; two taps; five groups of two experts
Z1 = _config(211, 96, 1e-5, 0.7, [
    _par(_left(6, 2, 24, 20, 0.3, 9, 3, _rot(10, 500.0)), _right(4, 2, 20, 24, 2), 0.7, 1.3, _moe(10, 3, 40, 5, 2)),
    _diff(6, 3, 20, 28, 3, 0.35, 0.3, 17, _rot(12, 1000.0, (2.0, 64, 8.0, 1.0)), None)])
# width 128: tensor-core sizes; differential heads all on one kv head; a right branch alone in its size
Z2 = _config(300, 128, 1e-6, 0.4, [
    _diff(4, 1, 32, 64, 4, 0.6, 0.2, 70, _rot(32, 10000.0, (8.0, 128, 32.0, 1.0)), _moe(8, 2, 48)),
    _par(_left(4, 1, 64, 64, 0.12, 33, 5, _rot(64, 10000.0)), _right(4, 1, 64, 40, 4), 1.0, 0.8, _moe(6, 1, 72, 2, 1)),
    _par(_left(2, 2, 32, 32, 0.2, 20, 2, _rot(16, 100.0)), _right(3, 3, 32, 32, 3), 1.5, 1.0, None)])
# nothing a multiple of 8, and everything that can be left out or 1: one head each, one tap, a window of one token, no kept
# tokens, no rotation, every group kept, a left branch that weighs nothing
Z3 = _config(77, 100, 1e-5, 1.0, [
    _par(_left(1, None, 9, 11, 0.4, 1, 0, None), _right(1, None, 13, 7, 1), 0.0, 1.0, _moe(4, 4, 30, 4, 4)),
    _diff(1, None, 7, 10, 1, 0.2, 0.5, None, None, _moe(3, 2, 21)),
    _par(_left(3, 1, 14, 6, 0.3, 4, 9, _rot(6, 30.0)), _right(5, 5, 10, 14, 5), 1.0, 0.5, _moe(6, 2, 28, 2, 2))])
# width 256: heads of 128; ten query heads on each kv head; kept tokens over more than a page; a window without kept tokens
Z4 = _config(160, 256, 1e-6, 0.3, [
    _par(_left(8, 8, 128, 128, 0.08, 64, 20, _rot(128, 50000.0)), _right(4, 2, 128, 128, 3), 0.9, 1.1, _moe(32, 6, 40, 8, 3)),
    _diff(20, 2, 64, 128, 5, 0.5, 0.12, 100, _rot(32, 5000.0), _moe(16, 4, 64, 2, 1)),
    _par(_left(4, 2, 64, 128, 0.12, 40, None, _rot(20, 5000.0)), _right(2, 1, 128, 64, 4), 1.0, 1.0, _moe(8, 2, 56, 4, 1))])
# memories the tensor cores are not built for (keys of 96 over values of 136: more columns than a CTA has) beside attention
# over everything; a causal differential head of 128
Z5 = _config(90, 64, 1e-6, 0.5, [
    _par(_left(4, 2, 32, 64, 0.2, None, None, _rot(32, 1000.0)), _right(2, 1, 96, 136, 4), 1.0, 2.0, None),
    _diff(2, 1, 128, 128, 2, 0.8, 0.09, None, _rot(64, 1000.0), _moe(5, 2, 24))])

TINY = {"Z1": (Z1, 51, 16), "Z2": (Z2, 52, 8), "Z3": (Z3, 53, 16), "Z4": (Z4, 54, 16), "Z5": (Z5, 55, 16)}   # config, weight seed, page size
# models whose routers decide by their corrections, far apart, so that rounding flips no choice
CALM = ("Z2", "Z4", "Z5")

GAIN, EMBED_GAIN, QK_GAIN = 5.0, 40.0, 12.0


def _far_corrections(router, rng):
    """Corrections 0.4 apart in an order in which the last kept group's mark and the next one's are 0.6 apart."""
    groups = router.get("groups") or {"count": 1, "keep": 1}
    while True:
        c = rng.permutation(np.arange(router["experts"]) * 0.4 - 2.0)
        marks = np.sort([np.sort(part)[::-1][:2].sum() for part in c.reshape(groups["count"], -1)])[::-1]
        if groups["keep"] == groups["count"] or marks[groups["keep"] - 1] - marks[groups["keep"]] > 0.6:
            return c


def _shaped(name, key, t, rng):
    """What the tests want of a tensor, from the engine's random one."""
    last = key.split(".")[-1]
    uniform = lambda lo, hi: rng.uniform(lo, hi, size=t.shape)
    if key == "embed":
        return t * EMBED_GAIN
    if last in ("norm1", "norm2") or key == "final.norm":
        return uniform(-0.4, 0.4)
    if last in ("ls1", "ls2"):
        return uniform(0.4, 1.2) * rng.choice([-1.0, 1.0], size=t.shape)
    if last == "A_log":
        return uniform(-4.0, 1.5)
    if last == "dt_bias":
        return uniform(-3.0, 0.5)
    if last == "conv":
        return rng.standard_normal(t.shape) * 0.6
    if last in ("lq1", "lk1", "lq2", "lk2"):
        return rng.standard_normal(t.shape) * (0.8 / np.sqrt(t.shape[0]))
    if last == "b" and t.ndim == 1:
        return t * 20.0
    if last == "router":
        return t * (0.1 if name in CALM else 0.6)
    if last == "correction":
        return _far_corrections(TINY[name][0]["layers"][int(key.split(".")[0][1:])]["mlp"]["router"], rng) if name in CALM else rng.uniform(-1.2, 0.4, size=t.shape)
    if ".left." in key and last in ("q", "k"):
        return t * QK_GAIN
    if ".right." in key and last in ("a", "b"):
        return t * 1.0
    return t * GAIN if t.ndim >= 2 else t


def make_model_dir(tmp_dir, name: str, storage_dtype: str = "float32", config=None, seed=None) -> str:
    """Random weights from the engine's random mode, reshaped as above, stored in ``storage_dtype``."""
    import torch

    from qwen25vl_lite.weights import write_random_model
    from qwen25vl_lite.weights.safetensors_io import write_safetensors

    from plain.decoder import read_safetensors

    cfg, s, _ = TINY.get(name, (config, seed, None))
    cfg, s = config or cfg, seed or s
    folder = write_random_model(os.path.join(str(tmp_dir), f"tiny-{name}-{storage_dtype}"), cfg, s, "float32", prefix="")
    path = os.path.join(folder, "model.safetensors")
    tensors = read_safetensors(path)
    dtype = {"float32": torch.float32, "bfloat16": torch.bfloat16}[storage_dtype]
    rng = np.random.default_rng(s)

    def named():
        for key, value in tensors.items():
            yield key, torch.from_numpy(np.array(_shaped(name, key, np.asarray(value), rng), dtype=np.float32, copy=True)).to(dtype)

    write_safetensors(path, named(), metadata={"format": "pt"})
    return folder
