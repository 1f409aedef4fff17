"""Tiny configurations of the Mezinex design for the tests, and the helper that writes them as model folders with
random weights.

The five differ in every size and option: widths and vocabularies (multiples of 8 and not), one to five rows of the
residual stream and none (a plain residual), the order of the three mixers, which stretch of layers runs several times
(the first layers, one layer alone, the whole model, none), with and without a table of token pairs, logits scaled and
not, state spaces whose heads share B and C in groups of one to six and whose norm is cut into parts that are heads,
halves of heads or several heads, convolutions of one to five taps, latents of sizes that the tensor-core attention is
built for and of sizes that it is not, more than 16 heads on one latent, recurrences of one to five blocks, layers
without a feed-forward.

The engine's random weights (N(0, 0.02) matrices) are replaced or made larger here, so that a fault shows: attention is
peaked; a state space has heads that forget within a few tokens beside heads that keep hundreds, and steps that differ
from token to token; the recurrences remember for tens to hundreds of tokens; the mixing matrices of the stream are far
from symmetric and from the identity; the pair table weighs as much as the token table.
"""

from __future__ import annotations

import os

import numpy as np

ARCH = "Mezinex"


def _ssm(heads, vdim, state, groups, norm_groups, conv, ff):
    return {"type": "mamba2", "mixer": dict(heads=heads, vdim=vdim, state=state, groups=groups, norm_groups=norm_groups, conv=conv),
            "mlp": ff and {"kind": "dense", "ff": ff}}


def _latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, base, ff):
    return {"type": "latent_attention", "mixer": dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, q_rank=q_rank, scale=scale,
                                                      rot={"dims": rot_dim, "base": base}), "mlp": ff and {"kind": "dense", "ff": ff}}


def _rec(width, blocks, conv, ff):
    return {"type": "rglru", "mixer": dict(width=width, blocks=blocks, conv=conv), "mlp": ff and {"kind": "dense", "ff": ff}}


def _config(vocab, width, eps, streams, logit_scale, pairs, layers, loop):
    c = {"architecture": ARCH, "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if streams is not None:
        c["streams"] = streams
    if logit_scale is not None:
        c["logit_scale"] = logit_scale
    if pairs:
        c["embedding"] = {"bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), pairs))}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


# width 96, three rows; the first two layers run three times; heads in groups of two, the norm in halves of the row; a
# recurrence of another width than the model without a feed-forward; a latent of sizes the general kernel takes
Z1 = _config(211, 96, 1e-5, 3, 0.7, (37, 5, 3), [
    _ssm(6, 16, 24, 3, 2, 4, 40), _rec(60, 5, 2, None), _latent(3, 20, 12, 28, 24, 20, 0.3, 1000.0, 56)], (0, 2, 3))
# width 128, two rows, no loop: a latent of tensor-core sizes first, a state of 64 shared by all heads, one norm part,
# three taps, multipliers whose products leave 32 bits
Z2 = _config(300, 128, 1e-6, 2, 3.0, (97, 900_000_007, 12_345), [
    _latent(5, 32, 32, 40, 64, 56, 0.14, 10000.0, 72), _ssm(4, 32, 64, 1, 1, 3, 80), _rec(128, 1, 4, 64)], None)
# nothing a multiple of 8: width 100, one row, no pair table; the recurrence alone runs twice; no sharing of B and C, a
# convolution of one tap, a norm in 7 parts that straddle the heads
Z3 = _config(77, 100, 1e-5, 1, 1.0, None, [
    _ssm(5, 14, 10, 5, 7, 1, 30), _rec(45, 3, 5, 28), _latent(3, 9, 6, 11, 10, 7, 0.4, 300.0, None)], (1, 2, 2))
# width 256, five rows, the whole model runs twice: a state of 128 x 64 (the sizes large models have), parts of a norm
# that are whole heads, 20 heads on one latent
Z4 = _config(160, 256, 1e-6, 5, 1.5, (61, 7, 11), [
    _ssm(4, 64, 128, 2, 4, 4, 96), _latent(20, 64, 32, 40, 64, 96, 0.12, 50000.0, 96), _rec(256, 2, 4, None)], (0, 3, 2))
# a plain residual (no 'streams'), logits as they are
Z5 = _config(90, 64, 1e-6, None, None, (11, 2, 9), [_rec(32, 1, 3, 24), _ssm(2, 24, 20, 1, 2, 2, None)], None)

TINY = {"Z1": (Z1, 41, 16), "Z2": (Z2, 42, 8), "Z3": (Z3, 43, 16), "Z4": (Z4, 44, 16), "Z5": (Z5, 45, 16)}   # config, weight seed, page size

GAIN, EMBED_GAIN, BIAS_GAIN = 5.0, 40.0, 10.0
LATENT_GAIN = 12.0                                    # queries and keys of the latent attention: a few keys carry the weight


def _shaped(key, t, rng):
    """What the tests want of a tensor, from the engine's random one."""
    last = key.split(".")[-1]
    uniform = lambda lo, hi: rng.uniform(lo, hi, size=t.shape)
    if key in ("embed", "bigram"):
        return t * EMBED_GAIN
    if last == "mix" and ".hc" in key:
        return 0.7 * np.eye(t.shape[0]) + 0.3 * rng.standard_normal(t.shape)
    if last == "in" and ".hc" in key:                 # of one sign: rows that are equal (at the start) must not cancel
        return uniform(0.2, 1.2)
    if last == "out" and ".hc" in key:
        return uniform(0.3, 1.2) * rng.choice([-1.0, 1.0, 1.0], size=t.shape)
    if last == "A_log":
        return uniform(-4.0, 1.5)
    if last == "dt_bias":
        return uniform(-3.0, 0.5)
    if last == "D":
        return uniform(-1.0, 1.0)
    if last == "lam":
        return uniform(-6.0, -2.0)
    if last == "conv":
        return rng.standard_normal(t.shape) * 0.6
    if last in ("ra", "ri"):
        return t * 2.0
    if last == "b":
        return t * BIAS_GAIN
    if last in ("uq", "uk"):
        return t * LATENT_GAIN
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
            yield key, torch.from_numpy(np.array(_shaped(key, np.asarray(value), rng), dtype=np.float32, copy=True)).to(dtype)

    write_safetensors(path, named(), metadata={"format": "pt"})
    return folder
