"""Mixers side by side: several mixers read the same input and their results make up one update.

``parallel_mixers``: each result is RMS-normed over the model width with a plain weight of its own (eps inside the
root), and the layer's update is the mean of the normed results.

``branches``: (name, ``PartSpec``) pairs; a branch's tensors live under ``<name>.`` and its output weight is
``<name>.out``.  Every branch is an ordinary registered mixer, built here with the layer's position encoding; at most
one of them may ask for pages of keys and values and at most one for a per-request state, which the stop's cache and
state then serve.  The norms and the mean are one kernel.

``summed_mixers``: the update is the sum of the results, each times a constant.  The branches' first products are one
product over all their rows and their last products one product over their columns side by side.
"""

from __future__ import annotations

from typing import Sequence, Tuple

import torch

from ..config.spec import PartSpec
from ..ops import kernels
from ..ops.linear import DeferredNorm, Linear
from . import base
from .base import Mixer, TensorSpec, register_mixer


@register_mixer("parallel_mixers")
class ParallelMixers(Mixer):
    def __init__(self, hidden_size: int, branches: Sequence[Tuple[str, PartSpec]], norm_eps: float, position=None):
        self.hidden_size, self.norm_eps = int(hidden_size), float(norm_eps)
        if not 1 <= len(branches) <= 4:
            raise ValueError(f"one to four mixers run side by side, got {len(branches)}")
        self.names = [name for name, _ in branches]
        if len(set(self.names)) != len(self.names):
            raise ValueError(f"the branches need names of their own, got {self.names}")
        self.branches = [base.build_part(base.MIXERS, spec, "mixer", position=position) for _, spec in branches]
        if sum(b.cache_need() is not None for b in self.branches) > 1 or sum(b.state_need() is not None for b in self.branches) > 1:
            raise ValueError("mixers side by side: at most one may keep pages of keys and values, at most one a state")
        self.graph_safe = all(getattr(b, "graph_safe", False) for b in self.branches)
        self.out_weights = None

    def sub_parts(self):
        return list(self.branches)

    def tensor_specs(self):
        specs = []
        for name, b in zip(self.names, self.branches):
            specs += [TensorSpec(f"{name}.{ts.name}", ts.shape, ts.init, ts.optional) for ts in b.tensor_specs()]
        specs += [TensorSpec(f"{name}.out", (self.hidden_size,), "norm") for name in self.names]
        return tuple(specs)

    def cache_need(self):
        return next((b.cache_need() for b in self.branches if b.cache_need() is not None), None)

    def state_need(self):
        return next((b.state_need() for b in self.branches if b.state_need() is not None), None)

    def load(self, tensors, device, dtype):
        for name, b in zip(self.names, self.branches):
            own = {k[len(name) + 1:]: t for k, t in tensors.items() if k.startswith(name + ".") and k != f"{name}.out"}
            b.load(own, device, dtype)
        self.out_weights = [tensors[f"{name}.out"].to(device=device, dtype=torch.float32).contiguous() for name in self.names]

    def forward(self, ctx, h, stop):
        results = [b.forward(ctx, h, stop) for b in self.branches]
        out = torch.empty_like(results[0])
        kernels.branch_mean_norm(results, self.out_weights, self.norm_eps, out)
        return out


@register_mixer("summed_mixers")
class SummedMixers(Mixer):
    """``branches``: (name, ``PartSpec``, constant) triples; a branch's tensors live under ``<name>.``.  Every branch is a
    registered mixer that offers its products apart (``Mixer.products``); at most one may ask for pages and at most one
    for a per-request state.

    A constant that is not 1 rides in a float32 weight that its branch multiplies its heads with (``scale_heads``), or else
    in the branch's columns of the last product; a factor that all branches share is better left to the scale of the
    update (``channel_scale``)."""

    accepts_residual = True          # the last product can add into the residual stream itself
    accepts_scaled_residual = True
    accepts_deferred_norm = True

    def __init__(self, hidden_size: int, branches: Sequence[Tuple[str, PartSpec, float]], position=None):
        self.hidden_size = int(hidden_size)
        self.names, self.scales = [b[0] for b in branches], [float(b[2]) for b in branches]
        if len(branches) < 1 or len(set(self.names)) != len(self.names):
            raise ValueError(f"mixers side by side need names of their own, got {self.names}")
        self.branches = [base.build_part(base.MIXERS, b[1], "mixer", position=position) for b in branches]
        if sum(b.cache_need() is not None for b in self.branches) > 1 or sum(b.state_need() is not None for b in self.branches) > 1:
            raise ValueError("mixers side by side: at most one may keep pages of keys and values, at most one a state")
        self.graph_safe = all(getattr(b, "graph_safe", False) for b in self.branches)
        self.in_proj = self.out_proj = None

    def sub_parts(self):
        return list(self.branches)

    def tensor_specs(self):
        return tuple(TensorSpec(f"{name}.{ts.name}", ts.shape, ts.init, ts.optional) for name, b in zip(self.names, self.branches) for ts in b.tensor_specs())

    def cache_need(self):
        return next((b.cache_need() for b in self.branches if b.cache_need() is not None), None)

    def state_need(self):
        return next((b.state_need() for b in self.branches if b.state_need() is not None), None)

    def load(self, tensors, device, dtype):
        ins, outs = [], []
        for name, b, scale in zip(self.names, self.branches, self.scales):
            b.load({k[len(name) + 1:]: t for k, t in tensors.items() if k.startswith(name + ".")}, device, dtype)
            first, last = b.products()
            if last.bias is not None:
                raise ValueError("a mixer beside others has no bias behind its last product")
            w = last.weight
            if scale != 1.0:
                if hasattr(b, "scale_heads"):
                    b.scale_heads(scale)
                else:
                    w = (w.float() * scale).to(w.dtype)
            ins.append(first)
            outs.append(w)
        self.in_cols, self.out_cols = [l.out_features for l in ins], [w.shape[1] for w in outs]
        bias = None
        if any(l.bias is not None for l in ins):
            bias = torch.cat([l.bias if l.bias is not None else torch.zeros(l.out_features, dtype=torch.float32, device=device) for l in ins])
        self.in_proj = Linear(torch.cat([l.weight for l in ins], dim=0).contiguous(), bias)
        self.out_proj = Linear(torch.cat(outs, dim=1).contiguous())
        for b in self.branches:
            b.drop_products()            # their rows and columns live on in the shared products

    def forward(self, ctx, h, stop, residual=None, residual_scale=None):
        if isinstance(h, DeferredNorm) and not kernels.gemm_skinny_norm_supports(h.x, self.in_proj.weight):
            h = h.materialize()
        x = self.in_proj(h)
        sides = [b.side_products(ctx, h) for b in self.branches]
        heads = torch.empty((x.shape[0], self.out_proj.in_features), dtype=x.dtype, device=x.device)
        c = k = 0
        for b, side, cols, width in zip(self.branches, sides, self.in_cols, self.out_cols):
            b.between(ctx, x[:, c:c + cols], stop, side=side, out=heads[:, k:k + width])
            c, k = c + cols, k + width
        return self.out_proj(heads, residual=residual, residual_scale=residual_scale)
