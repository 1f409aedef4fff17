"""Choice of the kernels for a step of the gated delta rule (``parts.memory.GatedDeltaRule``), and the work lists they read.

bfloat16 with sizes the tensor-core kernels take (``csrc/delta_rule.cu``): runs of ``MIN_RUN`` tokens or more are cut into
chunks of ``CHUNK`` tokens; what does not depend on the state before a chunk is computed for all chunks at once, then one
CTA follows a run's chunks per head and columns.  Single tokens and shorter runs are walked in float32 FMAs, beside them
or alone.  Everything else (float32, other sizes) is walked.
"""

from __future__ import annotations

from typing import Dict, Optional

import numpy as np
import torch

from . import kernels

CHUNK = 64              # tokens of a chunk
MIN_RUN = 16            # tokens from which on a run is worth the tensor-core kernels' start


def plan(q_lens, mma: bool) -> Dict[str, np.ndarray]:
    """``walked``: (first row, end, entry) of the entries that are walked (empty: all of them, or with ``runs`` none).  With
    ``mma``: ``runs``, (first row, end, entry, first chunk) of the tensor-core kernels' runs, and ``chunks``, (first row, end)
    of their chunks."""
    flat = lambda a: np.asarray(a, dtype=np.int32).reshape(-1)
    ends = np.cumsum(np.asarray(q_lens, dtype=np.int64))
    spans = [(int(e - n), int(e), i) for i, (n, e) in enumerate(zip(q_lens, ends))]
    runs, chunks, walked = [], [], []
    for begin, end, entry in spans:
        if mma and end - begin >= MIN_RUN:
            runs.append((begin, end, entry, len(chunks)))
            chunks += [(c, min(c + CHUNK, end)) for c in range(begin, end, CHUNK)]
        else:
            walked.append((begin, end, entry))
    return {"runs": flat(runs), "chunks": flat(chunks), "walked": flat(walked if runs else [])}


def run(work: Dict[str, Optional[torch.Tensor]], ctx, qkv: torch.Tensor, gates: torch.Tensor, step_bias: torch.Tensor, rate_log: torch.Tensor,
        state: torch.Tensor, out_gate: torch.Tensor, norm_weight: torch.Tensor, norm_eps: float, out: torch.Tensor, heads: int, kv_heads: int, dim: int,
        vdim: int, q_scale: float, unit_eps: float) -> None:
    """``out`` [N, heads * vdim] and the requests' states from the step's rows; ``work``: the device copies of what ``plan``
    returned.  ``qkv`` are the convolution's rows q | k | v, ``gates`` float32 [N, 2 * heads], ``out_gate`` the rows of the
    output gate."""
    runs, walked = work.get("runs"), work.get("walked")
    fused = runs is None and kernels.delta_walk_finishes(vdim, dim)
    o_raw = None if fused else torch.empty((qkv.shape[0], heads * vdim), dtype=torch.float32, device=qkv.device)
    if runs is not None:
        kernels.delta_runs_mma(qkv, gates, step_bias, rate_log, state, ctx.slot_ids, o_raw, work["chunks"], runs, heads, kv_heads, dim, vdim, q_scale,
                               unit_eps)
    if runs is None or walked is not None:
        kernels.delta_walk(qkv, gates, step_bias, rate_log, state, ctx.cu_q, ctx.slot_ids, ctx.n_seqs, walked, o_raw, heads, kv_heads, dim, vdim,
                           q_scale, unit_eps, *((out_gate, norm_weight, norm_eps, out) if fused else ()))
    if not fused:
        kernels.memory_output(o_raw, None, out_gate, 0, norm_weight, norm_eps, "silu", out, heads, vdim)
