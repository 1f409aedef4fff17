"""Choice of the kernels for a step of the state space (``parts.memory.Mamba2``), and the work lists they read.

bfloat16 with sizes the tensor-core kernel takes (``csrc/state_space.cu``): runs of ``MIN_RUN`` tokens or more go there, one
CTA after a request's whole run per head and columns; single tokens and shorter runs are walked in float32 FMAs
(``csrc/gated_memory.cu``), beside them or alone.  Everything else (float32, other sizes) is walked, long runs in
chunks in parallel (``kernels.plan_memory``).
"""

from __future__ import annotations

from typing import Dict, Optional

import numpy as np
import torch

from . import kernels

MIN_RUN = 16            # tokens from which on a run is worth the tensor-core kernel's start


def plan(q_lens, mma: bool) -> Dict[str, np.ndarray]:
    """``first``, ``runs``, ``second``: the chunked walk's lists (all empty: every entry is walked whole).  With ``mma``:
    ``tensor_runs``, (first row, end, entry) of the runs of the tensor-core kernel, and ``second``, the other entries of
    such a step."""
    flat = lambda a: np.asarray(a, dtype=np.int32).reshape(-1)
    if not mma:
        first, runs, second = kernels.plan_memory(q_lens)
        return {"first": flat(first), "runs": flat(runs), "second": flat(second)}
    ends = np.cumsum(np.asarray(q_lens, dtype=np.int64))
    spans = [(int(e - n), int(e), i) for i, (n, e) in enumerate(zip(q_lens, ends))]
    long = [s for s in spans if s[1] - s[0] >= MIN_RUN]
    short = [(b, e, i, 0, 0) for b, e, i in spans if e - b < MIN_RUN] if long else []
    return {"tensor_runs": flat(long), "second": flat(short)}


def run(work: Dict[str, Optional[torch.Tensor]], ctx, x: torch.Tensor, q_off: int, k_off: int, v_off: int, steps: torch.Tensor, step_bias: torch.Tensor,
        rate_log: torch.Tensor, state: torch.Tensor, o_raw: torch.Tensor, heads: int, groups: int, dim: int, vdim: int) -> None:
    """``o_raw`` and the requests' states from the step's rows; ``work``: the device copies of what ``plan`` returned."""
    runs = work.get("tensor_runs")
    if runs is not None:
        kernels.state_space_mma(x, q_off, k_off, v_off, steps, step_bias, rate_log, state, ctx.slot_ids, o_raw, heads, groups, dim, vdim, runs)
        if work.get("second") is None:
            return
    kernels.ssd_scan(x, q_off, k_off, v_off, steps, step_bias, rate_log, state, ctx.cu_q, ctx.slot_ids, o_raw, ctx.n_seqs, heads, groups, dim, vdim,
                     work.get("first"), work.get("runs"), work.get("second"))
