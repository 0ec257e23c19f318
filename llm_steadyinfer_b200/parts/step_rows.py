"""What kinds of sequences a step holds, as the kernels of mixers with state are told (from the host's copy of the step's layout; a
fixed-shape step holds single rows)."""
from __future__ import annotations

import numpy as np


def portions(ctx) -> int:
    """What the step holds beside sequences of one row, as ``ops.qkv_conv`` and ``ops.conv_rows`` take it: 1 portions from position 0,
    2 portions that go on, 3 both, 0 neither."""
    if ctx.seq_cap is not None:                          # fixed shapes hold single rows
        return 0
    got = ctx.plans.get("portions")
    if got is None:
        n = np.diff(ctx.h_q_start)
        fresh = np.asarray(ctx.h_ctx_len) == n
        got = ctx.plans["portions"] = (1 if (fresh & (n > 1)).any() else 0) | (2 if (~fresh & (n > 1)).any() else 0)
    return got


def row_kinds(ctx) -> int:
    """What the step holds: 1 sequences of one row, 2 longer portions, 3 both."""
    if ctx.seq_cap is not None:                          # fixed shapes hold single rows
        return 1
    got = ctx.plans.get("row_kinds")
    if got is None:
        n = np.diff(ctx.h_q_start)
        got = ctx.plans["row_kinds"] = (1 if (n == 1).any() else 0) | (2 if (n > 1).any() else 0)
    return got
