"""What the recurrent mixers share: the launch plan of a step, and the recurrence with a matrix state per head
(csrc/gated_linear.cu).

    per head:  S <- exp(la) S + g k v^T,  y = S^T q        (and n <- exp(la) n + g k, yn = n . q)

Single tokens and short portions walk a request's tokens in order; portions of CHUNKED_FROM tokens and more run the chunked
form of the same recurrence, which differs by rounding only.
"""
from __future__ import annotations

import numpy as np
import torch

from ..ops import kernels

CHUNKED_FROM = kernels.GATED_CHUNK
CONV_TILE = 16                   # tokens per tile of the short convolutions (at least taps - 1)


def conv_tile(taps: int) -> int:
    return max(CONV_TILE, taps - 1)


def recurrent_plan_key(taps: int = 1) -> tuple:
    return ("recurrence", CHUNKED_FROM, conv_tile(taps))


def recurrent_step_plan(host, taps: int = 1):
    """From the portion lengths alone: the chunks of the chunked recurrence (per chunk its request and its first token inside
    the portion, per request the index of its first chunk; portions below CHUNKED_FROM have none), and the tiles of
    neighbouring tokens of one request that the convolutions run."""
    from ..engine.batch import StepPlan

    tile = conv_tile(taps)
    chunk_req, chunk_t0, req_chunk0, tile_req, tile_t0, short = [], [], [], [], [], 0
    for r, n in enumerate(host.q_len):
        req_chunk0.append(len(chunk_req))
        for t0 in range(0, n, tile):
            tile_req.append(r)
            tile_t0.append(t0)
        if n < CHUNKED_FROM:
            short += 1
            continue
        for t0 in range(0, n, kernels.GATED_CHUNK):
            chunk_req.append(r)
            chunk_t0.append(t0)
    as_i32 = lambda values: np.asarray(values, dtype=np.int32)
    return StepPlan(arrays={"chunk_req": as_i32(chunk_req), "chunk_t0": as_i32(chunk_t0), "req_chunk0": as_i32(req_chunk0),
                            "tile_req": as_i32(tile_req), "tile_t0": as_i32(tile_t0)},
                    info={"n_chunks": len(chunk_req), "n_short": short, "n_tiles": len(tile_req), "longest": max(host.q_len, default=0)})


def conv_args(plan, ctx, taps: int) -> dict:
    """What `kernels.short_conv` takes from the step."""
    return dict(req_slot=ctx.req_slot, q_start=ctx.q_start, q_len=ctx.q_len, tile_req=plan["tile_req"], tile_t0=plan["tile_t0"],
                n_tiles=plan.info["n_tiles"], tile=conv_tile(taps))


def run_recurrence(plan, ctx, q, q_col, k, k_col, v, v_col, la, g, state, y, groups, key_dim, q_scale=1.0, yn=None):
    chunked = plan.info["n_chunks"] > 0
    chunks = (plan["chunk_req"], plan["chunk_t0"], plan["req_chunk0"], plan.info["n_chunks"]) if chunked else None
    return kernels.gated_recurrence(q, q_col, k, k_col, v, v_col, la, g, state, ctx.req_slot, ctx.q_start, ctx.q_len, ctx.n_requests, y, groups,
                                    key_dim, q_scale=q_scale, yn=yn, least=CHUNKED_FROM if chunked else 0, n_short=plan.info["n_short"],
                                    chunks=chunks)


def pad_rows(w: torch.Tensor, multiple: int = 16) -> torch.Tensor:
    """w [N, K] with zero rows appended until N is a multiple (the products' outputs then have whole 16-byte rows)."""
    extra = -w.shape[0] % multiple
    return w.contiguous() if not extra else torch.cat((w, torch.zeros((extra, w.shape[1]), dtype=w.dtype, device=w.device)), dim=0)


def padded(n: int, multiple: int = 4) -> int:
    return -(-n // multiple) * multiple
