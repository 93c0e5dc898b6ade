"""The selective state-space mixer in its matrix form (state-space duality): a decaying matrix state per head.

    z | x | B | C | dt = W_in h          z, x: heads x value_dim;  B, C: groups x state_dim;  dt: heads
    x, B, C <- silu(short causal convolution over time per channel, with bias; zeros before the sequence)
    dt <- softplus(dt + dt_bias)
    per head (its B and C are group head // (heads / groups)):  S <- exp(-exp(A_log) dt) S + dt B x^T,  y = S^T C + D x
    v = y * silu(z), each of norm_groups equal parts of the row divided by its root mean square, times a weight;  out = W_o v

A request's state is S of every head and the convolution's last taps - 1 inputs, float, one row of a state tensor of the
cache manager.  The mixer can also be one side of a pair that share their products (parts/parallel.py): `in_rows`, `mix`.
"""
from __future__ import annotations

from typing import Dict, Optional

import torch

from ..config.spec import CacheUse
from ..ops import kernels
from .base import MIXERS, Mixer, TensorNeed, register
from .feedforward import pad_columns
from .gated_linear import conv_args, pad_rows, padded, recurrent_plan_key, recurrent_step_plan, run_recurrence
from .linear import as_tensor, linear

DEFAULT_NAMES = {"in": "in", "conv": "conv", "conv_bias": "conv.b", "dt_bias": "dt_bias", "a_log": "A_log", "d": "D", "norm": "norm", "o": "o"}


@register(MIXERS, "state_space")
class StateSpace(Mixer):
    """params: hidden_size, num_heads, value_dim, state_dim, groups, conv (taps), norm_groups, eps (of the output norm), names."""

    # forward reads the step through device tensors only; captured steps' warm-up runs put the state back (engine/graph.py)
    graph_safe = True

    def __init__(self, spec, dtype):
        super().__init__(spec, dtype)
        self.hidden = int(spec["hidden_size"])
        self.heads, self.value_dim = int(spec["num_heads"]), int(spec["value_dim"])
        self.state_dim, self.groups = int(spec["state_dim"]), int(spec["groups"])
        self.taps, self.norm_groups = int(spec["conv"]), int(spec["norm_groups"])
        self.eps = float(spec["eps"])
        self.names = {**DEFAULT_NAMES, **dict(spec.get("names") or {})}
        self.inner = self.heads * self.value_dim
        if self.heads % self.groups or self.inner % self.norm_groups:
            raise ValueError("groups must divide the heads, norm_groups the row of all heads")
        if self.state_dim > kernels.GATED_MAX_KEY_DIM:
            raise ValueError(f"a state of {self.state_dim} rows is not supported: the recurrence holds up to {kernels.GATED_MAX_KEY_DIM}")
        if self.taps < 1:
            raise ValueError("the convolution needs at least one tap")
        self.channels = self.inner + 2 * self.groups * self.state_dim
        self.keep_offset = padded(self.heads * self.state_dim * self.value_dim)
        self.state_size = padded(self.keep_offset + (self.taps - 1) * self.channels)
        self.in_rows = self.w_in = self.out_rows = self.o = None

    def tensor_needs(self) -> Dict[str, TensorNeed]:
        n = self.names
        return {n["in"]: TensorNeed((self.inner + self.channels + self.heads, self.hidden)),
                n["conv"]: TensorNeed((self.channels, self.taps), role="vector", init_mean=1.0 / self.taps, init_std=0.2),
                n["conv_bias"]: TensorNeed((self.channels,), role="vector", init_mean=0.0),
                n["dt_bias"]: TensorNeed((self.heads,), role="vector", init_mean=-3.0, init_std=1.0),
                n["a_log"]: TensorNeed((self.heads,), role="vector", init_mean=1.0, init_std=0.5),
                n["d"]: TensorNeed((self.heads,), role="vector"), n["norm"]: TensorNeed((self.inner,), role="vector"),
                n["o"]: TensorNeed((self.hidden, self.inner))}

    def load(self, tensors):
        n = self.names
        self.in_rows = tensors[n["in"]]
        self.conv = tensors[n["conv"]].float().t().contiguous()          # tap by tap: neighbouring channels are neighbours in memory
        self.conv_bias, self.dt_bias = tensors[n["conv_bias"]].float().contiguous(), tensors[n["dt_bias"]].float().contiguous()
        self.a_log, self.d = tensors[n["a_log"]].float().contiguous(), tensors[n["d"]].float().contiguous()
        self.norm = tensors[n["norm"]].float().contiguous()
        self.out_rows = tensors[n["o"]]

    def kernel_jobs(self):
        return (kernels.gated_jobs() + kernels.recurrent_rows_jobs() + kernels.gemm_jobs(self.dtype)
                + (kernels.skinny_jobs() if self.dtype == torch.bfloat16 else []))

    def cache_use(self) -> CacheUse:
        return CacheUse("state", state_shape=(self.state_size,), state_dtype="float32")

    def plan_key(self):
        return recurrent_plan_key(self.taps)

    def step_plan(self, host):
        return recurrent_step_plan(host, self.taps)

    def mix(self, proj: torch.Tensor, col: int, ctx, state: torch.Tensor, width: int, lead: Optional[torch.Tensor] = None,
            scale: float = 1.0) -> torch.Tensor:
        """From the projection of h (this mixer's columns begin at `col`) to the operand of an output projection [tokens,
        width]: `lead` (another operand, copied) | scale * v | zeros."""
        tokens, device = ctx.n_tokens, ctx.device
        plan = ctx.plan_for(self)
        conv = torch.empty((tokens, self.channels), dtype=torch.float32, device=device)
        la = torch.empty((tokens, self.heads), dtype=torch.float32, device=device)
        dt = torch.empty((tokens, self.heads), dtype=torch.float32, device=device)
        kernels.short_conv(proj, col + self.inner, self.conv, self.conv_bias, state, self.keep_offset, **conv_args(plan, ctx, self.taps), out=conv,
                           silu=True, steps=(col + self.inner + self.channels, self.dt_bias, self.a_log, la, dt))
        y = torch.empty((tokens, self.heads, self.value_dim), dtype=torch.float32, device=device)
        b_col, c_col = self.inner, self.inner + self.groups * self.state_dim
        run_recurrence(plan, ctx, conv, c_col, conv, b_col, conv, 0, la, dt, state, y, self.groups, self.state_dim)
        out = torch.empty((tokens, width), dtype=self.dtype, device=device)
        return kernels.ssd_output(y, conv, self.d, proj, col, self.norm, self.eps, out, parts=self.norm_groups, scale=scale, lead=lead)

    def forward(self, h, ctx, cache):
        if self.w_in is None:
            self.w_in, self.o = pad_rows(self.in_rows), pad_columns(self.out_rows, 8)
        operand = self.mix(linear(as_tensor(h), self.w_in), 0, ctx, cache.state, self.o.shape[1])
        return linear(operand, self.o)
