"""A recurrent block with a real-gated linear recurrent unit: one float of state per channel, decays and inputs gated by
block-diagonal products of the convolved input.

    y = gelu(W_y h + b_y) (tanh form);  u = short causal convolution of (W_x h + b_x) per channel, with bias
    per part b of u:  r = sigmoid(R_b u_b + rb),  i = sigmoid(I_b u_b + ib)
    la = -factor * r * softplus(lam);  S <- exp(la) S + sqrt(1 - exp(2 la)) i u       (S zero before the first token)
    out = W_o (S * y)

A request's state is S and the convolution's last taps - 1 inputs (with b_x; zeros before the sequence), float, one row of a
state tensor of the cache manager.  The gates' products take u as float.  Steps of at most RGLRU_FUSED_TOKENS tokens: products,
gates, recurrence and output are one kernel.  bfloat16 steps of 128 tokens and more: the convolution also leaves u as three
bfloat16 summands, and one grouped tensor-core product over [u1 | u2 | u3] (weights repeated three times) makes the sums to
float accuracy; otherwise a row kernel makes them.  Then a scan kernel runs portions of any length.
"""
from __future__ import annotations

from typing import Dict

import numpy as np
import torch

from ..config.spec import CacheUse
from ..ops import kernels
from .base import MIXERS, Mixer, TensorNeed, register
from .feedforward import pad_columns
from .gated_linear import conv_args, pad_rows, padded, recurrent_plan_key, recurrent_step_plan
from .linear import as_tensor, linear

DEFAULT_NAMES = {"y": "y", "y_bias": "y.b", "x": "x", "x_bias": "x.b", "conv": "conv", "conv_bias": "conv.b", "r": "ra", "r_bias": "ra.b",
                 "i": "ri", "i_bias": "ri.b", "lam": "lam", "o": "o"}


@register(MIXERS, "rglru")
class RealGatedRecurrence(Mixer):
    """params: hidden_size, width, blocks, conv (taps), factor (of the decay's logarithm), names."""

    graph_safe = True

    def __init__(self, spec, dtype):
        super().__init__(spec, dtype)
        self.hidden, self.width, self.blocks = int(spec["hidden_size"]), int(spec["width"]), int(spec["blocks"])
        self.taps, self.factor = int(spec["conv"]), float(spec["factor"])
        self.names = {**DEFAULT_NAMES, **dict(spec.get("names") or {})}
        if self.width % self.blocks:
            raise ValueError("blocks must divide the width")
        if self.taps < 1:
            raise ValueError("the convolution needs at least one tap")
        self.block = self.width // self.blocks
        self.keep_offset = padded(self.width)
        self.state_size = padded(self.keep_offset + (self.taps - 1) * self.width)
        self.w_in = self.o = self.gates = self.gates3 = None

    def tensor_needs(self) -> Dict[str, TensorNeed]:
        n, w, b = self.names, self.width, self.block
        bias = lambda shape: TensorNeed(shape, role="vector", init_mean=0.0)
        return {n["y"]: TensorNeed((w, self.hidden)), n["y_bias"]: bias((w,)), n["x"]: TensorNeed((w, self.hidden)), n["x_bias"]: bias((w,)),
                n["conv"]: TensorNeed((w, self.taps), role="vector", init_mean=1.0 / self.taps, init_std=0.2), n["conv_bias"]: bias((w,)),
                n["r"]: TensorNeed((self.blocks, b, b)), n["r_bias"]: bias((self.blocks, b)), n["i"]: TensorNeed((self.blocks, b, b)),
                n["i_bias"]: bias((self.blocks, b)), n["lam"]: TensorNeed((w,), role="vector", init_mean=-4.0, init_std=1.0),
                n["o"]: TensorNeed((self.hidden, w))}

    def load(self, tensors):
        n = self.names
        self.w_in = pad_rows(torch.cat((tensors[n["y"]], tensors[n["x"]]), dim=0))
        self.y_bias, self.x_bias = tensors[n["y_bias"]].float().contiguous(), tensors[n["x_bias"]].float().contiguous()
        self.conv = tensors[n["conv"]].float().t().contiguous()          # tap by tap
        self.conv_bias = tensors[n["conv_bias"]].float().contiguous()
        self.gates = torch.cat((tensors[n["r"]], tensors[n["i"]]), dim=1).contiguous()           # [blocks, r rows | i rows, block]
        self.gate_bias = torch.cat((tensors[n["r_bias"]], tensors[n["i_bias"]]), dim=1).float().contiguous()
        if self.dtype == torch.bfloat16 and self.block % 8 == 0:
            self.gates3 = self.gates.repeat(1, 1, 3).contiguous()
        lam = tensors[n["lam"]].double()
        softplus = torch.clamp(lam, min=0.0) + torch.log1p(torch.exp(-lam.abs()))
        self.rate = (-self.factor * softplus).float().contiguous()       # what r is multiplied by: a constant of the weights
        self.o = pad_columns(tensors[n["o"]], 8)

    def kernel_jobs(self):
        return (kernels.rglru_jobs() + kernels.recurrent_rows_jobs() + kernels.gemm_jobs(self.dtype)
                + (kernels.skinny_jobs() if self.dtype == torch.bfloat16 else []))

    def cache_use(self) -> CacheUse:
        return CacheUse("state", state_shape=(self.state_size,), state_dtype="float32")

    # ---------------------------------------------------------------- the launch plan of a step
    def plan_key(self):
        return recurrent_plan_key(self.taps) + ("parts", self.blocks)

    def step_plan(self, host):
        """The shared plan, and which part each 128-row tile of the grouped product belongs to."""
        plan = recurrent_step_plan(host, self.taps)
        tiles = -(-host.n_tokens // kernels.MOE_TILE) if host.n_tokens >= kernels.TCGEN05_MIN_TOKENS else 0
        plan.arrays["part_of_tile"] = np.repeat(np.arange(self.blocks, dtype=np.int32), tiles)
        return plan

    def forward(self, h, ctx, cache):
        tokens, device = ctx.n_tokens, ctx.device
        plan = ctx.plan_for(self)
        proj = linear(as_tensor(h), self.w_in)                      # float [tokens, y | x | padding]
        rows = -(-tokens // kernels.MOE_TILE) * kernels.MOE_TILE
        tensor_cores = self.gates3 is not None and tokens >= kernels.TCGEN05_MIN_TOKENS
        u = torch.empty((tokens, self.width), dtype=torch.float32, device=device)
        # rows behind the step's tokens are never read back: a row of the product depends on its own row alone
        split = torch.empty((self.blocks, rows, 3, self.block), dtype=torch.bfloat16, device=device) if tensor_cores else None
        kernels.short_conv(proj, self.width, self.conv, self.conv_bias, cache.state, self.keep_offset, **conv_args(plan, ctx, self.taps), out=u,
                           silu=False, in_bias=self.x_bias, split=split)
        wide = self.o.shape[1]
        make = torch.zeros if wide != self.width else torch.empty
        out = make((tokens, wide), dtype=self.dtype, device=device)
        if tokens <= kernels.RGLRU_FUSED_TOKENS:
            kernels.rglru_step(u, self.gates, self.gate_bias, self.rate, cache.state, 0, ctx.token_req, ctx.req_slot, ctx.q_start, ctx.q_len, proj, 0,
                               self.y_bias, out)
            return linear(out, self.o)
        pre = torch.empty((self.blocks, rows, 2 * self.block), dtype=torch.float32, device=device)
        bias = None
        if tensor_cores:
            kernels.gemm_tcgen05_grouped(split.view(self.blocks * rows, 3 * self.block), self.gates3, pre.view(self.blocks * rows, 2 * self.block),
                                         plan["part_of_tile"], rows_in_use=self.blocks * tokens)
            bias = self.gate_bias
        else:
            kernels.rglru_gates(u, self.gates, self.gate_bias, pre)
        kernels.rglru_scan(pre, bias, u, self.rate, cache.state, 0, ctx.req_slot, ctx.q_start, ctx.q_len, ctx.n_requests, proj, 0, self.y_bias, out,
                           longest=plan.info["longest"])
        return linear(out, self.o)
