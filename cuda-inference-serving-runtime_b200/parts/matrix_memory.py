"""A matrix memory with exponential gates: a linear recurrence with a matrix state, a normaliser and a running maximum per head.

    q = W_q h * key_dim^-1/2, k = W_k h (heads x key_dim), v = W_v h (heads x value_dim)
    i = cap tanh((W_i h + b_i) / cap),  f = logsigmoid(cap tanh((W_f h + b_f) / cap))          one of each per head
    m' = max(f + m, i);  S <- exp(f + m - m') S + exp(i - m') k v^T;  n likewise with k alone;  m <- m'      (all start at zero)
    o = S^T q / (max(|n . q|, exp(-m)) + 1e-6);  o / sqrt(mean(o^2) + eps) per head, times a weight, times sigmoid(W_g h);  out = W_o o

A request's state is S, n and m of every head, float, one row of a state tensor of the cache manager.  One product serves
every projection that reads h (q | k | v | g | i | f, float sums).
"""
from __future__ import annotations

from typing import Dict

import torch

from ..config.spec import CacheUse
from ..ops import kernels
from .base import MIXERS, Mixer, TensorNeed, register
from .feedforward import pad_columns
from .gated_linear import pad_rows, padded, recurrent_plan_key, recurrent_step_plan, run_recurrence
from .linear import as_tensor, linear

DEFAULT_NAMES = {"q": "q", "k": "k", "v": "v", "gate": "g", "i": "i", "i_bias": "i.b", "f": "f", "f_bias": "f.b", "norm": "norm", "o": "o"}


@register(MIXERS, "matrix_memory")
class MatrixMemory(Mixer):
    """params: hidden_size, num_heads, key_dim, value_dim, gate_cap, eps (of the output norm), names."""

    graph_safe = True

    def __init__(self, spec, dtype):
        super().__init__(spec, dtype)
        self.hidden = int(spec["hidden_size"])
        self.heads, self.key_dim, self.value_dim = int(spec["num_heads"]), int(spec["key_dim"]), int(spec["value_dim"])
        self.cap, self.eps = float(spec["gate_cap"]), float(spec["eps"])
        self.names = {**DEFAULT_NAMES, **dict(spec.get("names") or {})}
        if self.key_dim > kernels.GATED_MAX_KEY_DIM:
            raise ValueError(f"key heads of {self.key_dim} are not supported: the recurrence holds up to {kernels.GATED_MAX_KEY_DIM}")
        if not self.cap > 0:
            raise ValueError("gate_cap must be positive")
        self.nk, self.nv = self.heads * self.key_dim, self.heads * self.value_dim
        self.m_offset = padded(self.nk * (self.value_dim + 1))
        self.state_size = padded(self.m_offset + self.heads)
        self.w_in = self.o = None

    def tensor_needs(self) -> Dict[str, TensorNeed]:
        n = self.names
        return {n["q"]: TensorNeed((self.nk, self.hidden)), n["k"]: TensorNeed((self.nk, self.hidden)), n["v"]: TensorNeed((self.nv, self.hidden)),
                n["gate"]: TensorNeed((self.nv, self.hidden)), n["i"]: TensorNeed((self.heads, self.hidden)),
                n["i_bias"]: TensorNeed((self.heads,), role="vector", init_mean=-1.0, init_std=0.5), n["f"]: TensorNeed((self.heads, self.hidden)),
                n["f_bias"]: TensorNeed((self.heads,), role="vector", init_mean=4.0, init_std=1.0),
                n["norm"]: TensorNeed((self.nv,), role="vector"), n["o"]: TensorNeed((self.hidden, self.nv))}

    def load(self, tensors):
        n = self.names
        self.w_in = pad_rows(torch.cat([tensors[n[key]] for key in ("q", "k", "v", "gate", "i", "f")], dim=0))
        self.i_bias, self.f_bias = tensors[n["i_bias"]].float().contiguous(), tensors[n["f_bias"]].float().contiguous()
        self.norm = tensors[n["norm"]].float().contiguous()
        self.o = pad_columns(tensors[n["o"]], 8)

    def kernel_jobs(self):
        return (kernels.gated_jobs() + kernels.recurrent_rows_jobs() + kernels.gemm_jobs(self.dtype)
                + (kernels.skinny_jobs() if self.dtype == torch.bfloat16 else []))

    def cache_use(self) -> CacheUse:
        return CacheUse("state", state_shape=(self.state_size,), state_dtype="float32")

    def plan_key(self):
        return recurrent_plan_key()

    def step_plan(self, host):
        return recurrent_step_plan(host)

    def forward(self, h, ctx, cache):
        tokens, device = ctx.n_tokens, ctx.device
        plan = ctx.plan_for(self)
        proj = linear(as_tensor(h), self.w_in)                      # float [tokens, q | k | v | gate | i | f | padding]
        gate_col = 2 * self.nk + self.nv
        per_head = lambda: torch.empty((tokens, self.heads), dtype=torch.float32, device=device)
        la, g, m, yn = per_head(), per_head(), per_head(), per_head()
        kernels.exp_gates(proj, gate_col + self.nv, gate_col + self.nv + self.heads, self.i_bias, self.f_bias, self.cap, cache.state, self.m_offset,
                          ctx.req_slot, ctx.q_start, ctx.q_len, ctx.n_requests, la, g, m, longest=plan.info["longest"])
        y = torch.empty((tokens, self.heads, self.value_dim), dtype=torch.float32, device=device)
        run_recurrence(plan, ctx, proj, 0, proj, self.nk, proj, 2 * self.nk, la, g, cache.state, y, self.heads, self.key_dim,
                       q_scale=self.key_dim ** -0.5, yn=yn)
        width = self.o.shape[1]
        make = torch.zeros if width != self.nv else torch.empty
        out = make((tokens, width), dtype=self.dtype, device=device)
        kernels.exp_output(y, yn, m, proj, gate_col, self.norm, self.eps, out)
        return linear(out, self.o)
