"""Two mixers side by side that read the same input: out = left_scale * left(h) + right_scale * right(h).

Left is a softmax attention (`windowed_attention`), right a state-space mixer (`state_space`); their tensors lie under
"left." and "right.".  Both input projections are one product, and so are both output projections: the right side's
operand, scaled by right_scale / left_scale before its one rounding, stands behind the left side's, and the product of
[left | right] with [W_o left | W_o right] is multiplied by left_scale.  The left side's keys and values are pages of the
cache manager, the right side's state is the run entry's side state.
"""
from __future__ import annotations

from typing import Dict, Optional

import torch

from ..config.spec import CacheUse
from ..ops import kernels
from .base import MIXERS, Mixer, TensorNeed, build_part, register
from .feedforward import pad_columns
from .gated_linear import pad_rows
from .linear import as_tensor, linear, linear_times


@register(MIXERS, "parallel")
class Parallel(Mixer):
    """params: left, right (PartSpecs of the two mixers), left_scale, right_scale."""

    def __init__(self, spec, dtype):
        super().__init__(spec, dtype)
        self.left = build_part(MIXERS, spec["left"], dtype, "mixer")
        self.right = build_part(MIXERS, spec["right"], dtype, "mixer")
        for side, need in ((self.left, "attend"), (self.right, "mix")):
            if not hasattr(side, need):
                raise ValueError(f"a mixer of kind {side.spec.kind!r} cannot stand on this side of a pair")
        left_scale, right_scale = float(spec["left_scale"]), float(spec["right_scale"])
        # out = outer * (W_left (inner_left * a_left) + W_right (inner_right * a_right))
        self.outer, self.inner_right = (left_scale, right_scale / left_scale) if left_scale != 0.0 else (right_scale, 1.0)
        self.left_counts = left_scale != 0.0
        self.graph_safe = self.left.graph_safe and self.right.graph_safe
        self.w_in = self.o = None

    def tensor_needs(self) -> Dict[str, TensorNeed]:
        return {f"{side}.{name}": need for side, part in (("left", self.left), ("right", self.right)) for name, need in part.tensor_needs().items()}

    def load(self, tensors):
        for side, part in (("left", self.left), ("right", self.right)):
            part.load({name[len(side) + 1:]: t for name, t in tensors.items() if name.startswith(side + ".")})
        self.right_col = self.left.w_in.shape[0]
        self.w_in = pad_rows(torch.cat((self.left.w_in, self.right.in_rows), dim=0))
        left_o = self.left.o if self.left_counts else torch.zeros_like(self.left.o)
        self.o = pad_columns(torch.cat((left_o, self.right.out_rows), dim=1), 8)
        # the sides' own copies are not used: their products are these two
        self.left.w_in = self.left.o = self.right.in_rows = self.right.out_rows = None

    def kernel_jobs(self):
        return self.left.kernel_jobs() + self.right.kernel_jobs()

    def cache_use(self) -> CacheUse:
        return self.left.cache_use()

    def side_state(self) -> Optional[CacheUse]:
        return self.right.cache_use()

    def planning_parts(self) -> list:
        return [self.left, self.right]

    def begin_step(self, ctx) -> None:
        self.left.begin_step(ctx)
        self.right.begin_step(ctx)

    def forward(self, h, ctx, cache):
        proj = linear(as_tensor(h), self.w_in)
        lead = self.left.attend(proj, ctx, cache)
        operand = self.right.mix(proj, self.right_col, ctx, cache.state, self.o.shape[1], lead=lead, scale=self.inner_right)
        return linear_times(operand, self.o, self.outer)
