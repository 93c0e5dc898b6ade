"""Sub-blocks with a norm after, and most with one before: x <- x + s * norm_out(sub_block(norm_in(x))), s one factor per
channel; without a norm before, the sub-block reads the stream itself.

The whole seam between two sub-blocks is one kernel (`kernels.post_norm`): a sub-block's output stays pending in the stream
object, with its output norm, until the next sub-block (or the final norm) asks for its normed input; the kernel then norms the
output, adds it to the stream, adds what comes ahead of the next sub-block (a per-pass vector, the embedding output again),
and norms the sum.  An output norm's weight and the layer scale enter as one float vector (the product of two bfloat16
numbers is exact in float).  The stream and every sum are float.
"""
from __future__ import annotations

from typing import Optional

import torch

from ..config.spec import LayerSpec
from ..ops import kernels
from .base import ARRANGEMENTS, FEED_FORWARDS, MIXERS, NORMS, STREAMS, build_part, register
from .block import ChannelScale


def float_weight(norm) -> torch.Tensor:
    """The norm's weight as a float vector, formed once."""
    w = getattr(norm, "_float_weight", None)
    if w is None:
        w = norm._float_weight = norm.weight.float().contiguous()
    return w


@register(STREAMS, "post_norm")
class PostNormStream:
    """The float residual stream x [tokens, hidden], an output not added to it yet (with the norm it is added through), and
    what else is to be added before the next sub-block reads it.  params of the spec: keep_embedding (bool: the embedding
    output is needed again later, so the stream leaves it as it is and continues in a buffer of its own)."""

    def __init__(self, embedded: torch.Tensor, spec):
        self.x = embedded
        self.embedded = embedded if spec.get("keep_embedding", False) else None
        self.pending: Optional[torch.Tensor] = None
        self.pending_norm = None                     # (float weight with the layer scale, eps, kind)
        self.extra: Optional[torch.Tensor] = None    # a tensor like x
        self.vector: Optional[torch.Tensor] = None   # one value per channel

    def write(self, y: torch.Tensor, norm: tuple) -> None:
        self.pending, self.pending_norm = y, norm

    def add_embedding(self) -> None:
        """The embedding output is added to the stream before the next sub-block reads it."""
        if self.embedded is None:
            raise ValueError("the stream was not told to keep the embedding output")
        self.extra = self.embedded

    def add_vector(self, vector: torch.Tensor) -> None:
        self.vector = vector

    def _pending(self) -> dict:
        if self.pending is None:
            return {}
        weight, eps, kind = self.pending_norm
        return {"y": self.pending, "post_w": weight, "post_eps": eps, "post_kind": kind}

    def read(self, norm, dtype: torch.dtype, rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        """Bring everything pending into the stream and return its norm in `dtype` (norm None: the stream itself); `rows`
        picks tokens, and the stream is then left as it is."""
        n = self.x.shape[0] if rows is None else rows.numel()
        as_it_is = norm is None and rows is None and dtype == self.x.dtype      # no copy: what reads it is done before the next write
        h = None if as_it_is else torch.empty((n, self.x.shape[1]), dtype=dtype, device=self.x.device)
        changed = self.pending is not None or self.extra is not None or self.vector is not None
        x_out = None
        if rows is None and changed:
            x_out = torch.empty_like(self.x) if self.x is self.embedded else self.x
        if x_out is not None or h is not None:
            pre = {"pre_kind": "none"} if norm is None else {"pre_w": float_weight(norm), "pre_eps": norm.eps, "pre_kind": norm.kind}
            kernels.post_norm(self.x, **self._pending(), extra=self.extra, vector=self.vector, x_out=x_out, **pre, h=h, rows=rows)
        if x_out is not None:
            self.x = x_out
            self.pending = self.pending_norm = self.extra = self.vector = None
        return self.x if as_it_is else h

    def finish(self, norm, dtype: torch.dtype, rows: torch.Tensor) -> torch.Tensor:
        """The model's last step: the normed stream at the wanted rows."""
        return self.read(norm, dtype, rows=rows)

    def total(self) -> torch.Tensor:
        """The stream with the pending output in it, as a new tensor; the stream object stays as it was."""
        x = torch.empty_like(self.x)
        kernels.post_norm(self.x, **self._pending(), x_out=x)
        return x


@register(ARRANGEMENTS, "pre_post_norm_scaled")
class PrePostNormBlock:
    """x += s1 * norm1b(mixer(norm1(x))); x += s2 * norm2b(feed_forward(norm2(x))); the feed-forward half may be absent, and so
    may the norms ahead (`mixer_norm`, `feed_forward_norm` None: the sub-block reads the stream itself).  The
    layer's `extras` give the output norms ("mixer_out_norm", "feed_forward_out_norm") and, where a layer has them, the
    scales ("mixer_scale", "feed_forward_scale": `ChannelScale`).  Norms name their kind (layer_norm, rms_norm)."""

    def __init__(self, spec: LayerSpec, dtype: torch.dtype):
        self.spec = spec
        self.dtype = dtype
        norm = lambda part: None if part is None else build_part(NORMS, part, dtype, "norm")
        scale = lambda name: ChannelScale(spec.extras[name], dtype) if name in spec.extras else None
        self.mixer_norm, self.mixer_out_norm = norm(spec.mixer_norm), norm(spec.extras["mixer_out_norm"])
        self.mixer = build_part(MIXERS, spec.mixer, dtype, "mixer")
        self.mixer_scale = scale("mixer_scale")
        self.feed_forward = self.feed_forward_norm = self.feed_forward_out_norm = self.feed_forward_scale = None
        if spec.feed_forward is not None:
            self.feed_forward_norm, self.feed_forward_out_norm = norm(spec.feed_forward_norm), norm(spec.extras["feed_forward_out_norm"])
            self.feed_forward = build_part(FEED_FORWARDS, spec.feed_forward, dtype, "feed-forward")
            self.feed_forward_scale = scale("feed_forward_scale")
        for part in (self.mixer_norm, self.mixer_out_norm, self.feed_forward_norm, self.feed_forward_out_norm):
            if part is not None and not hasattr(part, "kind"):
                raise ValueError("this arrangement takes norms that name their kind (layer_norm, rms_norm)")
        self._out = {}

    def parts(self):
        slots = ("mixer_norm", "mixer", "mixer_out_norm", "mixer_scale", "feed_forward_norm", "feed_forward", "feed_forward_out_norm",
                 "feed_forward_scale")
        return {slot: getattr(self, slot) for slot in slots if getattr(self, slot) is not None}

    def kernel_jobs(self):
        return kernels.post_norm_jobs()

    def _out_norm(self, norm, scale) -> tuple:
        found = self._out.get(id(norm))
        if found is None:
            w = float_weight(norm)
            found = self._out[id(norm)] = ((w * scale.weight).contiguous() if scale is not None else w, norm.eps, norm.kind)
        return found

    def forward(self, stream: PostNormStream, ctx, cache) -> None:
        y = self.mixer.forward(stream.read(self.mixer_norm, self.dtype), ctx, cache)
        stream.write(y, self._out_norm(self.mixer_out_norm, self.mixer_scale))
        if self.feed_forward is not None:
            y = self.feed_forward.forward(stream.read(self.feed_forward_norm, self.dtype), ctx)
            stream.write(y, self._out_norm(self.feed_forward_out_norm, self.feed_forward_scale))
