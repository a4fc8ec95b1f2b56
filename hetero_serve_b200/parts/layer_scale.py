"""A learned factor per channel for a sublayer's output, times a constant of the model."""

from __future__ import annotations

from .base import Scale, TensorRequest, register_scale


class ChannelScale(Scale):
    """``factor = weight * multiplier``, float32 in both precisions."""

    def __init__(self, *, width: int, weight: str, multiplier: float = 1.0):
        self.width, self.name, self.multiplier = width, weight, float(multiplier)

    def tensor_requests(self):
        return {self.name: TensorRequest((self.width,), "vector")}

    def bind(self, tensors):
        self.factor = (tensors[self.name] * self.multiplier).contiguous()


register_scale("channel_scale", ChannelScale)
