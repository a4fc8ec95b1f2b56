"""Hyper-connection of a sublayer: how it reads several copies of the stream and how its output
and the copies themselves go back into them.

With ``streams`` copies x_1 .. x_s of the residual stream and a sublayer f behind its norm:

    u   = sum_s read[s] x_s
    y   = f(norm(u))
    x_t <- sum_s mix[s, t] x_s + write[t] y          (all copies at once from the old ones)

The part holds the three learned tables (float32 in both precisions); an arrangement wires them
(``hyper_connected``).
"""

from __future__ import annotations

import torch

from .base import Part, TensorRequest, register_connection

MAX_STREAMS = 16


class HyperConnection(Part):
    def __init__(self, *, streams: int, read: str, mix: str, write: str):
        if not 1 <= streams <= MAX_STREAMS:
            raise ValueError(f"between 1 and {MAX_STREAMS} streams, got {streams}")
        self.streams, self.names = int(streams), (read, mix, write)
        self.read = self.mix = self.write = None

    def tensor_requests(self):
        S = self.streams
        read, mix, write = self.names
        return {read: TensorRequest((S,), "vector"), mix: TensorRequest((S, S), "float32"),
                write: TensorRequest((S,), "vector")}

    def bind(self, tensors):
        self.read, self.mix, self.write = (tensors[n].to(torch.float32) for n in self.names)


register_connection("hyper_connection", HyperConnection)
