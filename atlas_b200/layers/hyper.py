"""Hyper-connected residual streams.

The residual path of a decoder is one vector per token that every sublayer adds to.  With hyper-connections it is ``S``
vectors ("streams"), kept in fp32.  A sublayer ``f`` reads one learned mix of them and all streams are rewritten from the
old ones::

    u   = sum_s read[s] * x[s]
    y   = f(norm(u))
    x'[t] = sum_s mix[s, t] * x[s] + write[t] * y

Writing streams ``t`` of one sublayer and reading the mix of the next one touch the same data, so a sublayer's write is
left pending (:class:`atlas_b200.ops.StreamDelta`) and ``ops.hyper_norm`` applies it together with the next sublayer's read
and norm in one pass.
"""
from __future__ import annotations

from typing import Optional

import torch


class HyperConnection:
    """Connection weights of one sublayer: ``read [S]``, ``write [S]``, ``mix [S, S]`` (indexed [from, to]), all fp32."""

    def __init__(self, streams: int):
        self.streams = streams
        self.read: Optional[torch.Tensor] = None
        self.write: Optional[torch.Tensor] = None
        self.mix: Optional[torch.Tensor] = None

    def load(self, read: torch.Tensor, write: torch.Tensor, mix: torch.Tensor, device) -> None:
        put = lambda t: t.to(device=device, dtype=torch.float32).contiguous()
        self.read, self.write, self.mix = put(read), put(write), put(mix)
        assert self.read.shape == self.write.shape == (self.streams,) and self.mix.shape == (self.streams, self.streams)

    def init_random(self, gen, device) -> None:
        s = self.streams
        rnd = lambda *shape: torch.randn(*shape, generator=gen, device=gen.device)
        self.load(1.0 / s + 0.1 * rnd(s), 1.0 + 0.1 * rnd(s), torch.eye(s, device=gen.device) + 0.05 * rnd(s, s), device)
