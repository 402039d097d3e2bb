"""Hyper-connections: instead of one residual stream a model keeps S of them, and every sublayer has learned numbers that say
how it reads and writes them,

    u = sum_s in[s] x_s        y = sublayer(norm(u))        x_t <- sum_s mix[s, t] x_s + out[t] y   (all t from the old x)

(mix is indexed from, to).  All streams start as the embedding's output; the model's last norm reads their sum.

The streams are float32, [T, S, width]; until the first sublayer's output is written they are one row and kept as one.
Between two sublayers one kernel writes the first one's output, forms what the second one reads and norms it
(RMSNorm.read_streams, csrc/hyper_streams.cu): each stream is read once and written once a sublayer.  Experts leave their
weighted sum to that kernel."""
from __future__ import annotations

from typing import Callable, Optional

import torch

from .. import ops
from .base import Block, FeedForward, Mixer, Norm, ParamSpec, Part, Runtime, StepContext, StreamUpdate


class HyperConnection(Part):
    """The numbers of one sublayer: tensors <prefix>.in [S], <prefix>.out [S], <prefix>.mix [S, S]."""
    recordable = True

    def __init__(self, rt: Runtime, prefix: str, streams: int):
        self.rt, self.prefix, self.streams = rt, prefix, int(streams)
        self.read: torch.Tensor | None = None           # float32 on the device
        self.write: torch.Tensor | None = None
        self.mix: torch.Tensor | None = None

    def param_specs(self) -> list[ParamSpec]:
        s, p = self.streams, self.prefix
        return [ParamSpec(f"{p}.in", (s,), "ones"), ParamSpec(f"{p}.out", (s,), "ones"), ParamSpec(f"{p}.mix", (s, s), "ones")]

    def bind(self, get: Callable[[str], torch.Tensor]) -> None:
        f = lambda n: get(f"{self.prefix}.{n}").to(torch.float32).contiguous()
        self.read, self.write, self.mix = f("in"), f("out"), f("mix")


class HyperConnectionBlock(Block):
    """A mixer and (optionally) a feed-forward on S residual streams, each with a norm in front and a HyperConnection.  The
    first block of a model finds one row for all streams; `residual` is [T, S, width] from the second sublayer on."""
    recordable = True
    takes_streams = True

    def __init__(self, mixer: Mixer, feed_forward: Optional[FeedForward], mixer_norm: Norm, ffn_norm: Optional[Norm],
                 mixer_connection: HyperConnection, ffn_connection: Optional[HyperConnection], act_dtype: torch.dtype):
        if (feed_forward is None) != (ffn_norm is None) or (feed_forward is None) != (ffn_connection is None):
            raise ValueError("a feed-forward, its norm and its connection come together")
        if not all(n is None or n.takes_streams for n in (mixer_norm, ffn_norm)):
            raise ValueError("the norms in front of the sublayers must read streams (Norm.takes_streams)")
        self.mixer, self.feed_forward = mixer, feed_forward
        self.mixer_norm, self.ffn_norm = mixer_norm, ffn_norm
        self.mixer_connection, self.ffn_connection = mixer_connection, ffn_connection
        self.act_dtype = act_dtype
        self._rt = mixer_connection.rt

    def children(self) -> list[Part]:
        return [p for p in (self.mixer_norm, self.mixer_connection, self.mixer, self.ffn_norm, self.ffn_connection, self.feed_forward)
                if p is not None]

    def forward(self, residual: torch.Tensor, delta, step: StepContext, cache, write_cache: bool = True):
        c = self.mixer_connection
        if torch.is_tensor(delta):                      # a block of another kind left something to be added to its one stream
            ops.add_into(residual, delta, self._rt.stream)
        update = delta if isinstance(delta, StreamUpdate) else None
        residual, h = self.mixer_norm.read_streams(residual, update, c.read, c.streams, self.act_dtype)
        update = StreamUpdate(self.mixer.forward(h, step, cache, write_cache), c)
        if self.feed_forward is None:
            return residual, update
        c = self.ffn_connection
        residual, h = self.ffn_norm.read_streams(residual, update, c.read, c.streams, self.act_dtype)
        y = self.feed_forward.forward(h, step, unsummed=True) if self.feed_forward.offers_unsummed else self.feed_forward.forward(h, step)
        return residual, StreamUpdate(y, c)
