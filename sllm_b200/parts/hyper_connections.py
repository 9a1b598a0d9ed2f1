"""A residual stream that is several copies, which every sublayer reads as one weighted sum and mixes anew:

    u = sum_s into_s x_s;    y = sublayer(norm(u));    x_t <- sum_s mix_(s, t) x_s + mult out_t y

(all new streams from the old ones), once around the mixer and once around the feed-forward.  What leaves the model is the sum of
the streams.  The parts: the three small tensors of one sublayer, and the block that arranges them.  Each takes its sizes and
constants as parameters; none names a model.

The streams of a token lie side by side, float32 ``[T, streams, width]``.  A sublayer's output joins all of them and is read, with
all of them, by the next sublayer's sum, so one kernel per sublayer does both (`ops.streams_step`): it brings the term in, mixes,
writes the streams, sums them for the next reader and norms the sum.  A block therefore hands its last term on un-added
(`StreamsPending`); the next block's first kernel takes it in, or, at the model's end, `read_streams`, which computes the wanted
rows alone and writes no stream.
"""

from __future__ import annotations

from dataclasses import dataclass

import torch

from .. import ops
from .base import BLOCKS, SHIFTS, Part, TensorSpec


@SHIFTS.register("hyper_connection")
class HyperConnection(Part):
    """One sublayer's weights of the streams: ``in`` [streams] (what the sublayer reads), ``mix`` [streams, streams] (from, to) and
    ``out`` [streams] (each stream's share of the sublayer's term).  Parameters: ``streams``; ``mult`` (1 unless given), a factor on
    every term."""

    def __init__(self, params, **kw):
        super().__init__(params, **kw)
        self.streams = int(params["streams"])
        self.mult = float(params.get("mult", 1.0))
        if not 1 <= self.streams <= ops.MAX_STREAMS:
            raise ValueError(f"hyper_connection: {self.streams} streams are outside 1..{ops.MAX_STREAMS}, what the kernel takes")
        self.into = self.mix = self.share = None

    def tensor_specs(self):
        s = self.streams
        return [TensorSpec("in", (s,), role="share"), TensorSpec("out", (s,), role="gain"), TensorSpec("mix", (s, s), role="identity")]

    def bind(self, fetch):
        self.into, self.mix = self._f32(fetch("in")), self._f32(fetch("mix"))
        self.share = self._f32(fetch("out").to(torch.float32) * self.mult)

    def weight_bytes(self):
        return 4 * self.streams * (self.streams + 2)


@dataclass
class StreamsPending:
    """What such a block hands on: the streams still lack ``term``, which joins them as ``connection`` says."""
    term: torch.Tensor
    connection: HyperConnection


def _pending(delta):
    if delta is None:
        return None, None, None
    if not isinstance(delta, StreamsPending):
        raise ValueError("hyper-connected blocks stand among their own kind: the block before handed on another kind of term")
    return delta.term, delta.connection.mix, delta.connection.share


def read_streams(streams, delta, rows, into, norm, dtype):
    """The normed sum of the streams, weighted by ``into``, at ``rows``, with what the last block left pending."""
    term, mix, share = _pending(delta)
    return ops.streams_step(streams, term, mix, share, into, norm.weight, norm.eps, dtype, rows=rows)


@BLOCKS.register("hyper_connected")
class HyperConnectedBlock:
    """Roles: ``mixer``, ``mixer_norm``, ``mixer_hc`` and, for a feed-forward, ``ffn``, ``ffn_norm``, ``ffn_hc``.  The norms are RMS
    norms with a gain per channel (``weight`` float32 ``[size]`` and ``eps``), the connections `HyperConnection`s of one number of
    streams; the sublayers return their term (or a stack of partial sums) in float32."""

    ROLES = ("mixer", "mixer_norm", "mixer_hc", "ffn", "ffn_norm", "ffn_hc")

    def __init__(self, parts: dict):
        if set(parts) not in (set(self.ROLES), set(self.ROLES[:3])):
            raise ValueError(f"the hyper-connected block arranges {self.ROLES} (or the first three alone); the layer names {sorted(parts)}")
        g = parts.get
        self.mixer, self.mixer_norm, self.mixer_hc = g("mixer"), g("mixer_norm"), g("mixer_hc")
        self.ffn, self.ffn_norm, self.ffn_hc = g("ffn"), g("ffn_norm"), g("ffn_hc")
        for n in (self.mixer_norm, self.ffn_norm):
            if n is not None and not (hasattr(n, "eps") and hasattr(n, "weight")):
                raise ValueError("the hyper-connected block's norms are RMS norms with a gain per channel")
        if self.ffn_hc is not None and self.ffn_hc.streams != self.mixer_hc.streams:
            raise ValueError(f"the hyper-connected block: {self.mixer_hc.streams} and {self.ffn_hc.streams} streams in one layer")

    def cache_need(self):
        return self.mixer.cache_need()

    @staticmethod
    def _read(streams, delta, connection, norm):
        term, mix, share = _pending(delta)
        return ops.streams_step(streams, term, mix, share, connection.into, norm.weight, norm.eps, norm.dtype)

    def forward(self, streams, delta, step, cache, position, write_cache=True):
        h = self._read(streams, delta, self.mixer_hc, self.mixer_norm)
        pending = StreamsPending(self.mixer.forward(h, step, cache, position, write_cache), self.mixer_hc)
        if self.ffn is None:
            return pending
        h = self._read(streams, pending, self.ffn_hc, self.ffn_norm)
        return StreamsPending(self.ffn.forward(h, step), self.ffn_hc)
