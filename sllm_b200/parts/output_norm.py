"""A layer whose sublayers read the stream as it is and whose outputs alone are normed:

    x <- x + post(mixer(x));   x <- x + post(ffn(x));   x <- x + post(side(x))

and the side term that takes in a vector belonging to the token and the layer.  Each part takes its sizes and constants as
parameters; none names a model.

A sublayer's output is normed before it joins the stream, so no product can add into the stream itself; one kernel per
sublayer norms the output, adds it, and writes the stream in the compute dtype for the next reader (`ops.post_add_copy`), also
across the border between two such layers (`StreamCopy`).
"""

from __future__ import annotations

import torch

from .. import ops
from .base import BLOCKS, FEED_FORWARDS, FeedForward, StreamCopy, TensorSpec
from .parallel import pending_terms
from .standard import Linear


@FEED_FORWARDS.register("token_side")
class TokenSide(FeedForward):
    """proj(gelu_tanh(gate(x)) * e) with e the columns ``offset .. offset + dim`` of the model's table of token vectors at the
    token's id (`ModelPlan.token_table_name`; the model hands the table over).  Two matrices without biases, ``gate``
    ``[dim, hidden]`` and ``proj`` ``[hidden, dim]``."""

    def __init__(self, params, **kw):
        super().__init__(params, **kw)
        self.hidden = int(params["hidden_size"])
        self.dim = int(params["dim"])
        self.offset = int(params["offset"])
        self.gate = self.proj = self.table = None

    def tensor_specs(self):
        return [TensorSpec("gate", (self.dim, self.hidden)), TensorSpec("proj", (self.hidden, self.dim))]

    def bind(self, fetch):
        self.gate, self.proj = Linear(self._matrix(fetch("gate"))), Linear(self._matrix(fetch("proj")))

    def adopt_token_table(self, table):
        if self.offset + self.dim > table.shape[1]:
            raise ValueError(f"token_side: columns {self.offset}..{self.offset + self.dim} of a table with {table.shape[1]}")
        self.table = table

    def forward(self, x, step):
        g = ops.linear_plain_act(x, self.gate.weight, self.dtype, "token", ops.TokenColumns(self.table, step.token_ids, self.offset))
        return self.proj(g, torch.float32, True)

    def weight_bytes(self):
        return self.gate.nbytes() + self.proj.nbytes()


class StreamReader:
    """What such a block shows as its first norm: none; it reads the stream in ``dtype``."""

    def __init__(self, dtype):
        self.dtype = dtype

    def as_rms(self):
        return None


@BLOCKS.register("output_norm")
class OutputNormBlock:
    """Roles: ``mixer`` and ``mixer_post``; optionally ``ffn`` with ``ffn_post`` and ``side`` with ``side_post``, in this order.  The
    norms are RMS norms with a gain per channel (``weight`` float32 ``[size]`` and ``eps``); the sublayers return their term (or
    a stack of partial sums) in float32."""

    ROLES = ("mixer", "mixer_post", "ffn", "ffn_post", "side", "side_post")

    def __init__(self, parts: dict):
        unknown = set(parts) - set(self.ROLES)
        if unknown or not {"mixer", "mixer_post"} <= set(parts):
            raise ValueError(f"the output-norm block arranges {self.ROLES}; the layer names {sorted(parts)}")
        for role in ("ffn", "side"):
            if (role in parts) != (role + "_post" in parts):
                raise ValueError(f"the output-norm block: {role} comes with its norm, or not at all")
        self.mixer = parts["mixer"]
        self.terms = [(role, parts[role], parts[role + "_post"]) for role in ("mixer", "ffn", "side") if role in parts]
        for _, _, post in self.terms:
            if not (hasattr(post, "eps") and hasattr(post, "weight")):
                raise ValueError("the output-norm block's norms are RMS norms with a gain per channel")
        self.dtype = parts["mixer_post"].dtype

    def cache_need(self):
        return self.mixer.cache_need()

    accepts_next_norm = True

    @property
    def first_norm(self):
        return StreamReader(self.dtype)

    def forward(self, residual, delta, step, cache, position, write_cache=True, next_norm=None):
        if isinstance(delta, StreamCopy):
            h = delta.x
        else:
            terms = pending_terms(delta)
            if terms:
                ops.add_group_ssq(residual, terms, 1, 0.0, want_rinv=False)
            h = ops.post_add_copy(residual, None, None, 0.0, self.dtype)
        for i, (role, part, post) in enumerate(self.terms):
            term = part.forward(h, step, cache, position, write_cache) if role == "mixer" else part.forward(h, step)
            # the next reader of the stream: the layer's next sublayer, or another such layer; else nobody wants a copy
            wanted = i + 1 < len(self.terms) or isinstance(next_norm, StreamReader)
            h = ops.post_add_copy(residual, term, post.weight, post.eps, self.dtype if wanted else None)
        return StreamCopy(h) if h is not None else None
