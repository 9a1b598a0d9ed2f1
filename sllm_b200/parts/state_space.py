"""State-space mixers: a recurrence with one decay per token and head (Mamba-2, state-space duality).

    [z | x | B | C | dt] = W_in h;    x, B, C <- silu(causal convolution over time + bias);    dt <- softplus(dt + dt_bias)
    S_t = exp(-exp(A_log) dt_t) S_(t-1) + dt_t B_t x_t^T,      y_t = S_t^T C_t + D x_t            (per head; heads share B and C in groups)
    out = W_o (norm(y * silu(z)))      with the norm in equal parts, each over its own root mean square

The state and the convolution's last inputs live in the request's state slots, so a prompt's portions and single decoded tokens
continue one another.
"""

from __future__ import annotations

import torch

from .. import ops
from .base import MIXERS, LayerCache, Mixer, SlotState, StepContext, TensorSpec
from .standard import Linear


@MIXERS.register("mamba2")
class Mamba2(Mixer):
    """Parameters: ``hidden_size``, ``heads``, ``vdim`` (channels of a head), ``state`` (rows of a head's state), ``groups`` (of heads
    that share B and C), ``conv`` (the convolution's taps), ``norm_groups``, ``eps`` (of the output's norm).  W_in is one product that
    stays float32, as everything up to the gated norm does."""

    def __init__(self, params, **kw):
        super().__init__(params, **kw)
        p = params
        self.hidden = int(p["hidden_size"])
        self.heads, self.vdim, self.N = int(p["heads"]), int(p["vdim"]), int(p["state"])
        self.groups, self.taps = int(p["groups"]), int(p["conv"])
        self.norm_groups = int(p["norm_groups"])
        self.eps = float(p["eps"])
        self.inner = self.heads * self.vdim
        self.channels = self.inner + 2 * self.groups * self.N
        if self.heads % self.groups:
            raise ValueError(f"mamba2: {self.heads} heads are no multiple of {self.groups} groups")
        if self.inner % self.norm_groups:
            raise ValueError(f"mamba2: {self.norm_groups} parts of the norm do not divide {self.inner} channels")
        if self.taps < 1:
            raise ValueError(f"mamba2: conv={self.taps} must be at least 1")
        if not ops.delta_rule_supports(self.N, self.vdim):
            raise ValueError(f"mamba2: a state of {self.N} rows is outside what the recurrence kernel keeps in registers (1..256)")

    def cache_need(self):
        needs = (SlotState((self.heads, self.N, self.vdim), "ssm"),)
        return needs + (SlotState((self.channels, self.taps - 1), "conv"),) if self.taps > 1 else needs

    def tensor_specs(self):
        W, H, I = self.hidden, self.heads, self.inner
        return [TensorSpec("in", (I + self.channels + H, W)), TensorSpec("conv", (self.channels, self.taps)),
                TensorSpec("conv.b", (self.channels,), role="bias"), TensorSpec("dt_bias", (H,), role="bias"),
                TensorSpec("A_log", (H,), role="bias"), TensorSpec("D", (H,), role="gain"), TensorSpec("norm", (I,), role="gain"),
                TensorSpec("o", (W, I))]

    def bind(self, fetch):
        self.inp = Linear(self._matrix(fetch("in")))
        self.conv, self.conv_bias = self._f32(fetch("conv")), self._f32(fetch("conv.b"))
        self.dt_bias, self.a_log, self.skip = (self._f32(fetch(n)) for n in ("dt_bias", "A_log", "D"))
        self.gain = self._f32(fetch("norm"))
        self.out = Linear(self._matrix(fetch("o")))

    accepts_residual = True

    def mix(self, x, step: StepContext, cache: LayerCache, position=None, write_cache=True):
        I = self.inner
        proj = self.inp(x, torch.float32)                                            # [T, z | x B C | dt] float32
        xbc = ops.short_conv_silu(proj, I, self.conv, cache.states.get("conv"), step, bias=self.conv_bias)
        y = ops.state_space(xbc, proj, I + self.channels, self.dt_bias, self.a_log, self.skip, cache.states["ssm"], step, self.heads,
                            self.groups, self.N, self.vdim)                          # [T, inner] float32
        return ops.gated_group_norm(y, proj, 0, self.gain, self.eps, self.norm_groups, self.dtype)

    def forward(self, x, step, cache, position, write_cache=True, residual=None):
        return self.out.into(self.mix(x, step, cache, position, write_cache), residual)

    def weight_bytes(self):
        return self.inp.nbytes() + self.out.nbytes() + 4 * (self.channels * (self.taps + 1) + self.inner + 3 * self.heads)
