"""State-space duality (Mamba-2) as a mixer: a matrix state a head with one decay a token.

``W_in`` gives ``[z: inner | x: inner | B: groups * state | C: groups * state | dt: heads]``.  x, B and C pass one short causal
convolution per channel (with a bias) and SiLU.  Then for every head, with ``S [state, value_dim]`` starting at zero and the
head's group of B and C::

    dt <- softplus(dt + bias)
    S  <- exp(-exp(A_log) dt) S + dt B x^T
    y  =  S^T C + D x

(the recurrence of Dao and Gu, "Transformers are SSMs: Generalized Models and Efficient Algorithms Through Structured State
Space Duality").  ``y * silu(z)`` is RMS-normed in ``norm_groups`` equal parts of the row, weighted a column, and projected.
Step sizes, decays, state and norm are 32-bit whatever the compute dtype.  The state slot holds ``S [heads, state,
value_dim]`` and behind it the convolution's last ``taps - 1`` inputs.
"""
from __future__ import annotations

import torch

from .registry import Runtime, StateNeed, TensorInfo, register_mixer
from ._bind import bind_matrix


@register_mixer("state_space")
class StateSpace:
    pad_safe = True            # the kernels go by requests: rows of no request are never read or written

    @classmethod
    def expected_tensors(cls, spec):
        n, W, H = spec.names, spec.inner, spec.heads
        channels = W + 2 * spec.bc_size
        return {n["w_in"]: TensorInfo((W + channels + H, spec.hidden)), n["conv"]: TensorInfo((channels, spec.conv_taps), "conv"),
                n["conv_bias"]: TensorInfo((channels,)), n["dt_bias"]: TensorInfo((H,), "unit_normal"),
                n["a_log"]: TensorInfo((H,), "unit_normal"), n["skip"]: TensorInfo((H,), "one_plus_normal"),
                n["out_norm"]: TensorInfo((W,), "one_plus_normal"), n["o"]: TensorInfo((spec.hidden, W))}

    def __init__(self, spec, weights, rt: Runtime):
        if spec.heads % spec.groups or spec.inner % spec.norm_groups:
            raise ValueError("state space: groups must divide the heads, norm_groups the inner width")
        self.spec, self.rt = spec, rt
        n = spec.names
        self.w_in = bind_matrix(weights[n["w_in"]], rt)
        self.w_conv = bind_matrix(weights[n["conv"]], rt)
        self.w_o = bind_matrix(weights[n["o"]], rt)
        f32 = dict(device=rt.device, dtype=torch.float32)
        self.conv_bias = weights[n["conv_bias"]].to(**f32).contiguous()
        self.dt_bias = weights[n["dt_bias"]].to(**f32).contiguous()
        self.A = (-torch.exp(weights[n["a_log"]].to(torch.float64))).to(**f32).contiguous()
        self.skip = weights[n["skip"]].to(**f32).contiguous()
        self.out_norm = weights[n["out_norm"]].to(**f32).contiguous()
        self.channels = spec.inner + 2 * spec.bc_size
        self.matrix_numbers = spec.heads * spec.state * spec.value_dim

    def cache_need(self):
        return StateNeed((self.matrix_numbers + (self.spec.conv_taps - 1) * self.channels,), torch.float32)

    def inner(self, proj, step, cache, out=None, scale=1.0):
        """From the rows ``[T, z | x | B | C | dt]`` to what the output product reads."""
        s, ops, W, N = self.spec, self.rt.ops, self.spec.inner, self.spec.bc_size
        xbc = ops.causal_conv(proj[:, W:W + self.channels], self.w_conv, step=step, state=cache.state,
                              state_offset=self.matrix_numbers, out_bias=self.conv_bias, activation="silu")
        at = W + self.channels
        y = ops.state_space(xbc[:, W + N:], xbc[:, W:W + N], xbc[:, :W], proj[:, at:at + s.heads], dt_bias=self.dt_bias, A=self.A,
                            D=self.skip, state=cache.state, step=step, heads=s.heads, groups=s.groups, state_dim=s.state,
                            value_dim=s.value_dim)
        return ops.gated_part_rmsnorm(y.view(-1, W), proj[:, :W], self.out_norm, s.norm_groups, s.norm_eps, scale=scale, out=out)

    def forward(self, x, step, cache):
        ops = self.rt.ops
        return ops.linear(self.inner(ops.linear(x, self.w_in), step, cache), self.w_o)
