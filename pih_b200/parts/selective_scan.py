"""Selective scan as a mixer: a diagonal state per channel whose step sizes and read-out come from the token.

``W_in`` gives two branches ``[x | z]`` of ``inner`` channels.  x passes a short causal convolution per channel (with a
bias) and SiLU; ``W_x`` of it gives ``[dt: dt_rank | B: state | C: state]``, ``W_dt`` the step-size logits of the channels.
Then, for every channel, with its row of states starting at zero::

    dt  = softplus(logit + bias)       A = -exp(A_log)            (one step size, a row of rates)
    row <- exp(dt * A) * row + (dt * x) B                         (element by element)
    y   = <row, C> + D x

and the output is ``W_o (y * silu(z))``.  (The recurrence of Gu and Dao, "Mamba: Linear-Time Sequence Modeling with
Selective State Spaces".)  Step sizes, exponentials and the state are 32-bit whatever the compute dtype.  The state slot
holds ``S [inner, state]`` and behind it the convolution's last ``taps - 1`` inputs ``[taps - 1, inner]``.
"""
from __future__ import annotations

import torch

from .registry import Runtime, StateNeed, TensorInfo, register_mixer
from ._bind import bind_matrix, pad_columns, stack_rows


@register_mixer("selective_scan")
class SelectiveScan:
    pad_safe = True            # the kernels go by requests: rows of no request are never read or written

    @classmethod
    def expected_tensors(cls, spec):
        n, W, N = spec.names, spec.inner, spec.state
        return {n["w_in"]: TensorInfo((2 * W, spec.hidden)), n["conv"]: TensorInfo((W, spec.conv_taps), "conv"),
                n["conv_bias"]: TensorInfo((W,)), n["x"]: TensorInfo((spec.dt_rank + 2 * N, W)),
                n["dt"]: TensorInfo((W, spec.dt_rank)), n["dt_bias"]: TensorInfo((W,), "unit_normal"),
                n["a_log"]: TensorInfo((W, N), "unit_normal"), n["skip"]: TensorInfo((W,), "one_plus_normal"),
                n["o"]: TensorInfo((spec.hidden, W))}

    def __init__(self, spec, weights, rt: Runtime):
        self.spec, self.rt = spec, rt
        n = spec.names
        self.w_in = bind_matrix(weights[n["w_in"]], rt)                                            # [x | z]
        self.w_conv = bind_matrix(weights[n["conv"]], rt)
        w_x, R = weights[n["x"]], spec.dt_rank
        # rows of zeros behind the dt rows (and columns of zeros in W_dt) bring the second product to a size of the
        # few-rows kernel; they add zeros
        x, (_, self.bc_at) = stack_rows([w_x[:R], w_x[R:]], align=32)
        self.w_x = bind_matrix(x, rt)
        self.w_dt = bind_matrix(pad_columns(weights[n["dt"]], self.bc_at), rt)
        self.w_o = bind_matrix(weights[n["o"]], rt)
        f32 = dict(device=rt.device, dtype=torch.float32)
        self.conv_bias = weights[n["conv_bias"]].to(**f32).contiguous()
        self.dt_bias = weights[n["dt_bias"]].to(**f32).contiguous()
        self.A = (-torch.exp(weights[n["a_log"]].to(torch.float64))).to(**f32).contiguous()
        self.skip = weights[n["skip"]].to(**f32).contiguous()

    def cache_need(self):
        s = self.spec
        return StateNeed((s.inner * (s.state + s.conv_taps - 1),), torch.float32)

    def inner(self, proj, step, cache, out=None, scale=1.0):
        s, ops, W = self.spec, self.rt.ops, self.spec.inner
        u = ops.causal_conv(proj[:, :W], self.w_conv, step=step, state=cache.state, state_offset=W * s.state,
                            out_bias=self.conv_bias, activation="silu")
        p = ops.linear(u, self.w_x)                                         # [T, dt | zeros | B | C]
        dt = ops.linear(p[:, :self.bc_at], self.w_dt, out_dtype=torch.float32)
        return ops.selective_scan(u, dt, p[:, self.bc_at:], proj[:, W:2 * W], dt_bias=self.dt_bias, A=self.A, D=self.skip,
                                  state=cache.state, step=step, scale=scale, out=out)

    def forward(self, x, step, cache):
        ops = self.rt.ops
        return ops.linear(self.inner(ops.linear(x, self.w_in), step, cache), self.w_o)
