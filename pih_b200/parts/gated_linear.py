"""Gated linear attention as a mixer: a matrix state a head whose rows decay by numbers of their own.

For every head, with ``S [key_dim, value_dim]`` starting at zero, token by token::

    a = sigmoid(W_up (W_down x) + bias) ** (1 / temperature)      one number a head and key channel
    S <- diag(a) S + k v^T
    o = S^T q * key_dim ** -0.5                                   (the read-out sees this token's write)

(Yang et al., "Gated Linear Attention Transformers with Hardware-Efficient Training").  The read-out of a head is RMS-normed
over ``value_dim`` with one weight for all heads, multiplied by ``silu`` of a gate projection, and projected.

One product computes q, k, v, the gate and the narrow numbers in front of the decays; a second one widens these, 32-bit out.
Decays, state and the read-out's norm are 32-bit whatever the compute dtype.
"""
from __future__ import annotations

import torch

from .registry import Runtime, StateNeed, TensorInfo, register_mixer
from ._bind import bind_matrix, pad_columns, stack_rows


@register_mixer("gated_linear")
class GatedLinear:
    pad_safe = True            # the kernels go by requests: rows of no request are never read or written

    @classmethod
    def expected_tensors(cls, spec):
        n, QK, VS = spec.names, spec.qk_size, spec.v_size
        return {n["q"]: TensorInfo((QK, spec.hidden)), n["k"]: TensorInfo((QK, spec.hidden)),
                n["v"]: TensorInfo((VS, spec.hidden)), n["gate"]: TensorInfo((VS, spec.hidden)),
                n["o"]: TensorInfo((spec.hidden, VS)), n["out_norm"]: TensorInfo((spec.value_dim,), "one_plus_normal"),
                n["decay_down"]: TensorInfo((spec.decay_rank, spec.hidden)), n["decay_up"]: TensorInfo((QK, spec.decay_rank)),
                n["decay_bias"]: TensorInfo((QK,), "unit_normal")}

    def __init__(self, spec, weights, rt: Runtime):
        if spec.temperature <= 0:
            raise ValueError("gated linear attention: the temperature must be positive")
        self.spec, self.rt = spec, rt
        n = spec.names
        wide = torch.cat([weights[n[r]] for r in ("q", "k", "v", "gate")], dim=0)
        # the narrow numbers behind the others, at a multiple of 32 columns and as many as make a multiple of 32 (rows of
        # zeros, which meet columns of zeros): sizes of the few-rows product
        low = weights[n["decay_down"]]
        low = torch.cat([low, low.new_zeros((-low.shape[0] % 32, low.shape[1]))], dim=0)
        stacked, (_, self.low_at) = stack_rows([wide, low], align=32)
        self.low_size = low.shape[0]
        self.w_in = bind_matrix(stacked, rt)
        self.w_up = bind_matrix(pad_columns(weights[n["decay_up"]], self.low_size), rt)
        self.w_o = bind_matrix(weights[n["o"]], rt)
        f32 = dict(device=rt.device, dtype=torch.float32)
        self.decay_bias = weights[n["decay_bias"]].to(**f32).contiguous()
        self.out_norm = weights[n["out_norm"]].to(**f32).contiguous()

    def cache_need(self):
        s = self.spec
        return StateNeed((s.heads * s.key_dim * s.value_dim,), torch.float32)

    def inner(self, proj, step, cache, out=None, scale=1.0):
        """From the rows ``[T, q | k | v | gate | narrow numbers]`` to what the output product reads."""
        s, ops, QK, VS = self.spec, self.rt.ops, self.spec.qk_size, self.spec.v_size
        z = ops.linear(proj[:, self.low_at:self.low_at + self.low_size], self.w_up, out_dtype=torch.float32)
        o = ops.gated_linear(proj[:, :QK], proj[:, QK:2 * QK], proj[:, 2 * QK:2 * QK + VS], z, bias=self.decay_bias,
                             temperature=s.temperature, q_scale=s.key_dim ** -0.5, state=cache.state, step=step, heads=s.heads,
                             key_dim=s.key_dim, value_dim=s.value_dim)
        return ops.gated_rmsnorm(o, proj[:, 2 * QK + VS:2 * QK + 2 * VS], self.out_norm, s.norm_eps, scale=scale, out=out)

    def forward(self, x, step, cache):
        ops = self.rt.ops
        return ops.linear(self.inner(ops.linear(x, self.w_in), step, cache), self.w_o)
