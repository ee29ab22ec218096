"""Matrix memory with exponential gates (the mLSTM of Beck et al., "xLSTM: Extended Long Short-Term Memory") as a mixer.

For every head, with ``S [key_dim, value_dim]``, ``n [key_dim]`` and ``m`` starting at zero, token by token::

    i = cap tanh((W_i x + b_i) / cap)        f = logsigmoid(cap tanh((W_f x + b_f) / cap))        (log gates)
    m' = max(f + m, i)
    S <- exp(f + m - m') S + exp(i - m') k v^T        n <- exp(f + m - m') n + exp(i - m') k        m <- m'
    o = S^T q / (max(|n . q|, exp(-m)) + floor)

with q times ``key_dim ** -0.5``.  A head's read-out is divided by its root mean square; the heads side by side are multiplied
by a weight a column and by ``sigmoid`` of a gate projection, and projected.

One product computes q, k, v, the gate and the gates' logits; log gates, running maximum, state, key sum and the read-out's
norm are 32-bit whatever the compute dtype.  The state slot holds S, n, and the running maxima (as many a head as the kernel
wants copies of: each of its blocks reads and writes one of its own).
"""
from __future__ import annotations

import torch

from .registry import Runtime, StateNeed, TensorInfo, register_mixer
from ._bind import bind_matrix


@register_mixer("matrix_memory")
class MatrixMemory:
    pad_safe = True            # the kernels go by requests: rows of no request are never read or written

    @classmethod
    def expected_tensors(cls, spec):
        n, QK, VS, H = spec.names, spec.qk_size, spec.v_size, spec.heads
        return {n["q"]: TensorInfo((QK, spec.hidden)), n["k"]: TensorInfo((QK, spec.hidden)),
                n["v"]: TensorInfo((VS, spec.hidden)), n["gate"]: TensorInfo((VS, spec.hidden)),
                n["o"]: TensorInfo((spec.hidden, VS)), n["out_norm"]: TensorInfo((VS,), "one_plus_normal"),
                n["write"]: TensorInfo((H, spec.hidden)), n["write_bias"]: TensorInfo((H,), "unit_normal"),
                n["keep"]: TensorInfo((H, spec.hidden)), n["keep_bias"]: TensorInfo((H,), "unit_normal")}

    def __init__(self, spec, weights, rt: Runtime):
        if spec.gate_cap <= 0:
            raise ValueError("matrix memory: the cap of the gates must be positive")
        self.spec, self.rt = spec, rt
        n = spec.names
        rows = torch.cat([weights[n[r]] for r in ("q", "k", "v", "gate", "write", "keep")], dim=0)
        # (a whole number of 8 columns, so that every row of the product begins at a multiple of 16 bytes)
        self.w_in = bind_matrix(torch.cat([rows, rows.new_zeros((-rows.shape[0] % 8, rows.shape[1]))], dim=0), rt)
        self.w_o = bind_matrix(weights[n["o"]], rt)
        f32 = dict(device=rt.device, dtype=torch.float32)
        self.write_bias = weights[n["write_bias"]].to(**f32).contiguous()
        self.keep_bias = weights[n["keep_bias"]].to(**f32).contiguous()
        self.out_norm = weights[n["out_norm"]].to(**f32).contiguous()

    def cache_need(self):
        s = self.spec
        return StateNeed((s.heads * (s.key_dim * s.value_dim + s.key_dim + self.rt.ops.memory_copies(s.value_dim)),), torch.float32)

    def inner(self, proj, step, cache, out=None, scale=1.0):
        """From the rows ``[T, q | k | v | gate | write | keep]`` to what the output product reads."""
        s, ops, QK, VS, H = self.spec, self.rt.ops, self.spec.qk_size, self.spec.v_size, self.spec.heads
        at = 2 * QK + 2 * VS
        o, divisor = ops.matrix_memory(proj[:, :QK], proj[:, QK:2 * QK], proj[:, 2 * QK:2 * QK + VS], proj[:, at:at + H],
                                       proj[:, at + H:at + 2 * H], write_bias=self.write_bias, keep_bias=self.keep_bias,
                                       cap=s.gate_cap, floor=s.floor, q_scale=s.key_dim ** -0.5, state=cache.state, step=step,
                                       heads=H, key_dim=s.key_dim, value_dim=s.value_dim)
        return ops.gated_rmsnorm(o, proj[:, 2 * QK + VS:at], self.out_norm, s.norm_eps, activation="sigmoid", scale=scale,
                                 out=out, divisor=divisor)

    def forward(self, x, step, cache):
        ops = self.rt.ops
        return ops.linear(self.inner(ops.linear(x, self.w_in), step, cache), self.w_o)
