"""Gated delta rule as a mixer: a matrix state per head, carried in the request's state slot.

For every head, with ``S [key_dim, value_dim]`` starting at zero, token by token::

    S <- g * S                       g = exp(-exp(A) * softplus(a + bias))     decay, one number a head or one a head and
                                                                               key channel (which decays that row of S)
    u  = beta * (v - S^T k)          beta = sigmoid(b)                         how strongly the new value is written
    S <- S + k u^T
    o  = S^T q                       (the read-out sees this token's write)

q and k have ``kv_heads`` heads, each shared by ``heads / kv_heads`` value heads; q, k and v pass a short causal
convolution and SiLU; q and k are made unit vectors (q also times ``key_dim ** -0.5``).  The read-out of a head is
RMS-normed over ``value_dim``, weighted, and multiplied by ``silu`` or ``sigmoid`` of a gate projection; then the output
projection.  The decay logits and the gate come from one matrix each or through narrow projections of some ``rank``
numbers (``W_up (W_down x)``).

One product computes q, k, v, the write-strength logits and the gate and decay logits (or their narrow numbers, which a
second product widens, both at once) from the block's input; the convolution, the unit norms, decay and write strength,
the recurrence and the gated norm are kernels of ``csrc/sequence.cu``.  State, decays, write strengths and unit norms are
32-bit whatever the compute dtype.  The state slot holds ``S [heads, key_dim, value_dim]`` and behind it the convolution's
last ``taps - 1`` inputs ``[taps - 1, channels]``.
"""
from __future__ import annotations

import torch

from .registry import Runtime, StateNeed, TensorInfo, register_mixer
from ._bind import bind_matrix, stack_rows


@register_mixer("gated_delta")
class GatedDelta:
    pad_safe = True            # the kernels go by requests: rows of no request are never read or written

    @classmethod
    def expected_tensors(cls, spec):
        n = spec.names
        conv = spec.conv_taps
        out = {n["q"]: TensorInfo((spec.qk_size, spec.hidden)), n["k"]: TensorInfo((spec.qk_size, spec.hidden)),
               n["v"]: TensorInfo((spec.v_size, spec.hidden)),
               n["q_conv"]: TensorInfo((spec.qk_size, conv), "conv"), n["k_conv"]: TensorInfo((spec.qk_size, conv), "conv"),
               n["v_conv"]: TensorInfo((spec.v_size, conv), "conv"), n["beta"]: TensorInfo((spec.heads, spec.hidden)),
               n["decay_log"]: TensorInfo((spec.heads,), "unit_normal"),
               n["decay_bias"]: TensorInfo((spec.decays,), "unit_normal"),
               n["out_norm"]: TensorInfo((spec.value_dim,), "one_plus_normal"),
               n["o"]: TensorInfo((spec.hidden, spec.v_size))}
        for role, size, rank in (("decay", spec.decays, spec.decay_rank), ("gate", spec.v_size, spec.gate_rank)):
            if rank is None:
                out[n[role]] = TensorInfo((size, spec.hidden))
            else:
                out[n[role + "_down"]] = TensorInfo((rank, spec.hidden))
                out[n[role + "_up"]] = TensorInfo((size, rank))
        return out

    def __init__(self, spec, weights, rt: Runtime):
        if spec.heads % spec.kv_heads:
            raise ValueError(f"heads ({spec.heads}) must be a multiple of kv_heads ({spec.kv_heads})")
        if spec.decay_per not in ("head", "channel") or spec.gate_activation not in ("silu", "sigmoid"):
            raise ValueError("gated delta rule: decay_per is 'head' or 'channel', gate_activation 'silu' or 'sigmoid'")
        self.spec, self.rt = spec, rt
        n = spec.names
        # one product for everything that reads the block's input: [q | k | v | gate | beta | decay], narrow numbers
        # behind, the first at a multiple of 32 columns
        ranks = {"gate": spec.gate_rank, "decay": spec.decay_rank}
        wide = [weights[n[r]] for r in ("q", "k", "v", "gate", "beta", "decay") if ranks.get(r) is None]
        narrow = [r for r in ("gate", "decay") if ranks[r] is not None]
        wide = torch.cat(wide, dim=0)
        self.w_up = None
        if narrow:
            low = torch.cat([weights[n[r + "_down"]] for r in narrow], dim=0)
            low = torch.cat([low, low.new_zeros((-low.shape[0] % 32, low.shape[1]))], dim=0)
            wide, (_, self.low_at) = stack_rows([wide, low], align=32)
            # both second matrices as one, block by block (zeros elsewhere)
            up = wide.new_zeros((sum(weights[n[r + "_up"]].shape[0] for r in narrow), low.shape[0]))
            row = col = 0
            self._up_at = {}
            for r in narrow:
                w = weights[n[r + "_up"]]
                up[row:row + w.shape[0], col:col + w.shape[1]] = w
                self._up_at[r] = slice(row, row + w.shape[0])
                row, col = row + w.shape[0], col + w.shape[1]
            self.w_up = bind_matrix(up, rt)
        self.w_in = bind_matrix(wide, rt)
        self.w_conv = bind_matrix(torch.cat([weights[n[r]] for r in ("q_conv", "k_conv", "v_conv")], dim=0), rt)
        self.w_o = bind_matrix(weights[n["o"]], rt)
        f32 = dict(device=rt.device, dtype=torch.float32)
        self.decay_log = weights[n["decay_log"]].to(**f32).contiguous()
        self.decay_bias = weights[n["decay_bias"]].to(**f32).contiguous()
        self.out_norm = weights[n["out_norm"]].to(**f32).contiguous()
        self.channels = 2 * spec.qk_size + spec.v_size
        self.matrix_numbers = spec.heads * spec.key_dim * spec.value_dim

    def cache_need(self):
        return StateNeed((self.matrix_numbers + (self.spec.conv_taps - 1) * self.channels,), torch.float32)

    def inner(self, proj, step, cache, out=None, scale=1.0):
        """From the rows ``[T, q | k | v | gate | beta | decay]`` (or with narrow numbers behind) to what the output product
        reads."""
        s, ops = self.spec, self.rt.ops
        C, H = self.channels, s.heads
        logits, at = {}, C
        if self.w_up is not None:
            low = proj[:, self.low_at:self.low_at + self.w_up.shape[1]]
            wide = ops.linear(low, self.w_up, out_dtype=torch.float32)
            logits = {r: wide[:, cols] for r, cols in self._up_at.items()}
        for r, size in (("gate", s.v_size), ("beta", H), ("decay", s.decays)):
            if r not in logits:
                logits[r] = proj[:, at:at + size]
                at += size
        qkv = ops.causal_conv(proj[:, :C], self.w_conv, step=step, state=cache.state, state_offset=self.matrix_numbers,
                              activation="silu")
        o = ops.gated_delta_rule(qkv, logits["beta"], logits["decay"], decay_log=self.decay_log, decay_bias=self.decay_bias,
                                 state=cache.state, step=step, heads=H, kv_heads=s.kv_heads, key_dim=s.key_dim,
                                 value_dim=s.value_dim, unit_eps=s.unit_eps, q_scale=s.key_dim ** -0.5)
        if out is None:
            out = torch.empty(proj.shape[0], s.v_size, dtype=proj.dtype, device=proj.device)
        return ops.gated_rmsnorm(o, logits["gate"], self.out_norm, s.norm_eps, activation=s.gate_activation, scale=scale,
                                 out=out)

    def forward(self, x, step, cache):
        ops = self.rt.ops
        return ops.linear(self.inner(ops.linear(x, self.w_in), step, cache), self.w_o)
