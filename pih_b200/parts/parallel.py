"""Two mixers side by side: ``left_scale * left(x) + right_scale * right(x)``, both reading the same input.

Both mixers show their two products and the inner part between them (``w_in``, ``w_o``, ``inner``; see the registry), so
that the pair costs one product in front — the rows of both, the right one's beginning at a multiple of 32 — and one
behind, over the inner outputs side by side.  The two scales multiply the inner outputs in 32-bit, inside the kernels that
write them, so the sum of the two mixers is the second product's own sum.

With ``out_norm_eps`` each of the two outputs is RMS-normed over the width, with a weight of its own, before it is scaled and
added: then there is a product behind each inner part, and the two norms, which read 32-bit sums of the products and the
left and right output biases, are the business of the kernel that also norms the pair's sum and adds it to the stream
(``forward_pair``, which the block has to ask for).

The pair's cache is what both ask for: at most one paged cache, and one state vector per request with the left mixer's
numbers first.
"""
from __future__ import annotations

from dataclasses import replace

import torch

from .registry import PagedStateNeed, Runtime, StateNeed, TensorInfo, part_class, register_mixer
from ._bind import stack_rows


@register_mixer("parallel")
class ParallelMixers:
    @classmethod
    def _classes(cls, spec):
        return part_class("mixer", spec.left.kind), part_class("mixer", spec.right.kind)

    @classmethod
    def expected_tensors(cls, spec):
        left, right = cls._classes(spec)
        a, b = left.expected_tensors(spec.left), right.expected_tensors(spec.right)
        shared = set(a) & set(b)
        if shared:
            raise ValueError(f"two mixers side by side name the same tensors: {sorted(shared)}")
        out = {**a, **b}
        if spec.out_norm_eps is not None:
            for side in ("left", "right"):
                out[spec.names[side]] = TensorInfo((spec.hidden,), "one_plus_normal")
        return out

    def __init__(self, spec, weights, rt: Runtime):
        self.spec, self.rt = spec, rt
        self.parts = []
        for cls, sub in zip(self._classes(spec), (spec.left, spec.right)):
            if not hasattr(cls, "inner"):
                raise TypeError(f"mixer kind {sub.kind!r} cannot run beside another: it does not show its products")
            self.parts.append(cls(sub, {n: weights[n] for n in cls.expected_tensors(sub)}, rt))
        left, right = self.parts
        self.w_in, self.in_at = stack_rows([left.w_in, right.w_in], align=32)
        self.out_sizes = (left.w_o.shape[1], right.w_o.shape[1])
        # the parts' own matrices are views of the pair's from here on
        left.w_in, right.w_in = (self.w_in[at:at + p.w_in.shape[0]] for at, p in zip(self.in_at, self.parts))
        self.scales = (float(spec.left_scale), float(spec.right_scale))
        self.pairs = spec.out_norm_eps is not None
        biases = [getattr(p, "output_bias", None) for p in self.parts]
        self.output_bias = None
        if self.pairs:
            self.biases = biases
            # the scale of a side goes into the weight of its norm
            self.out_norms = [(weights[spec.names[side]].to(device=rt.device, dtype=torch.float32) * scale).contiguous()
                              for side, scale in zip(("left", "right"), self.scales)]
        else:
            self.w_o = torch.cat([left.w_o, right.w_o], dim=1).contiguous()
            left.w_o, right.w_o = self.w_o[:, :self.out_sizes[0]], self.w_o[:, self.out_sizes[0]:]
            scaled = [b * scale for b, scale in zip(biases, self.scales) if b is not None]
            if scaled:
                self.output_bias = torch.stack(scaled).sum(dim=0).contiguous()
        self.paged, self.state_sizes = None, []
        for i, part in enumerate(self.parts):
            need = part.cache_need()
            state = need.state if isinstance(need, PagedStateNeed) else (need if isinstance(need, StateNeed) else None)
            paged = need.paged if isinstance(need, PagedStateNeed) else (need if state is None else None)
            if paged is not None:
                if self.paged is not None:
                    raise ValueError("of two mixers side by side at most one may keep a paged cache")
                self.paged = (i, paged)
            if state is not None and (len(state.shape) != 1 or state.dtype != torch.float32):
                raise ValueError("two mixers side by side keep their states as vectors of 32-bit numbers")
            self.state_sizes.append(state.shape[0] if state is not None else 0)

    @property
    def pad_safe(self) -> bool:
        return all(getattr(p, "pad_safe", False) for p in self.parts)

    def cache_need(self):
        total = sum(self.state_sizes)
        state = StateNeed((total,), torch.float32) if total else None
        if self.paged is None:
            return state
        return PagedStateNeed(self.paged[1], state) if state is not None else self.paged[1]

    def _inner(self, proj, step, cache, outs, scales):
        """Both inner parts from the rows of the product in front; ``outs`` (two views, or None for new tensors)."""
        num, got = 0, []
        for i, part in enumerate(self.parts):
            n = self.state_sizes[i]
            view = cache
            if n:
                view = replace(cache, state=cache.state[:, num:num + n])
            got.append(part.inner(proj[:, self.in_at[i]:self.in_at[i] + part.w_in.shape[0]], step, view, out=outs[i],
                                  scale=scales[i]))
            num += n
        return got

    def forward_pair(self, x, step, cache):
        """``(left output, its bias, (right output, its bias, left weight, right weight, eps))``: what ``Pending`` wants for
        the sum of the two normed outputs."""
        ops = self.rt.ops
        left, right = self._inner(ops.linear(x, self.w_in), step, cache, (None, None), (1.0, 1.0))
        return (ops.linear(left, self.parts[0].w_o), self.biases[0],
                (ops.linear(right, self.parts[1].w_o), self.biases[1], *self.out_norms, float(self.spec.out_norm_eps)))

    def forward(self, x, step, cache):
        ops = self.rt.ops
        if self.pairs:
            raise TypeError("two mixers with norms on their outputs need a block that norms and adds pairs (forward_pair)")
        proj = ops.linear(x, self.w_in)                                     # [T, left | zeros | right]
        # rows of the side-by-side outputs begin at multiples of 16 bytes
        total = sum(self.out_sizes)
        both = torch.empty(x.shape[0], -(-total // 8) * 8, dtype=x.dtype, device=x.device)[:, :total]
        self._inner(proj, step, cache, (both[:, :self.out_sizes[0]], both[:, self.out_sizes[0]:]), self.scales)
        return ops.linear(both, self.w_o)
