"""Typed configuration of the Bipulorn design, read from its config.json keys.

A Bipulorn model is a list of layers with a norm before and a norm behind each sub-layer, whose result a vector multiplies
before it is added — ``x += ls1 * norm1b(mixer(norm1(x)))``, then ``x += ls2 * norm2b(ff(norm2(x)))``, all norm weights stored
around zero — and logits that a tanh caps.  A layer's mixer is one of

* ``"parallel"``: two mixers that read the same input, the result half the sum of their outputs, each RMS-normed with a
  weight of its own: **softmax attention** over a sliding window (biases, grouped key/value heads, a rotation of
  neighbouring pairs slowed down by one factor, a gate a column), and a **state-space dual** layer (Mamba-2);
* ``"gla"``: gated linear attention, a decay a key channel through a narrow projection;
* ``"mlstm"``: matrix memory with exponential gates and a running maximum;

and its feed-forward is a mixture of experts (softmax scores over all outputs, choice by score plus correction, the chosen
ones' scores divided by their sum and scaled, identity experts, a shared expert behind a sigmoid gate) or absent.
config.json holds::

    {"architecture": "Bipulorn", "vocab": V, "width": W, "norm": {"eps": e}, "logit_softcap": c,
     "layers": [{"type": ..., "mixer": {...}, "mlp": {...} | null}, ...]}

The width of the narrow projection is that of the tensor (``with_shapes``); ``decay_rank`` of a gla mixer says it where no
weights exist yet.  The residual stream is summed in 32-bit.  Tensor names: ``embed``, ``head``, ``final.norm``, and
``l<i>.`` + ``norm1`` / ``norm1b`` / ``ls1`` / ``norm2`` / ``norm2b`` / ``ls2`` / ``mix.*`` (``mix.left.*``,
``mix.right.*``) / ``mlp.*`` (see the name tables of the part specs).
"""
from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Optional, Tuple

from .kedavik import _prefixed
from .registry import register_architecture
from .specs import (BlockSpec, ComputedRopeSpec, GatedLinearSpec, MatrixMemorySpec, ModelSpec, NormSpec, ParallelSpec,
                    ScheduleEntry, ScoredMoESpec, StateSpaceSpec, SwiGLUSpec, WindowAttentionSpec)
from .tuganex import DEFAULT_MAX_CONTEXT, _int, _number, _object

_MIXERS = ("parallel", "gla", "mlstm")


@register_architecture("Bipulorn")
@dataclass(frozen=True)
class BipulornConfig:
    vocab: int
    width: int
    norm_eps: float
    logit_softcap: Optional[float]
    layers: Tuple[dict, ...] = field(default_factory=tuple)      # as in config.json, checked

    @classmethod
    def from_dict(cls, raw: dict) -> "BipulornConfig":
        norm = _object(raw, "norm", "config")
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ValueError("config.json: 'layers' must be a non-empty list")
        cap = _number(raw, "logit_softcap", "config") if raw.get("logit_softcap") is not None else None
        cfg = cls(vocab=_int(raw, "vocab", "config"), width=_int(raw, "width", "config"),
                  norm_eps=_number(norm, "eps", "norm"), logit_softcap=cap, layers=tuple(copy.deepcopy(layers)))
        cfg.model_spec()                      # every layer's keys and sizes are checked by building its spec
        return cfg

    def to_dict(self) -> dict:
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
               "layers": copy.deepcopy(list(self.layers))}
        if self.logit_softcap is not None:
            out["logit_softcap"] = self.logit_softcap
        return out

    def with_shapes(self, shapes) -> "BipulornConfig":
        """The configuration with the sizes that only the tensors' shapes give: the width of the narrow projection in front
        of a gla mixer's decays (``a1``)."""
        layers = copy.deepcopy(list(self.layers))
        for i, layer in enumerate(layers):
            shape = shapes.get(f"l{i}.mix.a1")
            if layer.get("type") == "gla" and shape is not None and len(shape) == 2:
                layer["mixer"]["decay_rank"] = int(shape[0])
        return BipulornConfig(self.vocab, self.width, self.norm_eps, self.logit_softcap, tuple(layers))

    # -- layers -----------------------------------------------------------------
    def _attention(self, m: dict, where: str) -> WindowAttentionSpec:
        heads, kv_heads, dim = _int(m, "heads", where), _int(m, "kv_heads", where), _int(m, "dim", where)
        if heads % kv_heads:
            raise ValueError(f"config.json: {where}.heads must be a multiple of kv_heads")
        position = None
        if m.get("rot") is not None:
            rot, rw = _object(m, "rot", where), where + ".rot"
            dims = _int(rot, "dims", rw, minimum=2)
            if dims % 2 or dims > dim:
                raise ValueError(f"config.json: {rw}.dims must be even and at most dim ({dim}), got {dims}")
            slowdown = 1.0
            if rot.get("scaling") is not None:
                slowdown = _number(_object(rot, "scaling", rw), "factor", rw + ".scaling")
            position = ComputedRopeSpec(head_dim=dim, rotary_dim=dims, theta=_number(rot, "base", rw), interleaved=True,
                                        slowdown=slowdown)
        window = 0
        if m.get("mask") is not None:
            window = _int(_object(m, "mask", where), "size", where + ".mask")
        return WindowAttentionSpec(hidden=self.width, heads=heads, kv_heads=kv_heads, key_dim=dim,
                                   value_dim=_int(m, "vdim", where), scale=_number(m, "scale", where, positive=False),
                                   window=window, position=position, sink="none", column_gate=True, biases=True,
                                   names=_prefixed(WindowAttentionSpec, "mix.left."))

    def _state_space(self, m: dict, where: str) -> StateSpaceSpec:
        heads, vdim = _int(m, "heads", where), _int(m, "vdim", where)
        groups, norm_groups = _int(m, "groups", where), _int(m, "norm_groups", where)
        if heads % groups:
            raise ValueError(f"config.json: {where}.heads must be a multiple of groups")
        if heads * vdim % norm_groups:
            raise ValueError(f"config.json: {where}.norm_groups must cut heads * vdim into equal parts")
        return StateSpaceSpec(hidden=self.width, heads=heads, value_dim=vdim, state=_int(m, "state", where), groups=groups,
                              norm_groups=norm_groups, conv_taps=_int(m, "conv", where), norm_eps=self.norm_eps,
                              names=_prefixed(StateSpaceSpec, "mix.right."))

    def _mixer_spec(self, i: int):
        layer = self.layers[i]
        if not isinstance(layer, dict):
            raise ValueError(f"config.json: layers[{i}] must be an object")
        where, kind = f"layers[{i}].mixer", layer.get("type")
        if kind not in _MIXERS:
            raise ValueError(f"config.json: layers[{i}].type must be one of {list(_MIXERS)}, got {kind!r}")
        m = _object(layer, "mixer", f"layers[{i}]")
        if kind == "parallel":
            return ParallelSpec(left=self._attention(_object(m, "left", where), where + ".left"),
                                right=self._state_space(_object(m, "right", where), where + ".right"), left_scale=0.5,
                                right_scale=0.5, out_norm_eps=self.norm_eps)
        sizes = dict(hidden=self.width, heads=_int(m, "heads", where), key_dim=_int(m, "dim", where),
                     value_dim=_int(m, "vdim", where), norm_eps=self.norm_eps)
        if kind == "gla":
            rank = _int(m, "decay_rank", where) if m.get("decay_rank") is not None else sizes["key_dim"]
            return GatedLinearSpec(decay_rank=rank, temperature=_number(m, "tau", where), **sizes)
        return MatrixMemorySpec(gate_cap=_number(m, "gate_cap", where), **sizes)

    def _ffn_spec(self, i: int):
        f = self.layers[i].get("mlp")
        if f is None:
            return None
        where = f"layers[{i}].mlp"
        if not isinstance(f, dict):
            raise ValueError(f"config.json: {where} must be null or an object")
        if f.get("kind") != "moe":
            raise ValueError(f"config.json: {where}.kind must be 'moe', got {f.get('kind')!r}")
        router, expert, rw = _object(f, "router", where), _object(f, "expert", where), where + ".router"
        shared = None
        if f.get("shared") is not None:
            shared = SwiGLUSpec(hidden=self.width, intermediate=_int(_object(f, "shared", where), "ff", where + ".shared"),
                                names={"gate": "mlp.shared.gate", "up": "mlp.shared.up", "down": "mlp.shared.down"})
        spec = ScoredMoESpec(hidden=self.width, experts=_int(router, "experts", rw),
                             identity=_int(router, "identity", rw, 0) if router.get("identity") is not None else 0,
                             top=_int(router, "top", rw), intermediate=_int(expert, "ff", where + ".expert"),
                             renormalize=True, shared=shared,
                             weight_scale=_number(router, "scale", rw) if router.get("scale") is not None else 1.0)
        if spec.top > spec.outputs:
            raise ValueError(f"config.json: {rw}.top exceeds the router's {spec.outputs} outputs")
        return spec

    # -- the model as parts --------------------------------------------------------
    def model_spec(self) -> ModelSpec:
        norm = NormSpec(width=self.width, eps=self.norm_eps, weight_name="", offset=1.0)
        blocks = []
        for i in range(len(self.layers)):
            mixer, ffn = self._mixer_spec(i), self._ffn_spec(i)
            behind = norm if ffn is not None else None
            blocks.append(BlockSpec(prefix=f"l{i}.", mixer=mixer, ffn=ffn, norm_in=norm, norm_post=behind,
                                    arrangement="sandwich", norm_in_out=norm, norm_post_out=behind, layer_scale=True,
                                    names={"norm_in": "norm1", "norm_in_out": "norm1b", "scale_in": "ls1",
                                           "norm_post": "norm2", "norm_post_out": "norm2b", "scale_post": "ls2"}))
        spec = ModelSpec(vocab=self.vocab, hidden=self.width, blocks=tuple(blocks),
                         schedule=tuple(ScheduleEntry(i) for i in range(len(blocks))), final_norm=norm, tie_embeddings=False,
                         embed_name="embed", final_norm_prefix="final.norm", head_name="head",
                         max_positions=DEFAULT_MAX_CONTEXT, stream_dtype="float32", logit_softcap=self.logit_softcap)
        spec.validate()
        return spec
