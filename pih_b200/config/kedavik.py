"""Typed configuration of the Kedavik design, read from its config.json keys.

A Kedavik model scales its embedding by one number, runs a list of pre-norm layers whose sub-layers' outputs are
multiplied by one number before they are added, and may run a stretch of the layers several times over with the same
tensors: every pass has caches and states of its own, every pass but the first adds the embedding output to the stream
once more, and every pass adds a learned vector of its own.  A layer's mixer is one of

* ``"mamba1"``: a selective scan behind a short convolution;
* ``"parallel"``: two mixers that read the same input, ``left_scale * left + right_scale * right``: softmax attention
  inside chunks of places (grouped key/value heads, a rotation in halves, a sigmoid gate a head), and a gated delta rule
  whose decay is one number a head and key channel and whose decay and output gate come through narrow projections;

and its feed-forward is dense (two matrices with biases around the error-function form of GELU) or absent.  config.json
holds::

    {"architecture": "Kedavik", "vocab": V, "width": W, "norm": {"eps": e}, "embedding": {"scale": s},
     "residual_mult": m, "loop": {"start": a, "stop": b, "times": n},
     "layers": [{"type": ..., "mixer": {...}, "mlp": {...} | null}, ...]}

The widths of the narrow projections are those of the tensors (``with_shapes``); ``decay_rank`` and ``gate_rank`` of the
right mixer say them where no weights exist yet.  The residual stream is summed in 32-bit.  Tensor names: ``embed``,
``head``, ``final.norm``, ``loop.step``, and ``l<i>.`` + ``norm1`` / ``norm2`` / ``mix.*`` (``mix.left.*``,
``mix.right.*``) / ``mlp.*`` (see the name tables of the part specs).
"""
from __future__ import annotations

import copy
from dataclasses import dataclass, field, fields
from typing import Optional, Tuple

from .registry import register_architecture
from .specs import (BiasedMLPSpec, BlockSpec, ComputedRopeSpec, GatedDeltaSpec, ModelSpec, NormSpec, ParallelSpec,
                    ScheduleEntry, SelectiveScanSpec, WindowAttentionSpec)
from .tuganex import DEFAULT_MAX_CONTEXT, _int, _number, _object


def _prefixed(spec_class, prefix: str) -> dict:
    """The default tensor names of a part spec with ``mix.`` replaced by ``prefix``."""
    names = next(f for f in fields(spec_class) if f.name == "names").default_factory()
    return {role: prefix + name[len("mix."):] for role, name in names.items()}


def _optional_number(d: dict, key: str, where: str, default: float) -> float:
    return _number(d, key, where, positive=False) if d.get(key) is not None else default


@register_architecture("Kedavik")
@dataclass(frozen=True)
class KedavikConfig:
    vocab: int
    width: int
    norm_eps: float
    embed_scale: float
    residual_mult: float
    loop: Optional[Tuple[int, int, int]]      # (start, stop, times)
    layers: Tuple[dict, ...] = field(default_factory=tuple)      # as in config.json, checked

    @classmethod
    def from_dict(cls, raw: dict) -> "KedavikConfig":
        norm = _object(raw, "norm", "config")
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ValueError("config.json: 'layers' must be a non-empty list")
        scale = 1.0
        if raw.get("embedding") is not None:
            scale = _optional_number(_object(raw, "embedding", "config"), "scale", "embedding", 1.0)
        loop = None
        if raw.get("loop") is not None:
            lp = _object(raw, "loop", "config")
            loop = (_int(lp, "start", "loop", 0), _int(lp, "stop", "loop"), _int(lp, "times", "loop"))
            if not loop[0] < loop[1] <= len(layers):
                raise ValueError(f"config.json: loop must name layers start < stop <= {len(layers)}")
        cfg = cls(vocab=_int(raw, "vocab", "config"), width=_int(raw, "width", "config"),
                  norm_eps=_number(norm, "eps", "norm"), embed_scale=scale,
                  residual_mult=_optional_number(raw, "residual_mult", "config", 1.0), loop=loop,
                  layers=tuple(copy.deepcopy(layers)))
        cfg.model_spec()                      # every layer's keys and sizes are checked by building its spec
        return cfg

    def to_dict(self) -> dict:
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
               "norm": {"eps": self.norm_eps}, "embedding": {"scale": self.embed_scale},
               "residual_mult": self.residual_mult, "layers": copy.deepcopy(list(self.layers))}
        if self.loop is not None:
            out["loop"] = {"start": self.loop[0], "stop": self.loop[1], "times": self.loop[2]}
        return out

    def with_shapes(self, shapes) -> "KedavikConfig":
        """The configuration with the sizes that only the tensors' shapes give: the widths of the narrow projections in
        front of the decays (``a1``) and the output gate (``g1``) of a right mixer."""
        layers = copy.deepcopy(list(self.layers))
        for i, layer in enumerate(layers):
            if layer.get("type") != "parallel":
                continue
            for key, name in (("decay_rank", "a1"), ("gate_rank", "g1")):
                shape = shapes.get(f"l{i}.mix.right.{name}")
                if shape is not None and len(shape) == 2:
                    layer["mixer"]["right"][key] = int(shape[0])
        return KedavikConfig(self.vocab, self.width, self.norm_eps, self.embed_scale, self.residual_mult, self.loop,
                             tuple(layers))

    # -- layers -----------------------------------------------------------------
    def _scan(self, m: dict, where: str) -> SelectiveScanSpec:
        return SelectiveScanSpec(hidden=self.width, inner=_int(m, "inner", where), state=_int(m, "state", where),
                                 dt_rank=_int(m, "dt_rank", where), conv_taps=_int(m, "conv", where))

    def _heads(self, m: dict, where: str):
        heads, kv_heads = _int(m, "heads", where), _int(m, "kv_heads", where)
        if heads % kv_heads:
            raise ValueError(f"config.json: {where}.heads must be a multiple of kv_heads")
        return dict(hidden=self.width, heads=heads, kv_heads=kv_heads, key_dim=_int(m, "dim", where),
                    value_dim=_int(m, "vdim", where))

    def _attention(self, m: dict, where: str) -> WindowAttentionSpec:
        sizes = self._heads(m, where)
        position = None
        if m.get("rot") is not None:
            rot = _object(m, "rot", where)
            dims = _int(rot, "dims", where + ".rot", minimum=2)
            if dims % 2 or dims > sizes["key_dim"]:
                raise ValueError(f"config.json: {where}.rot.dims must be even and at most dim, got {dims}")
            position = ComputedRopeSpec(head_dim=sizes["key_dim"], rotary_dim=dims,
                                        theta=_number(rot, "base", where + ".rot"))
        chunk = 0
        if m.get("mask") is not None:
            chunk = _int(_object(m, "mask", where), "size", where + ".mask")
        return WindowAttentionSpec(scale=_number(m, "scale", where, positive=False), window=0, chunk=chunk,
                                   position=position, sink="none", head_gate=True,
                                   names=_prefixed(WindowAttentionSpec, "mix.left."), **sizes)

    def _delta(self, m: dict, where: str) -> GatedDeltaSpec:
        sizes = self._heads(m, where)

        def rank(key):
            return _int(m, key, where) if m.get(key) is not None else sizes["key_dim"]

        return GatedDeltaSpec(conv_taps=_int(m, "conv", where), norm_eps=self.norm_eps, decay_per="channel",
                              decay_rank=rank("decay_rank"), gate_rank=rank("gate_rank"), gate_activation="sigmoid",
                              names=_prefixed(GatedDeltaSpec, "mix.right."), **sizes)

    def _mixer_spec(self, i: int):
        layer = self.layers[i]
        if not isinstance(layer, dict):
            raise ValueError(f"config.json: layers[{i}] must be an object")
        where = f"layers[{i}].mixer"
        kind = layer.get("type")
        if kind not in ("mamba1", "parallel"):
            raise ValueError(f"config.json: layers[{i}].type must be 'mamba1' or 'parallel', got {kind!r}")
        m = _object(layer, "mixer", f"layers[{i}]")
        if kind == "mamba1":
            return self._scan(m, where)
        return ParallelSpec(left=self._attention(_object(m, "left", where), where + ".left"),
                            right=self._delta(_object(m, "right", where), where + ".right"),
                            left_scale=_number(m, "left_scale", where, positive=False),
                            right_scale=_number(m, "right_scale", where, positive=False))

    def _ffn_spec(self, i: int):
        f = self.layers[i].get("mlp")
        if f is None:
            return None
        where = f"layers[{i}].mlp"
        if not isinstance(f, dict):
            raise ValueError(f"config.json: {where} must be null or an object")
        if f.get("kind") != "dense":
            raise ValueError(f"config.json: {where}.kind must be 'dense', got {f.get('kind')!r}")
        return BiasedMLPSpec(hidden=self.width, intermediate=_int(f, "ff", where), activation="gelu_erf")

    # -- the model as parts --------------------------------------------------------
    def schedule(self):
        n = len(self.layers)
        if self.loop is None:
            return tuple(ScheduleEntry(i) for i in range(n))
        a, b, times = self.loop
        return (tuple(ScheduleEntry(i) for i in range(a))
                + tuple(ScheduleEntry(i, add_embedding=i == a and t > 0, add_vector=t if i == a else None)
                        for t in range(times) for i in range(a, b))
                + tuple(ScheduleEntry(i) for i in range(b, n)))

    def model_spec(self) -> ModelSpec:
        norm = NormSpec(width=self.width, eps=self.norm_eps, weight_name="")
        blocks = []
        for i in range(len(self.layers)):
            mixer, ffn = self._mixer_spec(i), self._ffn_spec(i)
            blocks.append(BlockSpec(prefix=f"l{i}.", mixer=mixer, ffn=ffn, norm_in=norm,
                                    norm_post=norm if ffn is not None else None,
                                    names={"norm_in": "norm1", "norm_post": "norm2"}, residual_scale=self.residual_mult))
        spec = ModelSpec(vocab=self.vocab, hidden=self.width, blocks=tuple(blocks), schedule=self.schedule(),
                         final_norm=norm, tie_embeddings=False, embed_name="embed", final_norm_prefix="final.norm",
                         head_name="head", max_positions=DEFAULT_MAX_CONTEXT, stream_dtype="float32",
                         embed_scale=self.embed_scale, vectors_name="loop.step" if self.loop is not None else None,
                         vectors=self.loop[2] if self.loop is not None else 0)
        spec.validate()
        return spec
