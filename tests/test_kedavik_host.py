"""Host-side logic of the Kedavik design without a GPU: configuration, tensor names, sizes that only the tensors give, the
loop's caches and states, pages of finished chunks, two mixers side by side, and the real parts, cache manager and step
function over stand-in kernels (tests/fake_ops.py) against the plain float64 restatement."""
import copy
import json
import math
import os

import pytest
import torch

import kedavik_models as km
import plain_kedavik as plain
import traces
from fake_ops import FakeOps


def _runner(folder, dtype="float32", **kw):
    from pih_b200.engine.factory import create_runner
    kw = {"page_size": 4, "max_cache_tokens": 64, "max_requests": 1, **kw}
    return create_runner(folder, dtype, device="cpu", ops=FakeOps(), **kw)


def test_configuration_to_parts():
    from pih_b200.config import config_from_dict
    cfg = config_from_dict(copy.deepcopy(km.K1))
    spec = cfg.model_spec()
    assert cfg.architecture == "Kedavik" and spec.stream_dtype == "float32" and not spec.tie_embeddings
    assert spec.embed_scale == 0.7 and (spec.vectors_name, spec.vectors) == ("loop.step", 3)
    assert [b.arrangement for b in spec.blocks] == ["prenorm"] * 4 and {b.residual_scale for b in spec.blocks} == {0.45}
    assert [b.mixer.kind for b in spec.blocks] == ["selective_scan", "parallel", "selective_scan", "parallel"]
    assert [e.layer for e in spec.schedule] == [0, 1, 2, 1, 2, 1, 2, 3]
    assert [e.add_embedding for e in spec.schedule] == [False] * 3 + [True, False, True, False, False]
    assert [e.add_vector for e in spec.schedule] == [None, 0, None, 1, None, 2, None, None]
    m = spec.blocks[1].mixer
    assert (m.left_scale, m.right_scale) == (0.7, 1.3) and (m.left.kind, m.right.kind) == ("window_attention", "gated_delta")
    assert m.left.chunk == 20 and m.left.window == 0 and m.left.head_gate and m.left.sink == "none" and m.left.scale == 0.3
    assert m.left.norm_eps is None and m.left.position.rotary_dim == 8 and not m.left.position.interleaved
    r = m.right
    assert (r.decay_per, r.decay_rank, r.gate_rank, r.gate_activation, r.conv_taps) == ("channel", 10, 14, "sigmoid", 3)
    assert r.decays == 64 and r.norm_eps == 1e-5 and r.unit_eps == 1e-6
    assert spec.blocks[0].ffn is None and spec.blocks[1].ffn.activation == "gelu_erf" and spec.blocks[1].ffn.intermediate == 100
    assert spec.blocks[3].ffn is None and spec.blocks[2].ffn is not None
    assert config_from_dict(cfg.to_dict()) == cfg
    plain_spec = config_from_dict(copy.deepcopy(km.K3)).model_spec()               # what the configuration leaves out
    assert plain_spec.embed_scale == 1.0 and plain_spec.vectors_name is None and plain_spec.blocks[0].residual_scale == 1.0
    assert plain_spec.blocks[2].mixer.left.chunk == 0 and plain_spec.blocks[2].mixer.left.position is None
    first = config_from_dict(copy.deepcopy(km.K2)).model_spec().schedule          # a loop of all layers
    assert [(e.layer, e.add_embedding, e.add_vector) for e in first] == [
        (0, False, 0), (1, False, None), (2, False, None), (0, True, 1), (1, False, None), (2, False, None)]


def test_tensor_names():
    from pih_b200.config import config_from_dict
    from pih_b200.models import expected_tensors
    names = {n: i.shape for n, i in expected_tensors(config_from_dict(copy.deepcopy(km.K1)).model_spec()).items()}
    assert names["embed"] == names["head"] == (307, 72) and names["loop.step"] == (3, 72) and names["final.norm"] == (72,)
    assert {n[3:]: s for n, s in names.items() if n.startswith("l0.")} == {
        "norm1": (72,), "mix.in": (176, 72), "mix.conv": (88, 4), "mix.conv.b": (88,), "mix.x": (16, 88), "mix.dt": (88, 6),
        "mix.dt.b": (88,), "mix.A_log": (88, 5), "mix.D": (88,), "mix.o": (72, 88)}
    assert {n[3:]: s for n, s in names.items() if n.startswith("l1.")} == {
        "norm1": (72,), "norm2": (72,), "mlp.up": (100, 72), "mlp.up.b": (100,), "mlp.down": (72, 100), "mlp.down.b": (72,),
        "mix.left.q": (64, 72), "mix.left.k": (32, 72), "mix.left.v": (48, 72), "mix.left.g": (4, 72), "mix.left.o": (72, 96),
        "mix.right.q": (32, 72), "mix.right.k": (32, 72), "mix.right.v": (48, 72), "mix.right.q.conv": (32, 3),
        "mix.right.k.conv": (32, 3), "mix.right.v.conv": (48, 3), "mix.right.b": (4, 72), "mix.right.A_log": (4,),
        "mix.right.dt_bias": (64,), "mix.right.norm": (12,), "mix.right.a1": (10, 72), "mix.right.a2": (64, 10),
        "mix.right.g1": (14, 72), "mix.right.g2": (48, 14), "mix.right.o": (72, 48)}
    assert "loop.step" not in expected_tensors(config_from_dict(copy.deepcopy(km.K3)).model_spec())


@pytest.mark.parametrize("change, message", [
    (lambda c: c["layers"][0].update(type="mamba2"), "type"),
    (lambda c: c["layers"][0]["mixer"].pop("state"), "state"),
    (lambda c: c["layers"][1]["mixer"].pop("left"), "left"),
    (lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=3), "kv_heads"),
    (lambda c: c["layers"][1]["mixer"]["right"].update(heads=3), "kv_heads"),
    (lambda c: c["layers"][1]["mixer"]["left"]["rot"].update(dims=18), "dims"),
    (lambda c: c["layers"][1]["mixer"]["left"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][1]["mixer"].update(right_scale=None), "right_scale"),
    (lambda c: c["layers"][1]["mlp"].update(kind="moe"), "kind"),
    (lambda c: c["loop"].update(stop=5), "loop"),
    (lambda c: c["loop"].update(start=3), "loop"),
    (lambda c: c["loop"].update(times=0), "times"),
    (lambda c: c.pop("norm"), "norm"),
])
def test_configuration_errors(change, message):
    from pih_b200.config import config_from_dict
    raw = copy.deepcopy(km.K1)
    change(raw)
    with pytest.raises(ValueError, match=message):
        config_from_dict(raw)


def test_narrow_widths_come_from_the_tensors(tmp_path):
    """A configuration that does not say how wide the narrow projections are: the weight file's tensors do."""
    folder = km.write_model(tmp_path / "m", km.K2, seed=3, sigma=0.15)
    path = os.path.join(folder, "config.json")
    with open(path) as f:
        raw = json.load(f)
    for lay in raw["layers"]:
        for key in ("decay_rank", "gate_rank"):
            lay["mixer"].get("right", {}).pop(key, None)
    with open(path, "w") as f:
        json.dump(raw, f)
    config, model, _, runner = _runner(folder)
    assert [(b.mixer.spec.right.decay_rank, b.mixer.spec.right.gate_rank) for b in model.blocks
            if b.mixer.spec.kind == "parallel"] == [(5, 7), (33, 4)]
    requests = {"r0": traces.make_requests(259, [11], seed=1)["r0"]}
    got = traces.replay(runner, traces.whole(requests))["r0"]
    ref = km.plain_logits(folder, requests)["r0"]
    assert float((got.double() - ref).abs().max()) < 2e-4 * float(ref.abs().max())


def test_only_a_pre_norm_layer_on_a_wide_stream_takes_additions_and_factors():
    from dataclasses import replace
    from pih_b200.config import ScheduleEntry, config_from_dict
    spec = config_from_dict(copy.deepcopy(km.K1)).model_spec()
    for bad in (replace(spec, stream_dtype=None), replace(spec, vectors=2),
                replace(spec, blocks=tuple(replace(b, arrangement="outnorm") for b in spec.blocks)),
                replace(spec, schedule=spec.schedule + (ScheduleEntry(0, add_vector=7),)),
                replace(spec, streams=2)):
        with pytest.raises(ValueError):
            bad.validate()


def test_two_mixers_side_by_side_must_fit():
    """Mixers that do not show their products, or that both want pages, are refused; tensor names must not meet."""
    from pih_b200.config import AttentionSpec, ParallelSpec, RetentionSpec, WindowAttentionSpec
    from pih_b200.parts import Runtime, part_class
    from pih_b200.weights import random_tensors
    cls = part_class("mixer", "parallel")
    rt = Runtime(torch.device("cpu"), torch.float32, FakeOps())
    win = dict(hidden=8, heads=1, kv_heads=1, key_dim=4, value_dim=4, scale=1.0, window=3, sink="none")
    left = WindowAttentionSpec(**win, names=dict(q="a.q", k="a.k", v="a.v", o="a.o"))
    right = WindowAttentionSpec(**win, names=dict(q="b.q", k="b.k", v="b.v", o="b.o"))

    def build(spec):
        return cls(spec, random_tensors(cls.expected_tensors(spec), 1, dtype=torch.float32), rt)

    with pytest.raises(ValueError, match="paged"):
        build(ParallelSpec(left, right))
    with pytest.raises(ValueError, match="same tensors"):
        cls.expected_tensors(ParallelSpec(left, left))
    with pytest.raises(TypeError, match="side|beside"):
        build(ParallelSpec(left, AttentionSpec(hidden=8, heads=1, kv_heads=1, head_dim=4, scale=1.0, qk_norm_eps=None,
                                               window=None, position=None)))
    ret = RetentionSpec(hidden=8, heads=1, key_dim=4, value_dim=6, decays=(0.9,), key_scale=0.5, norm_eps=1e-5, position=None,
                        names=dict(q="c.q", k="c.k", v="c.v", gate="c.g", o="c.o"))
    both = build(ParallelSpec(left, ret))                   # any two that show their products go together
    assert both.cache_need().paged.width == 8 and both.cache_need().state.shape == (24,) and both.w_o.shape == (8, 10)
    assert both.in_at == [0, 32] and bool((both.w_in[12:32] == 0).all())
    assert both.parts[0].w_in.data_ptr() == both.w_in.data_ptr()


def test_the_order_of_layers_by_hand():
    assert plain.runs({"layers": [0] * 4, "loop": {"start": 1, "stop": 3, "times": 2}}) == [
        (0, None, False), (1, 0, True), (2, 0, False), (1, 1, True), (2, 1, False), (3, None, False)]
    assert plain.runs({"layers": [0] * 2}) == [(0, None, False), (1, None, False)]


def test_plain_mechanisms_by_hand():
    """Chunk edges; the exact GELU; one token of the scan and of the delta rule; a channel's decay acts on the row of the
    state that belongs to that key channel."""
    assert [plain.chunk_start(p, 5) for p in (0, 4, 5, 9, 10, 23)] == [0, 0, 5, 5, 10, 20]
    z = torch.tensor([-1.0, 0.0, 2.0], dtype=torch.float64)
    assert float((plain.gelu(z) - torch.tensor([-0.15865525, 0.0, 1.95449974], dtype=torch.float64)).abs().max()) < 1e-8
    one = lambda *v: torch.tensor([v], dtype=torch.float64)
    y, S = plain.selective_scan(one(3.0), one(0.5), torch.tensor([[-1.0, -2.0]], dtype=torch.float64), one(1.0, 2.0),
                                one(4.0, 0.5), torch.tensor([10.0], dtype=torch.float64),
                                torch.tensor([[1.0, 1.0]], dtype=torch.float64))
    s = (math.exp(-0.5) + 1.5, math.exp(-1.0) + 3.0)
    assert abs(float(S[0, 0]) - s[0]) < 1e-12 and abs(float(S[0, 1]) - s[1]) < 1e-12
    assert abs(float(y) - (4.0 * s[0] + 0.5 * s[1] + 30.0)) < 1e-12
    S0 = torch.tensor([[[2.0], [6.0]]], dtype=torch.float64)                       # one head, two key channels, one value
    q = torch.tensor([[[1.0, 1.0]]], dtype=torch.float64)
    k = torch.tensor([[[1.0, 0.0]]], dtype=torch.float64)
    o, S1 = plain.delta_rule(q, k, torch.tensor([[[5.0]]], dtype=torch.float64), torch.tensor([[[0.5, 0.25]]], dtype=torch.float64),
                             torch.tensor([[0.5]], dtype=torch.float64), S0)
    # the rows decay to 1 and 1.5; the first is moved half of the way to 5
    assert S1.flatten().tolist() == [3.0, 1.5] and float(o) == 4.5


def test_the_plain_implementation_cut_in_two():
    """The oracle itself: a sequence fed in parts through its state gives what it gives whole."""
    from pih_b200.config import config_from_dict
    from pih_b200.models import expected_tensors
    for name, cfg in km.CONFIGS.items():
        g = torch.Generator().manual_seed(0)
        w = {n: torch.randn(i.shape, generator=g, dtype=torch.float64) * 0.3
             for n, i in expected_tensors(config_from_dict(copy.deepcopy(cfg)).model_spec()).items()}
        toks = traces.make_requests(cfg["vocab"], [21], seed=1)["r0"]
        _, whole, _ = plain.model_layers(cfg, w, toks)
        parts, st = [], None
        for a, b in ((0, 13), (13, 15), (15, 16), (16, 21)):
            _, y, st = plain.model_layers(cfg, w, toks[a:b], st)
            parts.append(y)
        assert float((torch.cat(parts) - whole).abs().max()) < 1e-9, name


@pytest.mark.parametrize("name", ["K1", "K2", "K3"])
@pytest.mark.parametrize("family", ["whole", "portions", "mixed"])
def test_cut_invariance_with_stand_in_kernels(tmp_path, name, family):
    """Block tables, slot mappings, state slots, the states and caches of each pass of the loop and their reuse: the real
    parts and step function with torch stand-ins for the kernels agree with the plain implementation however the
    requests are cut."""
    d = km.write_model(tmp_path / name, km.CONFIGS[name], seed=1, sigma=km.SIGMA[name])
    requests = traces.make_requests(km.CONFIGS[name]["vocab"], [19, 6, 58, 1, 12], seed=3)
    kw = dict(max_live=2, decode_tail=3, max_portion=7) if family == "mixed" else {}
    steps = getattr(traces, family)(requests, **kw)
    _, model, cache, runner = _runner(d, max_cache_tokens=traces.peak_tokens(steps, round_to=4), max_requests=2)
    # every pass has pages and states of its own
    order = plain.runs(km.CONFIGS[name])
    kinds = [km.CONFIGS[name]["layers"][i]["type"] for i, _, _ in order]
    assert len(cache.state_tensors) == len(order) and sum(len(g.entries) for g in cache.groups) == kinds.count("parallel")
    got = traces.replay(runner, steps)
    for rid, ref in km.plain_logits(d, requests).items():
        assert float((got[rid].double() - ref).abs().max()) < 2e-4 * float(ref.abs().max()), (family, rid)
    cache.check()
    assert cache.slots.num_free == 2 and all(f == cache.num_pages for f in cache.num_free_pages())
    if family == "mixed":
        assert all(g.pool.pages_handed_out > g.pool.num_pages for g in cache.groups)


def test_pages_of_finished_chunks_go_back(tmp_path):
    """A request far longer than the chunks holds, at any time, only pages of the chunk that its next token lies in (a
    page on the border belongs to both): a cache pool much smaller than the request is enough."""
    from pih_b200.engine import StepEntry
    d = km.write_model(tmp_path / "m", km.K1, seed=2, sigma=0.15)
    toks = traces.make_requests(307, [130], seed=4)["r0"]
    _, model, cache, runner = _runner(d, max_cache_tokens=48)
    assert sorted(g.need.chunk for g in cache.groups) == [20, 37]
    got, at = [], 0
    for n in [7, 13, 1, 19, 2, 6, 12, 1, 1, 15, 3, 17, 6, 5, 9, 13]:
        got.append(runner.step([StepEntry("a", toks[at:at + n], list(range(n)))]).clone())
        at += n
        for g in cache.groups:
            first = at - at % g.need.chunk
            held = g.pool.num_pages - g.pool.num_free
            assert held == -(-at // 4) - first // 4, (at, g.need.chunk, held)
    assert at == 130
    ref = km.plain_logits(d, {"a": toks})["a"]
    assert float((torch.cat(got).double() - ref).abs().max()) < 2e-4 * float(ref.abs().max())


def test_a_failed_step_leaves_the_states_as_they_were(tmp_path):
    """A step that raises after the layers have advanced their states (scan, delta rule, convolutions) is rolled back."""
    from pih_b200.engine import StepEntry
    d = km.write_model(tmp_path / "m", km.K2, seed=2, sigma=0.15)
    toks = traces.make_requests(259, [14], seed=1)["r0"]
    _, model, cache, runner = _runner(d, max_cache_tokens=32)
    runner.step([StepEntry("a", toks[:9], [])])
    head = model.head
    model.head = None                                   # the head product fails, after every layer has run
    with pytest.raises(Exception):
        runner.step([StepEntry("a", toks[9:], [4])])
    model.head = head
    again = runner.step([StepEntry("a", toks[9:], [4])])
    ref = km.plain_logits(d, {"a": toks})["a"][-1]
    assert float((again[0].double() - ref).abs().max()) < 2e-4 * float(ref.abs().max())


@pytest.mark.parametrize("seed", range(6))
def test_configurations_drawn_at_random_with_stand_in_kernels(tmp_path, seed):
    raw = km.random_config(seed)
    d = km.write_model(tmp_path / "m", raw, seed=seed, sigma=0.15)
    requests = traces.make_requests(raw["vocab"], [23, 9, 1, 14], seed=seed)
    steps = traces.mixed(requests, seed=seed, max_live=2, decode_tail=3, max_portion=6)
    _, model, cache, runner = _runner(d, max_cache_tokens=traces.peak_tokens(steps, round_to=4), max_requests=2)
    got = traces.replay(runner, steps)
    for rid, ref in km.plain_logits(d, requests).items():
        assert float((got[rid].double() - ref).abs().max()) < 3e-4 * max(1.0, float(ref.abs().max())), rid
    cache.check()


def test_the_stream_stays_wide_in_bfloat16(tmp_path):
    """bfloat16 over stand-in kernels that round after each step: the stream, the factors and what the loop adds stay
    32-bit, and the logits are within rounding of the plain implementation."""
    d = km.write_model(tmp_path / "m", km.K1, seed=4, sigma=0.15)
    requests = traces.make_requests(307, [31, 5], seed=3)
    _, model, cache, runner = _runner(d, "bfloat16", max_cache_tokens=48, max_requests=2)
    seen = set()
    ops = model.rt.ops
    inner = ops.rmsnorm_stream
    ops.rmsnorm_stream = lambda h, *a, **kw: (seen.add(h.dtype), inner(h, *a, **kw))[1]
    got = traces.replay(runner, traces.portions(requests))
    assert seen == {torch.float32}
    for rid, ref in km.plain_logits(d, requests).items():
        err = (got[rid].double() - ref).pow(2).mean().sqrt() / ref.std()
        assert float(err) < 0.05, (rid, float(err))


def test_memory_for_pages_and_states():
    """The engine's sizing counts the pages of a layer that keeps pages AND a state, and the state slots."""
    from types import SimpleNamespace
    from pih_b200.config import config_from_dict
    from pih_b200.engine.factory import cache_tokens_for_memory
    from pih_b200.models import CausalLM, expected_tensors
    from pih_b200.parts import Runtime
    from pih_b200.weights import random_tensors
    spec = config_from_dict(copy.deepcopy(km.K1)).model_spec()
    model = CausalLM(spec, random_tensors(expected_tensors(spec), seed=1), Runtime(torch.device("cpu"), torch.bfloat16, FakeOps()))
    # bytes a token: three passes of the first pair (2 x 16 + 2 x 24 numbers) and the second pair (24 + 40), two bytes each
    per_token = 2 * (3 * (2 * 16 + 2 * 24) + (24 + 40))
    fit = lambda free: cache_tokens_for_memory(model, page_size=16, max_requests=1000, max_batch_tokens=64, max_context=1 << 14,
                                               free_and_total=(free, free))
    a, b = fit(4 << 30), fit(4 << 30 | 1 << 28)
    assert b > a and abs((b - a) - 0.9 * (1 << 28) / per_token) <= 16
