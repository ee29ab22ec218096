"""Host-side logic of the Bipulorn design without a GPU: configuration, tensor names, sizes that only the tensors give, the
norms before and behind the sub-layers, two normed mixers side by side, pages behind the window, state slots, and the real
parts, cache manager and step function over stand-in kernels (tests/fake_ops.py) against the plain float64 restatement."""
import copy
import json
import math
import os

import pytest
import torch

import bipulorn_models as bm
import plain_bipulorn as plain
import traces
from fake_ops import FakeOps


def _runner(folder, dtype="float32", **kw):
    from pih_b200.engine.factory import create_runner
    kw = {"page_size": 4, "max_cache_tokens": 64, "max_requests": 1, **kw}
    return create_runner(folder, dtype, device="cpu", ops=FakeOps(), **kw)


def test_configuration_to_parts():
    from pih_b200.config import config_from_dict
    cfg = config_from_dict(copy.deepcopy(bm.B1))
    spec = cfg.model_spec()
    assert cfg.architecture == "Bipulorn" and spec.stream_dtype == "float32" and not spec.tie_embeddings
    assert spec.logit_softcap == 20.0 and spec.final_norm.offset == 1.0
    assert [b.arrangement for b in spec.blocks] == ["sandwich"] * 4 and all(b.layer_scale for b in spec.blocks)
    assert [b.mixer.kind for b in spec.blocks] == ["parallel", "gated_linear", "matrix_memory", "parallel"]
    m = spec.blocks[0].mixer
    assert (m.left_scale, m.right_scale, m.out_norm_eps) == (0.5, 0.5, 1e-5)
    left, right = m.left, m.right
    assert left.window == 21 and left.chunk == 0 and left.column_gate and not left.head_gate and left.biases and left.sink == "none"
    assert left.scale == 0.3 and left.norm_eps is None
    assert left.position.interleaved and left.position.rotary_dim == 8 and left.position.slowdown == 3.0
    assert (right.heads, right.value_dim, right.state, right.groups, right.norm_groups, right.conv_taps) == (6, 16, 24, 3, 4, 4)
    assert right.inner == 96 and right.bc_size == 72 and right.norm_eps == 1e-5
    g = spec.blocks[1].mixer
    assert (g.heads, g.key_dim, g.value_dim, g.temperature, g.decay_rank) == (3, 16, 40, 8.0, 10)
    assert spec.blocks[2].mixer.gate_cap == 9.0 and spec.blocks[2].mixer.floor == 1e-6
    assert spec.blocks[2].ffn is None and spec.blocks[2].norm_post_out is None and spec.blocks[2].norm_in_out is not None
    f = spec.blocks[0].ffn
    assert (f.experts, f.identity, f.top, f.intermediate, f.weight_scale, f.renormalize, f.scoring) == (5, 3, 2, 24, 1.7, True, "softmax")
    assert f.shared.intermediate == 40 and f.shared_gate and f.correction and f.gated
    assert config_from_dict(cfg.to_dict()) == cfg
    bare = config_from_dict(copy.deepcopy(bm.B3)).model_spec()                   # what the configuration leaves out
    assert bare.logit_softcap is None and bare.blocks[3].mixer.left.window == 0 and bare.blocks[3].mixer.left.position is None
    assert bare.blocks[1].ffn.identity == 0 and bare.blocks[1].ffn.weight_scale == 1.0 and bare.blocks[1].ffn.shared is None


def test_tensor_names():
    from pih_b200.config import config_from_dict
    from pih_b200.models import expected_tensors
    names = {n: i.shape for n, i in expected_tensors(config_from_dict(copy.deepcopy(bm.B1)).model_spec()).items()}
    assert names["embed"] == names["head"] == (311, 72) and names["final.norm"] == (72,)
    frame = {n: (72,) for n in ("norm1", "norm1b", "ls1", "norm2", "norm2b", "ls2")}
    expert = lambda n, ff: {f"mlp.{n}.gate": (ff, 72), f"mlp.{n}.up": (ff, 72), f"mlp.{n}.down": (72, ff)}
    want = {**frame, "mix.left.q": (64, 72), "mix.left.k": (32, 72), "mix.left.v": (48, 72), "mix.left.g": (96, 72),
            "mix.left.o": (72, 96), "mix.left.q.b": (64,), "mix.left.k.b": (32,), "mix.left.v.b": (48,), "mix.left.o.b": (72,),
            "mix.right.in": (96 + 96 + 144 + 6, 72), "mix.right.conv": (240, 4), "mix.right.conv.b": (240,),
            "mix.right.dt_bias": (6,), "mix.right.A_log": (6,), "mix.right.D": (6,), "mix.right.norm": (96,),
            "mix.right.o": (72, 96), "mix.left.out": (72,), "mix.right.out": (72,), "mlp.router": (8, 72),
            "mlp.correction": (8,), "mlp.shared.sg": (1, 72), **expert("shared", 40)}
    for e in range(5):
        want.update(expert(f"e{e}", 24))
    assert {n[3:]: s for n, s in names.items() if n.startswith("l0.")} == want
    assert {n[3:]: s for n, s in names.items() if n.startswith("l1.") and "mlp" not in n} == {
        **frame, "mix.q": (48, 72), "mix.k": (48, 72), "mix.v": (120, 72), "mix.g": (120, 72), "mix.o": (72, 120),
        "mix.norm": (40,), "mix.a1": (10, 72), "mix.a2": (48, 10), "mix.a2.b": (48,)}
    assert {n[3:]: s for n, s in names.items() if n.startswith("l2.")} == {
        "norm1": (72,), "norm1b": (72,), "ls1": (72,), "mix.q": (48, 72), "mix.k": (48, 72), "mix.v": (32, 72), "mix.g": (32, 72),
        "mix.o": (72, 32), "mix.norm": (32,), "mix.i": (2, 72), "mix.i.b": (2,), "mix.f": (2, 72), "mix.f.b": (2,)}


@pytest.mark.parametrize("change, message", [
    (lambda c: c["layers"][0].update(type="mamba2"), "type"),
    (lambda c: c["layers"][1]["mixer"].pop("tau"), "tau"),
    (lambda c: c["layers"][2]["mixer"].update(gate_cap=0), "gate_cap"),
    (lambda c: c["layers"][0]["mixer"].pop("left"), "left"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3), "kv_heads"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(groups=4), "groups"),
    (lambda c: c["layers"][0]["mixer"]["right"].update(norm_groups=5), "norm_groups"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=18), "dims"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(scaling={"factor": 0}), "factor"),
    (lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "kind"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=9), "top"),
    (lambda c: c.update(logit_softcap=-1.0), "logit_softcap"),
    (lambda c: c.pop("norm"), "norm"),
])
def test_configuration_errors(change, message):
    from pih_b200.config import config_from_dict
    raw = copy.deepcopy(bm.B1)
    change(raw)
    with pytest.raises(ValueError, match=message):
        config_from_dict(raw)


def test_narrow_widths_come_from_the_tensors(tmp_path):
    """A configuration that does not say how wide the narrow projection is: the weight file's tensor does."""
    folder = bm.write_model(tmp_path / "m", bm.B2, seed=3, sigma=0.15)
    path = os.path.join(folder, "config.json")
    with open(path) as f:
        raw = json.load(f)
    raw["layers"][2]["mixer"].pop("decay_rank")
    with open(path, "w") as f:
        json.dump(raw, f)
    _, model, _, runner = _runner(folder)
    assert model.blocks[2].mixer.spec.decay_rank == 33
    requests = {"r0": traces.make_requests(263, [11], seed=1)["r0"]}
    got = traces.replay(runner, traces.whole(requests))["r0"]
    ref = bm.plain_logits(folder, requests)["r0"]
    assert float((got.double() - ref).abs().max()) < 2e-4 * float(ref.abs().max())


def test_parts_that_do_not_fit_are_refused():
    """Norms on a pair's outputs need a block that adds pairs; a layer with norms behind its sub-layers needs a wide stream
    and one norm a sub-layer; a layer over several streams takes no output bias; one kind of gate at a time."""
    from dataclasses import replace
    from pih_b200.config import HyperSpec, config_from_dict
    from pih_b200.parts import Runtime, part_class
    from pih_b200.weights import random_tensors
    spec = config_from_dict(copy.deepcopy(bm.B1)).model_spec()
    with pytest.raises(ValueError):
        replace(spec, stream_dtype=None).validate()
    with pytest.raises(ValueError):
        replace(spec, logit_softcap=0.0).validate()
    rt = Runtime(torch.device("cpu"), torch.float32, FakeOps())

    def build(block):
        cls = part_class("block", block.arrangement)
        return cls(block, random_tensors(cls.expected_tensors(block), 1, dtype=torch.float32), rt)

    block = spec.blocks[0]
    assert build(block).mixer.pairs
    with pytest.raises(ValueError, match="names one of each"):
        build(replace(block, norm_post_out=None))
    with pytest.raises(TypeError, match="forward_pair"):
        build(block).mixer.forward(torch.zeros(1, 72), None, None)
    left = replace(block.mixer.left, names=block.mixer.left.names)
    with pytest.raises(TypeError, match="bias"):
        build(replace(block, arrangement="hyper", mixer=left, hyper=HyperSpec(streams=2)))
    with pytest.raises(ValueError, match="gate"):
        build(replace(block, mixer=replace(left, head_gate=True)))


def test_a_pair_without_norms_hands_its_biases_on(tmp_path):
    """The attention's output bias reaches the stream through every arrangement: alone and in a pair that is scaled and
    added, in layers with norms in front and with norms behind."""
    from dataclasses import replace
    from pih_b200.config import BlockSpec, config_from_dict
    from pih_b200.engine import StepEntry
    from pih_b200.engine.factory import runner_for
    from pih_b200.models import CausalLM, expected_tensors
    from pih_b200.parts import Runtime
    from pih_b200.weights import random_tensors
    spec = config_from_dict(copy.deepcopy(bm.B1)).model_spec()
    pair = replace(spec.blocks[0].mixer, out_norm_eps=None, left_scale=0.7, right_scale=1.2)
    norm = replace(spec.final_norm, offset=0.0)
    toks = traces.make_requests(311, [9], seed=1)["r0"]
    for mixer in (pair, pair.left):
        for arrangement in ("prenorm", "outnorm"):
            block = BlockSpec(prefix="l0.", mixer=mixer, ffn=None, norm_in=norm, norm_post=None, arrangement=arrangement,
                              names={"norm_in": "norm1", "norm_post": "norm2"})
            s = replace(spec, blocks=(block,), schedule=spec.schedule[:1], logit_softcap=None)
            w = random_tensors(expected_tensors(s), 5, sigma=0.2, dtype=torch.float32)
            model = CausalLM(s, w, Runtime(torch.device("cpu"), torch.float32, FakeOps()))
            _, runner = runner_for(model, page_size=4, max_cache_tokens=16, max_requests=1)
            got = runner.step([StepEntry("a", toks, list(range(9)))]).double()
            d = {n: t.double() for n, t in w.items()}
            raw = bm.B1["layers"][0]["mixer"]
            x = d["embed"][torch.tensor(toks)]
            h = x if arrangement == "outnorm" else plain.rms_unit(x, 1e-5) * d["l0.norm1"]
            y, _ = plain.attention(h, raw["left"], d, "l0.mix.left.", None, 0)
            if mixer is pair:
                z, _ = plain.mamba2(h, raw["right"], d, "l0.mix.right.", 1e-5, None)
                y = 0.7 * y + 1.2 * z
            x = x + (plain.rms_unit(y, 1e-5) * d["l0.norm1"] if arrangement == "outnorm" else y)
            ref = (plain.rms_unit(x, 1e-5) * (1.0 + d["final.norm"])) @ d["head"].T
            assert float((got - ref).abs().max()) < 1e-4 * float(ref.abs().max()), arrangement


def test_plain_mechanisms_by_hand():
    """One token of each recurrence, the running maximum, the routing weights, the rotation's slowdown and pairs, norm parts."""
    t = lambda *v: torch.tensor(v, dtype=torch.float64)
    y, S = plain.state_space(t(3.0).view(1, 1, 1), t(2.0).view(1, 1, 1), t(5.0).view(1, 1, 1), t(0.5).view(1, 1), t(-2.0), t(10.0),
                             t(4.0).view(1, 1, 1))
    s = 4.0 * math.exp(-1.0) + 0.5 * 2.0 * 3.0
    assert abs(float(S) - s) < 1e-12 and abs(float(y) - (5.0 * s + 30.0)) < 1e-12
    o, S = plain.decayed_memory(t(1.0, 1.0).view(1, 1, 2), t(1.0, 0.0).view(1, 1, 2), t(7.0).view(1, 1, 1), t(0.5, 0.25).view(1, 1, 2),
                                t(2.0, 8.0).view(1, 2, 1))
    assert S.flatten().tolist() == [8.0, 2.0] and float(o) == 10.0
    # the maximum starts at 0: a first write gate below it leaves the state small instead of being scaled up
    o, S, n, m = plain.matrix_memory(t(2.0).view(1, 1, 1), t(1.0).view(1, 1, 1), t(3.0).view(1, 1, 1), t(-4.0).view(1, 1),
                                     t(-1.0).view(1, 1), torch.zeros(1, 1, 1, dtype=torch.float64), torch.zeros(1, 1, dtype=torch.float64),
                                     torch.zeros(1, dtype=torch.float64))
    assert float(m) == -1.0 and abs(float(S) - 3.0 * math.exp(-3.0)) < 1e-12 and abs(float(n) - math.exp(-3.0)) < 1e-12
    assert abs(float(o) - 6.0 * math.exp(-3.0) / (math.exp(1.0) + 1e-6)) < 1e-12
    got = dict(plain.route(t(0.0, math.log(2.0), 0.0, math.log(4.0)), t(0.0, 0.0, 0.9, 0.0), 2, 3.0))
    assert set(got) == {2, 3} and abs(got[3] - 3.0 * 0.8) < 1e-12 and abs(got[2] - 3.0 * 0.2) < 1e-12
    x = t(1.0, 0.0, 1.0, 0.0, 9.0).view(1, 1, 5)
    r = plain.rotate(x, torch.tensor([2]), {"dims": 4, "base": 16.0, "scaling": {"factor": 4.0}}).flatten().tolist()
    want = [math.cos(0.5), math.sin(0.5), math.cos(0.125), math.sin(0.125), 9.0]
    assert max(abs(a - b) for a, b in zip(r, want)) < 1e-12
    assert plain.part_norm(t(3.0, 3.0, -0.5, 0.5), 2, 0.0).tolist() == [1.0, 1.0, -1.0, 1.0]


def test_the_plain_implementation_cut_in_two():
    """The oracle itself: a sequence fed in parts through its state gives what it gives whole."""
    from pih_b200.config import config_from_dict
    from pih_b200.models import expected_tensors
    for name, cfg in bm.CONFIGS.items():
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


@pytest.mark.parametrize("name", ["B1", "B2", "B3"])
@pytest.mark.parametrize("family", ["whole", "portions", "mixed"])
def test_cut_invariance_with_stand_in_kernels(tmp_path, name, family):
    """Block tables, slot mappings, state slots and their reuse: the real parts and step function with torch stand-ins for
    the kernels agree with the plain implementation however the requests are cut."""
    d = bm.write_model(tmp_path / name, bm.CONFIGS[name], seed=1, sigma=bm.SIGMA[name])
    requests = traces.make_requests(bm.CONFIGS[name]["vocab"], [19, 6, 58, 1, 12], seed=3)
    kw = dict(max_live=2, decode_tail=3, max_portion=7) if family == "mixed" else {}
    steps = getattr(traces, family)(requests, **kw)
    _, model, cache, runner = _runner(d, max_cache_tokens=traces.peak_tokens(steps, round_to=4), max_requests=2)
    got = traces.replay(runner, steps)
    for rid, ref in bm.plain_logits(d, requests).items():
        assert float((got[rid].double() - ref).abs().max()) < 2e-4 * float(ref.abs().max()), (family, rid)
    cache.check()
    assert cache.slots.num_free == 2 and all(f == cache.num_pages for f in cache.num_free_pages())
    if family == "mixed":
        assert all(g.pool.pages_handed_out > g.pool.num_pages for g in cache.groups)


def test_pages_behind_the_window_go_back(tmp_path):
    """A request far longer than the windows holds only the pages that its next token may look into: a pool much smaller
    than the request is enough."""
    from pih_b200.engine import StepEntry
    d = bm.write_model(tmp_path / "m", bm.B1, seed=2, sigma=0.15)
    toks = traces.make_requests(311, [130], seed=4)["r0"]
    _, model, cache, runner = _runner(d, max_cache_tokens=64)
    assert sorted(g.need.window for g in cache.groups) == [21, 40]
    got, at = [], 0
    for n in [7, 13, 1, 19, 2, 6, 12, 1, 1, 15, 3, 17, 6, 5, 9, 13]:
        got.append(runner.step([StepEntry("a", toks[at:at + n], list(range(n)))]).clone())
        at += n
    assert at == 130
    ref = bm.plain_logits(d, {"a": toks})["a"]
    assert float((torch.cat(got).double() - ref).abs().max()) < 2e-4 * float(ref.abs().max())


def test_a_failed_step_leaves_the_states_as_they_were(tmp_path):
    """A step that raises after the layers have advanced their states (running maxima included) is rolled back."""
    from pih_b200.engine import StepEntry
    d = bm.write_model(tmp_path / "m", bm.B2, seed=2, sigma=0.15)
    toks = traces.make_requests(263, [14], seed=1)["r0"]
    _, model, cache, runner = _runner(d, max_cache_tokens=32)
    runner.step([StepEntry("a", toks[:9], [])])
    head = model.head
    model.head = None                                   # the head product fails, after every layer has run
    with pytest.raises(Exception):
        runner.step([StepEntry("a", toks[9:], [4])])
    model.head = head
    again = runner.step([StepEntry("a", toks[9:], [4])])
    ref = bm.plain_logits(d, {"a": toks})["a"][-1]
    assert float((again[0].double() - ref).abs().max()) < 2e-4 * float(ref.abs().max())


@pytest.mark.parametrize("seed", range(6))
def test_configurations_drawn_at_random_with_stand_in_kernels(tmp_path, seed):
    raw = bm.random_config(seed)
    d = bm.write_model(tmp_path / "m", raw, seed=seed, sigma=0.15)
    requests = traces.make_requests(raw["vocab"], [23, 9, 1, 14], seed=seed)
    steps = traces.mixed(requests, seed=seed, max_live=2, decode_tail=3, max_portion=6)
    _, model, cache, runner = _runner(d, max_cache_tokens=traces.peak_tokens(steps, round_to=4), max_requests=2)
    got = traces.replay(runner, steps)
    for rid, ref in bm.plain_logits(d, requests).items():
        assert float((got[rid].double() - ref).abs().max()) < 3e-4 * max(1.0, float(ref.abs().max())), rid
    cache.check()


def test_the_stream_stays_wide_in_bfloat16(tmp_path):
    """bfloat16 over stand-in kernels that round after each step: the stream, the norms behind the sub-layers and the pair's
    sum stay 32-bit, and the logits are within rounding of the plain implementation."""
    d = bm.write_model(tmp_path / "m", bm.B1, seed=4, sigma=0.15)
    requests = traces.make_requests(311, [31, 5], seed=3)
    _, model, cache, runner = _runner(d, "bfloat16", max_cache_tokens=64, max_requests=2)
    seen = set()
    ops = model.rt.ops
    inner = ops.stream_norm_norm

    def spy(h, y, w, eps, *a, **kw):
        seen.add((h.dtype, w.dtype, y.dtype))
        return inner(h, y, w, eps, *a, **kw)
    ops.stream_norm_norm = spy
    got = traces.replay(runner, traces.portions(requests))
    assert seen == {(torch.float32, torch.float32, torch.bfloat16)}
    for rid, ref in bm.plain_logits(d, requests).items():
        err = (got[rid].double() - ref).pow(2).mean().sqrt() / ref.std()
        assert float(err) < 0.05, (rid, float(err))
