"""The Bipulorn design on the GPU against the plain float64 restatement (tests/plain_bipulorn.py): each mechanism alone,
every way of cutting requests into steps, batches against requests alone, pages and state slots that are used again, keys
that must be found far back / at page borders / at a window's edge, in prompts and in decoding, the first tokens of a
sequence, states carried over many tokens, long decoding, configurations drawn at random, and greedy generation through
the engine's own entry point and command lines."""
import math
from types import SimpleNamespace

import pytest
import torch

import bipulorn_models as bm
import plain_bipulorn as plain
import traces

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
F64 = torch.float64


@pytest.fixture(scope="module")
def dirs(tmp_path_factory):
    return {n: bm.write_model(tmp_path_factory.mktemp(f"bipulorn_{n}"), raw, seed=5 + i, sigma=bm.SIGMA[n])
            for i, (n, raw) in enumerate(bm.CONFIGS.items())}


def _ops():
    from pih_b200.kernels import get_ops
    return get_ops(torch.device(DEV))


def _errors(got, truth):
    errs = []
    for rid, ref in truth.items():
        g = got[rid].double()
        assert g.shape == ref.shape, rid
        d = g - ref
        d = d - d.mean(dim=1, keepdim=True)
        errs.append(d.pow(2).mean(dim=1).sqrt() / ref.std())
    return torch.cat(errs)


def _check(got, truth, dtype, what, rounding=None):
    """Per position: how far the logits are off, up to a constant (root mean square), relative to the logits' spread.
    32-bit: every position.  bfloat16, over the positions of all requests together: the median within rounding, and at most
    one position in ten beyond three times that (a rounded router logit may choose another expert).  ``rounding``: a function
    that gives the errors of a plain bfloat16 evaluation of the same steps (torch operations with a rounding after each), for
    a model so steep that rounding alone exceeds the fixed bound."""
    err = _errors(got, truth)
    if dtype == "float32":
        assert float(err.max()) < 5e-5, f"{what}: error {float(err.max()):.3e} of the logits' spread at row {int(err.argmax())}"
        return
    bound = 0.03
    if rounding is not None and (float(err.median()) >= bound or int((err > 3 * bound).sum()) > len(err) // 10):
        plain_err = rounding()
        bound = max(bound, 1.5 * float(plain_err.median()), float(plain_err.quantile(0.9)) / 2)
    over = int((err > 3 * bound).sum())
    assert float(err.median()) < bound and over <= len(err) // 10, \
        f"{what}: median {float(err.median()):.3e}, {over} of {len(err)} positions beyond {3 * bound:.3f}, worst {float(err.max()):.3e}"


def _rounding(folder, steps, requests, **kw):
    def errors():
        from fake_ops import FakeOps
        from pih_b200.engine.factory import create_runner
        _, _, _, runner = create_runner(folder, "bfloat16", device="cpu", ops=FakeOps(), **kw)
        return _errors(traces.replay(runner, steps), bm.plain_logits(folder, requests))
    return errors


LENGTHS = {"B1": [70, 45, 131, 33, 64, 50, 1, 2], "B2": [65, 33, 97, 128, 80, 3, 35, 66], "B3": [50, 21, 1, 2, 34, 90]}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["B1", "B2", "B3"])
@pytest.mark.parametrize("family", ["whole", "tail_decode", "portions", "mixed"])
def test_cuttings_against_the_plain_implementation(dirs, name, dtype, family):
    """Whole prompts; most of a prompt and then token by token; portions down to two tokens; up to three live requests
    mixed, with a pool so small and so few state slots that pages and slots are used again.  The requests are longer than
    most windows, and than the chunks in which prompts go through the recurrences."""
    from pih_b200.engine.factory import create_runner
    requests = traces.make_requests(bm.CONFIGS[name]["vocab"], LENGTHS[name], seed=21)
    steps = getattr(traces, family)(requests, **(dict(max_live=3, max_portion=40) if family == "mixed" else {}))
    kw = dict(page_size={"B1": 16, "B2": 8, "B3": 4}[name], max_cache_tokens=traces.peak_tokens(steps, round_to=16),
              max_requests=3)
    _, model, cache, runner = create_runner(dirs[name], dtype, **kw)
    got = traces.replay(runner, steps)
    model.rt.ops.check_errors()
    _check(got, bm.plain_logits(dirs[name], requests), dtype, f"{name} {family} {dtype}",
           rounding=_rounding(dirs[name], steps, requests, **kw))
    cache.check()
    assert all(f == cache.num_pages for f in cache.num_free_pages()) and cache.slots.num_free == 3
    if family == "mixed":
        assert all(g.pool.pages_handed_out > g.pool.num_pages for g in cache.groups)


def test_the_stream_behind_every_layer(dirs):
    """The residual stream behind every layer against the plain implementation, in 32-bit: the blocks one by one through the
    model's own schedule and caches; what is pending behind a block is added by the norm's own kernel."""
    from pih_b200.engine import StepEntry
    from pih_b200.engine.factory import create_runner
    for name in ("B1", "B2"):
        toks = traces.make_requests(bm.CONFIGS[name]["vocab"], [53], seed=4)["r0"]
        cfg, w = bm.load_plain(dirs[name])
        layers, _, _ = plain.model_layers(cfg, w, toks)
        _, model, cache, runner = create_runner(dirs[name], "float32", page_size=16, max_cache_tokens=64, max_requests=1)
        seen = []
        for block in model.blocks:
            def spy(h, delta, step, c, inner=block.forward):
                h, delta = inner(h, delta, step, c)
                assert delta.norm is not None
                there = h.clone()
                model.final_norm.add_forward(there, delta)
                seen.append(there.double().cpu())
                return h, delta
            block.forward = spy
        runner.step([StepEntry("a", toks, [len(toks) - 1])])
        model.rt.ops.check_errors()
        assert len(seen) == layers.shape[0]
        for i, (got, ref) in enumerate(zip(seen, layers)):
            assert float((got - ref).abs().max()) < 2e-5 * float(ref.abs().max()), f"{name}: behind layer {i}"


LEFT, RIGHT = bm.att(4, 2, 12, 20, 0.4, window=13, rot=4, base=50.0, factor=2.5), bm.ssd(6, 8, 12, 2, 3, 3)


@pytest.mark.parametrize("mixer", [
    bm.pair(LEFT, RIGHT), bm.pair(bm.att(1, 1, 40, 8, 0.2, window=1, rot=40, base=3.0), bm.ssd(1, 20, 1, 1, 1, 1)),
    bm.pair(bm.att(2, 2, 8, 24, 0.3), bm.ssd(4, 6, 130, 4, 8, 2)), bm.pair(bm.att(3, 1, 16, 16, 0.5, window=1000, rot=2), bm.ssd(8, 4, 20, 1, 2, 6)),
    bm.gla(3, 12, 20, 2.0, 5), bm.gla(1, 1, 1, 16.0, 1), bm.gla(2, 65, 34, 1.0, 40), bm.gla(4, 4, 40, 8.0, 64),
    bm.mlstm(3, 12, 20, 6.0), bm.mlstm(1, 1, 1, 1.0), bm.mlstm(2, 65, 34, 30.0), bm.mlstm(5, 4, 40, 3.0)])
@pytest.mark.parametrize("mlp", [None, bm.moe(5, 3, 20, identity=2, scale=1.9, shared=28), bm.moe(2, 1, 16, shared=14)])
def test_a_layer_alone(tmp_path, mixer, mlp):
    """One layer, with experts and without, whole and token by token: windows of one place and wider than the requests, no
    window and no rotation, one group and as many groups as heads, norm parts inside and across heads, narrow projections
    of one number and wider than the heads, low and high caps."""
    from pih_b200.engine.factory import create_runner
    d = bm.write_model(tmp_path / "m", bm.single_layer(mixer, mlp), seed=3, sigma=0.2)
    requests = traces.make_requests(120, [40, 7], seed=2)
    truth = bm.plain_logits(d, requests)
    for family in ("whole", "tail_decode"):
        _, model, cache, runner = create_runner(d, "float32", page_size=8, max_cache_tokens=64, max_requests=2)
        _check(traces.replay(runner, getattr(traces, family)(requests)), truth, "float32", family)
        model.rt.ops.check_errors()


def _step(positions, request_of_row, cu_q, slots=None):
    t = lambda v: torch.tensor(v, dtype=torch.int32, device=DEV)
    slots = list(range(len(cu_q) - 1)) if slots is None else slots
    return SimpleNamespace(positions=t(positions), request_of_row=t(request_of_row), cu_q=t(cu_q), state_slots=t(slots),
                           num_requests=len(slots), host_cu_q=list(cu_q),
                           host_q_start=[positions[c] if c < len(positions) else 0 for c in cu_q[:-1]],
                           q_start=t([positions[c] if c < len(positions) else 0 for c in cu_q[:-1]]), meta=None, attention_plans={})


def _close(got, ref, tol, what=""):
    err, scale = float((got.double().cpu() - ref).abs().max()), max(1.0, float(ref.abs().max()))
    assert err < tol * scale, f"{what}: {err:.3e} of {scale:.3e}"


# -- the three recurrences -----------------------------------------------------------------------------------------------
class Memory:
    """One of the recurrences with random inputs: ``run`` feeds rows through the kernels (from strided views), ``plain`` gives
    what they have to be; the state of a slot is ``numbers`` 32-bit numbers and ``spare`` behind them."""
    spare = 5

    def __init__(self, kind, heads, groups, dim, vdim, T, dtype, seed=0, forget=1.0):
        g = torch.Generator().manual_seed(seed + dim + vdim)
        self.kind, self.heads, self.groups, self.dim, self.vdim, self.dtype = kind, heads, groups, dim, vdim, dtype
        rnd = lambda *s: torch.randn(*s, generator=g)
        cols = (2 * groups * dim + heads * vdim + 2 * heads + 7) // 8 * 8
        self.rows = (rnd(T, cols) * 0.7).to(dtype)
        self.q_at, self.k_at, self.v_at = 0, groups * dim, 2 * groups * dim
        self.g_at = 2 * groups * dim + heads * vdim
        self.z = rnd(T, heads * dim) * 2
        self.bias = [rnd(heads * dim if kind == "channel" else heads) * 0.5 for _ in range(2)]
        if kind == "channel":
            self.bias[0] -= forget
        self.A, self.D = -torch.exp(rnd(heads)) * forget, rnd(heads)
        self.temperature, self.cap = 1.5, 5.0
        self.copies = _ops().memory_copies(vdim)
        self.numbers = heads * dim * vdim + (heads * (dim + self.copies) if kind == "exp" else 0)
        self.divisor = torch.zeros(T, heads)

    def state(self, slots):
        return torch.zeros(slots, self.numbers + self.spare, device=DEV)

    def run(self, rows, cu, slots, state):
        ops, sel = _ops(), torch.tensor(rows)
        x = self.rows[sel].to(DEV)
        cut = lambda at, n: x[:, at:at + n]
        q, k = cut(self.q_at, self.groups * self.dim), cut(self.k_at, self.groups * self.dim)
        v, step = cut(self.v_at, self.heads * self.vdim), _step([0] * len(rows), [0] * len(rows), cu, slots)
        bias = [b.to(DEV) for b in self.bias]
        kw = dict(state=state, step=step, heads=self.heads, value_dim=self.vdim)
        if self.kind == "channel":
            return ops.gated_linear(q, k, v, self.z[sel].to(DEV), bias=bias[0], temperature=self.temperature,
                                    q_scale=self.dim ** -0.5, key_dim=self.dim, **kw).double().cpu()
        g0, g1 = cut(self.g_at, self.heads), cut(self.g_at + self.heads, self.heads)
        if self.kind == "step":
            return ops.state_space(q, k, v, g0, dt_bias=bias[0], A=self.A.to(DEV), D=self.D.to(DEV), groups=self.groups,
                                   state_dim=self.dim, **kw).double().cpu()
        out, div = ops.matrix_memory(q, k, v, g0, g1, write_bias=bias[0], keep_bias=bias[1], cap=self.cap, floor=1e-6,
                                     q_scale=self.dim ** -0.5, key_dim=self.dim, **kw)
        return (out / div[:, :, None]).double().cpu()

    def plain(self, r):
        """(outputs, the state's numbers) of the rows ``r`` as one sequence."""
        x, n = self.rows[r].double(), len(self.rows[r])
        H, G, d, p = self.heads, self.groups, self.dim, self.vdim
        q, k = x[:, :G * d].view(n, G, d), x[:, G * d:2 * G * d].view(n, G, d)
        v = x[:, self.v_at:self.v_at + H * p].view(n, H, p)
        g0, g1 = x[:, self.g_at:self.g_at + H], x[:, self.g_at + H:self.g_at + 2 * H]
        b0, b1 = (b.double() for b in self.bias)
        S0 = torch.zeros(H, d, p, dtype=F64)
        if self.kind == "channel":
            a = torch.exp(plain.log_sigmoid(self.z[r].double() + b0) / self.temperature).view(n, H, d)
            o, S = plain.decayed_memory(q * d ** -0.5, k, v, a, S0)
            return o, S.flatten()
        if self.kind == "step":
            o, S = plain.state_space(v, k, q, plain.softplus(g0 + b0), self.A.double(), self.D.double(), S0)
            return o, S.flatten()
        i = self.cap * torch.tanh((g0 + b0) / self.cap)
        f = plain.log_sigmoid(self.cap * torch.tanh((g1 + b1) / self.cap))
        o, S, nn, m = plain.matrix_memory(q * d ** -0.5, k, v, i, f, S0, torch.zeros(H, d, dtype=F64), torch.zeros(H, dtype=F64))
        return o, torch.cat([S.flatten(), nn.flatten(), m[:, None].expand(H, self.copies).flatten()])


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("kind", ["channel", "step", "exp"])
@pytest.mark.parametrize("dim, vdim", [(16, 24), (8, 64), (48, 40), (64, 72), (128, 128), (72, 136), (256, 64), (12, 8), (20, 7),
                                       (1, 1), (272, 200), (520, 8)])
def test_recurrences_of_every_size(kind, dim, vdim, dtype):
    """Every instance of the token-by-token kernel and of the kernels that take a prompt in chunks (bf16, sizes that are
    multiples of 8): two requests of unequal length (one of padding between them) in three steps — long portions, short
    ones and single tokens side by side — against plain loops; nothing beyond the state and no other slot is touched."""
    heads, groups = (4, 2) if kind == "step" else (2, 2)
    lens = [210, 95]
    mem = Memory(kind, heads, groups, dim, vdim, sum(lens), dtype)
    state = mem.state(4)
    got = torch.zeros(sum(lens), heads, vdim, dtype=F64)
    at, ends = [0, lens[0]], [lens[0], sum(lens)]
    for cuts in ([130, 20], [17, 3], [63, 1], [0, 71]):
        parts = [list(range(a, a + c)) for a, c in zip(at, cuts)]
        rows = parts[0] + parts[1]
        got[torch.tensor(rows)] = mem.run(rows, [0, cuts[0], cuts[0], len(rows)], [3, -1, 0], state)
        at = [a + c for a, c in zip(at, cuts)]
    assert at == ends
    _ops().check_errors()
    tol = 2e-5 if dtype == torch.float32 else 1e-4
    held = state.double().cpu()
    for r, slot in ((slice(0, lens[0]), 3), (slice(lens[0], None), 0)):
        o, S = mem.plain(r)
        _close(got[r], o, 4 * tol if kind == "exp" else tol, f"slot {slot}")
        _close(held[slot, :mem.numbers], S, tol, f"state of slot {slot}")
    assert float(held[[1, 2]].abs().max()) == 0.0 and float(held[:, mem.numbers:].abs().max()) == 0.0


@pytest.mark.parametrize("kind", ["channel", "step", "exp"])
def test_recurrences_in_32_bit_do_not_depend_on_the_cut(kind):
    """In 32-bit a row's result and the state are the same bit by bit wherever the portions are cut."""
    mem = Memory(kind, 2, 2, 24, 40, 150, torch.float32)
    outs = []
    for cuts in ([150], [64, 2, 1, 16, 17, 50], [1] * 20 + [130]):
        state, at, out = mem.state(1), 0, []
        for c in cuts:
            out.append(mem.run(list(range(at, at + c)), [0, c], [0], state))
            at += c
        outs.append((torch.cat(out), state.cpu()))
    for o, s in outs[1:]:
        assert torch.equal(o, outs[0][0]) and torch.equal(s, outs[0][1])


@pytest.mark.parametrize("forget", [0.001, 1.0, 20.0, 300.0])
@pytest.mark.parametrize("kind", ["channel", "step"])
def test_decays_of_every_strength(kind, forget):
    """Prompts in chunks with decays from next to one to such that forget everything within a token (so that the ratio of two
    decays of a chunk leaves the range of 32-bit numbers), against plain loops and against token by token."""
    mem = Memory(kind, 2, 2, 72, 64, 200, torch.bfloat16, forget=forget)
    state = mem.state(1)
    got = torch.cat([mem.run(list(range(0, 140)), [0, 140], [0], state), mem.run(list(range(140, 200)), [0, 60], [0], state)])
    o, S = mem.plain(slice(0, 200))
    assert bool(torch.isfinite(got).all())
    _close(got, o, 1e-4)
    _close(state[0, :mem.numbers], S, 1e-4)
    ops = _ops()
    try:
        ops.chunked_memory = False
        alone = mem.state(1)
        one_by_one = mem.run(list(range(200)), [0, 200], [0], alone)
    finally:
        ops.chunked_memory = True
    _close(one_by_one, o, 2e-5)
    _close(alone[0, :mem.numbers], S, 2e-5)


def test_channels_that_forget_beside_channels_that_remember():
    """Values written under orthogonal keys; one key channel forgets at once, the others do not decay: hundreds of tokens
    later, over several steps, the state returns every value but the one under the forgetting channel — in 32-bit, and in
    bf16 through the kernels that go by chunks."""
    ops = _ops()
    D, V, n = 32, 24, 432
    g = torch.Generator().manual_seed(3)
    v = torch.randn(n, V, generator=g).bfloat16().float()
    v[D:] = 0.0                                                                   # later tokens write nothing
    k = torch.eye(D)[torch.arange(n) % D]
    z = torch.full((n, D), 200.0)
    z[:, 7] = -200.0
    for dtype, tol in ((torch.float32, 1e-6), (torch.bfloat16, 1e-4)):
        state, outs, at = torch.zeros(1, D * V, device=DEV), [], 0
        kk, vv = k.to(dtype).to(DEV), v.to(dtype).to(DEV)
        for cut in (5, 90, 1, 1, 2, 133, 200):
            sl = slice(at, at + cut)
            outs.append(ops.gated_linear(kk[sl], kk[sl], vv[sl], z[sl].to(DEV), bias=torch.zeros(D, device=DEV), temperature=2.0,
                                         q_scale=1.0, state=state, step=_step([0] * cut, [0] * cut, [0, cut]), heads=1, key_dim=D,
                                         value_dim=V))
            at += cut
        ops.check_errors()
        out = torch.cat(outs)[:, 0].cpu()
        for t in list(range(D)) + list(range(n - D, n)):
            want = torch.zeros(V) if t % D == 7 and t >= D else v[t % D]
            assert float((out[t] - want).abs().max()) < tol * 4, (dtype, t)


def test_the_running_maximum_starts_at_zero_and_lives_on():
    """Matrix memory with write gates far below and far above zero: the first tokens of a sequence feel the maximum's start,
    a strong write lowers what came before for good, and n's divisor never falls below exp(-m)."""
    T = 120
    for dtype in (torch.float32, torch.bfloat16):
        mem = Memory("exp", 2, 2, 16, 24, T, dtype)
        mem.cap = 30.0
        mem.rows[:, mem.g_at:mem.g_at + 2] = -12.0                                # weak writes ...
        mem.rows[50, mem.g_at] = 25.0                                             # ... and one strong one on head 0
        mem.rows[:, mem.g_at + 2:mem.g_at + 4] = 8.0                              # hardly any forgetting
        mem.bias = [torch.zeros(2), torch.zeros(2)]
        o, S = mem.plain(slice(0, T))
        assert float(S[-mem.copies]) < -0.0 or float(S[-2 * mem.copies]) > 20.0
        for cuts in ([120], [1, 2, 47, 1, 69], [30, 90]):
            state, at, out = mem.state(1), 0, []
            for c in cuts:
                out.append(mem.run(list(range(at, at + c)), [0, c], [0], state))
                at += c
            got = torch.cat(out)
            _close(got / o.abs().amax(-1, keepdim=True).clamp(min=1e-30), o / o.abs().amax(-1, keepdim=True).clamp(min=1e-30),
                   3e-5 if dtype == torch.float32 else 1e-3, f"{dtype} {cuts}")
            _close(state[0, :mem.numbers], S, 1e-5 if dtype == torch.float32 else 1e-4)
