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
    bound, allowed = 0.03, len(err) // 10
    if rounding is not None and (float(err.median()) >= bound or int((err > 3 * bound).sum()) > allowed):
        plain_err = rounding()
        bound = max(bound, 1.5 * float(plain_err.median()))
        allowed = max(allowed, 3 * int((plain_err > 3 * bound).sum()) // 2)
    over = int((err > 3 * bound).sum())
    assert float(err.median()) < bound and over <= allowed, \
        f"{what}: median {float(err.median()):.3e}, {over} of {len(err)} positions beyond {3 * bound:.3f} (at most {allowed}), " \
        f"worst {float(err.max()):.3e}"


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


# -- attention, norms, gates -----------------------------------------------------------------------------------------------
def _plain_rows(q, K, V, positions, scale, window, gate, group):
    """softmax(q k scale) v over the last ``window`` keys (0: all), times the gate of the column."""
    out = torch.zeros(q.shape[0], q.shape[1], V.shape[-1], dtype=F64)
    for t, p in enumerate(positions):
        lo = max(0, p - window + 1) if window else 0
        for h in range(q.shape[1]):
            s = (K[lo:p + 1, h // group] @ q[t, h]) * scale
            out[t, h] = torch.softmax(s, dim=0) @ V[lo:p + 1, h // group]
    return out * torch.sigmoid(gate).view(out.shape)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rows_of_step", [260, 17, 5, 1])
@pytest.mark.parametrize("window, dim, vdim", [(64, 64, 64), (50, 64, 128), (7, 32, 40), (1, 16, 24), (150, 96, 48), (0, 64, 64),
                                               (40, 72, 136), (33, 20, 6)])
def test_keys_that_stand_out_at_the_windows_edges(dtype, rows_of_step, window, dim, vdim):
    """A key that scores high wherever it is seen, at every place in turn where rows exist for which it is the last one
    inside the window (head 0) or at a page border (head 1); a gate a column; a prompt of several row tiles (the tensor-core
    kernel in bf16), short portions and single rows (the warp kernel, its keys cut into parts).  Windows one place longer or
    shorter would give something else."""
    ops = _ops()
    heads, kv_heads, page, n = 4, 2, 16, 300
    g = torch.Generator().manual_seed(window + dim)
    V = torch.randn(n, kv_heads, vdim, generator=g, dtype=F64)
    K = 0.05 * torch.randn(n, kv_heads, dim, generator=g, dtype=F64)
    unit = torch.zeros(dim, dtype=F64)
    unit[3] = 1.0
    edge = n - 1 - (window - 1 if window else 250)                # the last row's oldest key
    for j in {edge, edge - 1, edge - 3, 40, 41}:
        K[max(j, 0), 0] += (5.0 + 0.5 * (j % 3)) * unit
    K[page - 1::page, 1] += 4.0 * unit
    K[::page, 1] += 4.0 * unit
    first = n - rows_of_step
    positions = list(range(first, n))
    q = 0.05 * torch.randn(rows_of_step, heads, dim, generator=g, dtype=F64) + 3.0 * unit
    gate = torch.randn(rows_of_step, heads * vdim, generator=g, dtype=F64)
    qd, Kd, Vd, gd = (x.to(dtype).double() for x in (q, K, V, gate))
    want = 0.6 * _plain_rows(qd, Kd, Vd, positions, 0.5, window, gd, heads // kv_heads)
    pages = -(-n // page)
    order = torch.randperm(pages + 3, generator=g)[:pages]
    cache = torch.zeros(pages + 3, page, kv_heads * (dim + vdim), dtype=dtype, device=DEV)
    flat = torch.cat([Kd.reshape(n, -1), Vd.reshape(n, -1)], dim=1).to(dtype).to(DEV)
    for i in range(pages):
        rows = flat[i * page:(i + 1) * page]
        cache[order[i], :rows.shape[0]] = rows
    table = order.to(torch.int32).clone()
    if window:
        table[:max(0, first - window + 1) // page] = -1            # pages behind the window were given back
    out = torch.full((rows_of_step, heads * vdim + 6), 9.0, dtype=dtype, device=DEV)
    wide_gate = torch.cat([torch.full((rows_of_step, 3), 50.0, dtype=F64), gd], dim=1).to(dtype).to(DEV)[:, 3:]
    ops.window_attention(qd.to(dtype).reshape(rows_of_step, -1).contiguous().to(DEV), cache=cache,
                         block_table=table.to(DEV).reshape(1, -1).contiguous(),
                         step=_step(positions, [0] * rows_of_step, [0, rows_of_step]), scale=0.5, window=window, keep_first=0,
                         softcap=0.0, bias=None, sink=None, gate=wide_gate, gate_per="column", heads=heads, kv_heads=kv_heads,
                         key_dim=dim, value_dim=vdim, scale_out=0.6, out=out[:, 2:2 + heads * vdim])
    ops.check_errors()
    assert bool((out[:, :2] == 9.0).all()) and bool((out[:, -4:] == 9.0).all())
    got = out[:, 2:2 + heads * vdim].double().cpu().reshape(rows_of_step, heads, vdim)
    limit = 1e-5 if dtype == torch.float32 else 2e-2
    assert float((got - want).abs().max()) < limit * float(want.abs().max())
    if window > 1:
        for other in (window + 1, window - 1):                     # the check would see a fault
            moved = 0.6 * _plain_rows(qd[-1:], Kd, Vd, positions[-1:], 0.5, other, gd[-1:], heads // kv_heads)
            assert float((moved - want[-1:]).abs().max()) > 0.05 * float(want[-1].abs().max())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("dim, vdim, rot", [(64, 128, 48), (64, 64, 64), (16, 24, 8), (10, 6, 6), (12, 20, 2), (320, 24, 320), (64, 48, 0)])
def test_biases_and_rotation_of_neighbouring_pairs(dtype, dim, vdim, rot):
    """q, k and v with their biases added before the rotation, into the queries' buffer and the cache; far positions; pairs of
    halves and of neighbours; rows of padding write nothing."""
    ops = _ops()
    heads, kv_heads, page, T = 4, 2, 8, 21
    g = torch.Generator().manual_seed(dim + rot)
    cols = heads * dim + kv_heads * (dim + vdim)
    src = torch.randn(T, cols + 8, generator=g).to(dtype)
    bias = torch.randn(cols, generator=g)
    positions = [0, 1, 2, 100, 1023] + list(range(3000, 3000 + T - 5))
    slots = torch.arange(T, dtype=torch.int32) + 3
    slots[6] = -2
    for interleaved in (True, False):
        if rot:
            freq = torch.tensor([5000.0 ** (-2.0 * i / rot) / 4.0 for i in range(rot // 2)], dtype=F64)
        cache = torch.zeros(4, page, kv_heads * (dim + vdim), dtype=dtype, device=DEV)
        q = ops.window_qk_prepare(src.to(DEV), q_norm=None, k_norm=None, eps=0.0, rope_table=None, rotary_dim=rot,
                                  interleaved=interleaved, positions=torch.tensor(positions, dtype=torch.int32, device=DEV),
                                  slot_mapping=slots.to(DEV), cache=cache, heads=heads, kv_heads=kv_heads, key_dim=dim,
                                  value_dim=vdim, values_from_keys=False, frequencies=freq.float().to(DEV) if rot else None,
                                  in_bias=bias.to(DEV))
        ops.check_errors()
        x = src[:, :cols].double() + bias.double()

        def turned(v, n):
            v = v.reshape(T, n, dim)
            if not rot:
                return v
            if interleaved:
                return plain.rotate(v, torch.tensor(positions), {"dims": rot, "base": 5000.0, "scaling": {"factor": 4.0}})
            ang = torch.tensor(positions, dtype=F64)[:, None] * freq[None, :]
            c, s = torch.cos(ang)[:, None], torch.sin(ang)[:, None]
            a, b = v[..., :rot // 2], v[..., rot // 2:rot]
            return torch.cat([a * c - b * s, b * c + a * s, v[..., rot:]], dim=-1)

        tol = 2e-3 if dtype == torch.float32 else 3e-2             # (32-bit angles of positions in the thousands)
        _close(q, turned(x[:, :heads * dim], heads).reshape(T, -1), tol, "q")
        flat = cache.view(-1, cache.shape[-1]).double().cpu()
        want = torch.cat([turned(x[:, heads * dim:heads * dim + kv_heads * dim], kv_heads).reshape(T, -1),
                          x[:, heads * dim + kv_heads * dim:]], dim=1)
        for t, s in enumerate(slots.tolist()):
            if s >= 0:
                _close(flat[s], want[t], tol, f"cache row {t}")
        assert float(flat[9].abs().max()) == 0.0 and float(flat[:3].abs().max()) == 0.0


@pytest.mark.parametrize("width", [6, 72, 1000, 1024, 2050, 3001, 8192, 16384])
def test_the_norm_behind_the_sum_and_the_next_norm(width):
    """h += norm(y + bias) * w1, then norm(h) * w2; with a pair of outputs in y's place; stored back, or for gathered rows
    not stored; sizes in 16-byte pieces, odd ones, and ones that need every piece a thread can hold."""
    ops = _ops()
    g = torch.Generator().manual_seed(width)
    rows = 7
    vec = lambda: torch.randn(width, generator=g)
    h0, y, y2 = (torch.randn(rows, width, generator=g) for _ in range(3))
    h0[3] *= 1e-3
    y[4] *= 50.0
    bias, bias2, left, right, w1, w2 = (vec() for _ in range(6))
    pick = torch.tensor([6, 0, 3], dtype=torch.int32)
    for dtype in (torch.float32, torch.bfloat16):
        a, b = y.to(dtype), y2.to(dtype)
        for parts in ("", "b", "p", "bp", "bpq"):
            u = a.double() + (bias.double() if "b" in parts else 0.0)
            kw = dict(bias=bias.to(DEV)) if "b" in parts else {}
            if "p" in parts:
                kw["pair"] = (b.to(DEV), bias2.to(DEV) if "q" in parts else None, left.to(DEV), right.to(DEV), 1e-3)
                other = b.double() + (bias2.double() if "q" in parts else 0.0)
                u = plain.rms_unit(u, 1e-3) * left.double() + plain.rms_unit(other, 1e-3) * right.double()
            want = h0.double() + plain.rms_unit(u, 1e-5) * w1.double()
            normed = plain.rms_unit(want, 1e-4) * w2.double()
            tol = 3e-5 if dtype == torch.float32 else 2e-2
            h = h0.to(DEV)
            out = ops.stream_norm_norm(h, a.to(DEV), w1.to(DEV), 1e-5, w2.to(DEV), 1e-4, out_dtype=dtype, **kw)
            assert out.dtype == dtype
            _close(h, want, 1e-5)
            _close(out, normed, tol)
            h = h0.to(DEV)
            out = ops.stream_norm_norm(h, a.to(DEV), w1.to(DEV), 1e-5, w2.to(DEV), 1e-4, out_dtype=dtype, rows=pick.to(DEV), **kw)
            assert torch.equal(h.cpu(), h0)
            _close(out, normed[pick.long()], tol)
    ops.check_errors()


@pytest.mark.parametrize("width, parts", [(96, 4), (96, 1), (50, 5), (3, 3), (4096, 1), (6000, 2), (2048, 8)])
def test_norms_of_the_read_outs(width, parts):
    """The gate before a norm in parts; the norm of a head divided by a number first, with a weight a head and column; both
    into strided views, scaled; the capped logits."""
    ops = _ops()
    g = torch.Generator().manual_seed(width)
    rows = 9
    y, gate, w = torch.randn(rows, width, generator=g), torch.randn(rows, width + 3, generator=g), torch.randn(width, generator=g)
    div = torch.rand(rows, parts, generator=g) + 1e-4
    for dtype in (torch.float32, torch.bfloat16):
        gd = gate.to(dtype)
        tol = 1e-5 if dtype == torch.float32 else 2e-2
        z = gd[:, 3:].double()
        for what in ("parts", "heads"):
            out = torch.full((rows, width + 4), 3.0, dtype=dtype, device=DEV)
            if what == "parts":
                ops.gated_part_rmsnorm(y.to(DEV), gd.to(DEV)[:, 3:], w.to(DEV), parts, 1e-4, scale=1.7, out=out[:, 2:width + 2])
                ref = 1.7 * plain.part_norm(y.double() * plain.silu(z), parts, 1e-4) * w.double()
            else:
                o = y.view(rows, parts, -1).contiguous()
                ops.gated_rmsnorm(o.to(DEV), gd.to(DEV)[:, 3:], w.to(DEV), 1e-4, activation="sigmoid", scale=1.7,
                                  out=out[:, 2:width + 2], divisor=div.to(DEV))
                ref = 1.7 * plain.rms_unit(o.double() / div.double()[:, :, None], 1e-4).reshape(rows, width) * w.double() * torch.sigmoid(z)
            _close(out[:, 2:width + 2], ref, tol, what)
            assert bool((out[:, :2] == 3.0).all()) and bool((out[:, width + 2:] == 3.0).all())
    x = torch.linspace(-90, 90, 1001, device=DEV)[None, :].contiguous()
    want = 7.5 * torch.tanh(x.double() / 7.5)
    assert float((ops.softcap_(x, 7.5).double() - want).abs().max()) < 2e-6
    ops.check_errors()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rows", [1, 8, 50, 300])
def test_routing_weights_are_divided_and_scaled(rows, dtype):
    """Experts and identity experts whose weights are the chosen scores over their sum, scaled — through the kernels of few
    rows, of the library's grouped products and of the 32-bit path; the correction moves the choice and not the weights."""
    ops = _ops()
    g = torch.Generator().manual_seed(rows)
    hidden, ff, experts, identity, top = 48, 24, 5, 3, 3
    x = torch.randn(rows, hidden, generator=g).to(dtype)
    logits, correction = torch.randn(rows, experts + identity + 1, generator=g), torch.randn(experts + identity, generator=g) * 0.3
    bad = rows - 1 if rows > 1 else None                              # a row of padding may hold anything
    if bad is not None:
        logits[bad] = float("nan")
    w = {}
    for e in range(experts):
        for n, shape in (("gate", (ff, hidden)), ("up", (ff, hidden)), ("down", (hidden, ff))):
            w[f"e{e}.{n}"] = (torch.randn(*shape, generator=g) * 0.2).to(dtype)
    gu = torch.stack([torch.cat([w[f"e{e}.gate"], w[f"e{e}.up"]]) for e in range(experts)])
    dn = torch.stack([w[f"e{e}.down"] for e in range(experts)])
    out = ops.moe_experts(x.to(DEV), logits.to(DEV), gu.to(DEV), dn.to(DEV), top,
                          routing=dict(outputs=experts + identity, correction=correction.to(DEV), renormalize=True, weight_scale=2.3))
    ops.check_errors()
    ref = torch.zeros(rows, hidden, dtype=F64)
    wd = {n: t.double() for n, t in w.items()}
    out = out.double().cpu()
    for t in range(rows):
        if t == bad:
            out[t] = 0.0
            continue
        for e, weight in plain.route(logits[t, :-1].double(), correction.double(), top, 2.3):
            ref[t] += weight * (plain.gated(x[t].double(), wd, f"e{e}.") if e < experts else x[t].double())
    _close(out, ref, 1e-5 if dtype == torch.float32 else 2e-2)


# -- whole models ------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("name", ["B1", "B2"])
def test_batches_against_each_request_alone(dirs, name):
    """Unequal requests side by side in one step — a long portion, a short one, single tokens — give each request
    what it gets alone (32-bit: every reduction has an order fixed by the row)."""
    from pih_b200.engine import StepEntry
    from pih_b200.engine.factory import create_runner
    requests = traces.make_requests(bm.CONFIGS[name]["vocab"], [61, 18, 40, 9], seed=8)
    alone = {}
    for rid, toks in requests.items():
        _, _, _, runner = create_runner(dirs[name], "float32", page_size=16, max_cache_tokens=128, max_requests=1)
        alone[rid] = traces.replay(runner, traces.whole({rid: toks}))[rid]
    _, model, cache, runner = create_runner(dirs[name], "float32", page_size=16, max_cache_tokens=256, max_requests=4)
    cuts = {"r0": [33, 27, 1], "r1": [1, 16, 1], "r2": [2, 37, 1], "r3": [7, 1, 1]}
    got, at = {rid: [] for rid in requests}, {rid: 0 for rid in requests}
    for i in range(3):
        entries = []
        for rid, toks in requests.items():
            n = cuts[rid][i]
            entries.append(StepEntry(rid, toks[at[rid]:at[rid] + n], list(range(n))))
            at[rid] += n
        logits = runner.step(entries)
        j = 0
        for e in entries:
            got[e.rid].append(logits[j:j + len(e.tokens)].clone())
            j += len(e.tokens)
    model.rt.ops.check_errors()
    for rid in requests:
        assert float((torch.cat(got[rid]).cpu() - alone[rid]).abs().max()) < 1e-5 * float(alone[rid].abs().max()), rid


@pytest.mark.parametrize("seed", range(12))
def test_configurations_drawn_at_random(tmp_path, seed):
    """Sizes, orders of layers and constants drawn at random (odd sizes and sizes that only the plain kernels take among
    them): a mixed schedule in 32-bit against the plain implementation position by position, and in bfloat16 within
    rounding."""
    from pih_b200.engine.factory import create_runner
    raw = bm.random_config(seed)
    requests = traces.make_requests(raw["vocab"], [150, 45, 33, 18, 1, 2], seed=seed)
    steps = traces.mixed(requests, seed=seed, max_live=3, max_portion=60)
    d = bm.write_model(tmp_path / "m", raw, seed=seed, sigma=0.15)
    kw = dict(page_size=16, max_cache_tokens=traces.peak_tokens(steps, round_to=16), max_requests=3)
    for dtype in ("float32", "bfloat16"):
        _, model, cache, runner = create_runner(d, dtype, **kw)
        got = traces.replay(runner, steps)
        model.rt.ops.check_errors()
        _check(got, bm.plain_logits(d, requests), dtype, f"seed {seed} {dtype}", rounding=_rounding(d, steps, requests, **kw))
        cache.check()


def test_long_decoding(dirs):
    """A short prompt and 300 tokens one by one: pages fill and go back behind the windows, the states run on."""
    from pih_b200.engine.factory import create_runner
    for name in ("B1", "B3"):
        requests = traces.make_requests(bm.CONFIGS[name]["vocab"], [310], seed=9)
        steps = traces.tail_decode(requests, tail=300)
        _, model, cache, runner = create_runner(dirs[name], "float32", page_size=8, max_cache_tokens=320, max_requests=1)
        _check(traces.replay(runner, steps), bm.plain_logits(dirs[name], requests), "float32", f"{name} long decoding")
        model.rt.ops.check_errors()


@pytest.mark.parametrize("cuda_graphs", [False, True])
@pytest.mark.parametrize("name", ["B1", "B2", "B3"])
def test_greedy_generation_through_the_engine(dirs, name, cuda_graphs):
    """Engine.complete (scheduler, cache, sampler, graphs, padded steps, ids fed on the device) against greedy decoding
    with the plain implementation; three requests at once with room for two, so they queue."""
    from pih_b200.engine import Engine
    cfg, w = bm.load_plain(dirs[name])
    prompts = list(traces.make_requests(bm.CONFIGS[name]["vocab"], [9, 21, 5], seed=13).values())
    new, want = 12, []
    for p in prompts:
        _, logits, state = plain.model_layers(cfg, w, p)
        toks = [int(logits[-1].argmax())]
        while len(toks) < new:
            _, logits, state = plain.model_layers(cfg, w, toks[-1:], state)
            toks.append(int(logits[-1].argmax()))
        want.append(toks)
    engine = Engine(dirs[name], "float32", page_size=16, max_cache_tokens=256, maximum_batch_sequences=2,
                    maximum_batch_tokens=64, maximum_context_tokens=64, cuda_graphs=cuda_graphs)
    results = engine.complete_batch(prompts, max_tokens=new, temperature=0.0, ignore_eos=True)
    engine.rt.ops.check_errors()
    for r, expect in zip(results, want):
        assert r["token_ids"] == expect


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_graphs_and_padded_steps_against_plain_launches(dirs, dtype):
    """The same mixed requests through a runner that pads its steps and replays them from graphs and through one that
    does not: padding leaves states, pages and logits alone."""
    from pih_b200.engine import StepEntry
    from pih_b200.engine.factory import create_runner
    requests = traces.make_requests(bm.B1["vocab"], [33, 20, 47], seed=17)
    logits = []
    for graphs in (False, True):
        _, model, cache, runner = create_runner(dirs["B1"], dtype, page_size=16, max_cache_tokens=512, max_requests=4,
                                                cuda_graphs=graphs)
        out = []
        for turn in range(3):                                        # the same shapes again: seen, captured, replayed
            at = {r: 0 for r in requests}
            for cuts in ([17, 3, 30], [1, 9, 1], [9, 1, 10], [1, 1, 1], [1, 1, 1], [4, 5, 4]):
                entries = []
                for rid, n in zip(requests, cuts):
                    entries.append(StepEntry(f"{rid}.{turn}", requests[rid][at[rid]:at[rid] + n], [n - 1]))
                    at[rid] += n
                out.append(runner.step(entries).clone())
            for rid in requests:
                runner.finish(f"{rid}.{turn}")
        model.rt.ops.check_errors()
        logits.append(torch.stack([o.float() for o in out]))
    scale = float(logits[0].std())
    assert float((logits[0] - logits[1]).abs().max()) < (1e-5 if dtype == "float32" else 0.2) * scale
    six = logits[1].view(3, 6, *logits[1].shape[1:])
    assert float((six[0] - six[2]).abs().max()) < (1e-5 if dtype == "float32" else 0.2) * scale


def test_command_lines(dirs, tmp_path):
    """bin/pih-worker makes a random Bipulorn model from a configuration file and generates from it; bin/trace_run replays
    a trace on it, in both precisions; all agree with the plain implementation."""
    import json
    import os
    import subprocess
    import sys

    import numpy as np
    from conftest import ROOT
    worker = [sys.executable, os.path.join(ROOT, "bin", "pih-worker")]
    cfg_file = tmp_path / "config.json"
    cfg_file.write_text(json.dumps(bm.B1))
    folder = str(tmp_path / "made")
    proc = subprocess.run(worker + ["--random-model", folder, "--config", str(cfg_file), "--seed", "4", "--sigma", "0.15"],
                          capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    prompt = [5, 17, 3, 200, 9]
    proc = subprocess.run(worker + ["--model", folder, "--generate-tokens", ",".join(map(str, prompt)), "--max-tokens", "7",
                                    "--dtype", "float32", "--ignore-eos"], capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    res = json.loads(proc.stdout.strip().splitlines()[-1])
    cfg, w = bm.load_plain(folder)
    toks = list(prompt)
    for _ in range(7):
        toks.append(int(plain.model_layers(cfg, w, toks)[1][-1].argmax()))
    assert res["token_ids"] == toks[len(prompt):]

    requests = traces.make_requests(bm.B1["vocab"], [40, 9, 23], seed=6)
    steps = traces.mixed(requests, seed=1, max_live=3)
    for s_ in steps:
        for e in s_["entries"]:
            e["want"] = e["want"][-1:]                              # the last place of every portion
    truth = bm.plain_logits(folder, requests)
    for dtype, tol in (("float32", 1e-4), ("bfloat16", 0.1)):
        out_dir = str(tmp_path / dtype)
        cmd = [sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", out_dir,
               "--max-tokens", str(traces.peak_tokens(steps))]
        proc = subprocess.run(cmd, input="\n".join(json.dumps(s_) for s_ in steps) + "\n", capture_output=True, text=True,
                              timeout=600)
        assert proc.returncode == 0, proc.stderr[-2000:]
        assert [l for l in proc.stdout.splitlines() if l.startswith("done ")] == [f"done {s_['step']}" for s_ in steps]
        at = {rid: 0 for rid in requests}
        over = total = 0
        for s_ in steps:
            got = np.fromfile(os.path.join(out_dir, f"{s_['step']}.f32"), dtype="<f4").reshape(-1, bm.B1["vocab"])
            for j, e in enumerate(s_["entries"]):
                at[e["id"]] += len(e["tokens"])
                ref = truth[e["id"]][at[e["id"]] - 1].numpy()
                total += 1
                over += int(np.abs(got[j] - ref).max() >= tol * max(1.0, np.abs(ref).max()))
        # (in bfloat16 a rounded router logit may choose another expert at a few places)
        assert over <= (0 if dtype == "float32" else total // 10), (dtype, over, total)
