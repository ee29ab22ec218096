"""The Kedavik design on the GPU against the plain float64 restatement (tests/plain_kedavik.py): each mechanism alone,
every way of cutting requests into steps, batches against requests alone, pages and state slots that are used again, keys
that must be found far back / at page borders / at a chunk's edges, in prompts and in decoding, the first tokens of a
sequence, states carried over many tokens, long decoding, configurations drawn at random, and greedy generation through
the engine's own entry point and command lines."""
import math
from types import SimpleNamespace

import pytest
import torch

import kedavik_models as km
import plain_kedavik as plain
import traces

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
F64 = torch.float64


@pytest.fixture(scope="module")
def dirs(tmp_path_factory):
    return {n: km.write_model(tmp_path_factory.mktemp(f"kedavik_{n}"), raw, seed=5 + i, sigma=km.SIGMA[n])
            for i, (n, raw) in enumerate(km.CONFIGS.items())}


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
    """Per position: how far the logits are off, up to a constant (root mean square), relative to the logits' spread.  32-bit: every position.  bfloat16, over the positions of all requests together: the median within
    rounding, and at most one position in ten beyond three times that.  ``rounding``: a function that gives the errors of
    a plain bfloat16 evaluation of the same steps (torch operations with a rounding after each), for a model so steep that
    rounding alone exceeds the fixed bound."""
    err = _errors(got, truth)
    if dtype == "float32":
        assert float(err.max()) < 5e-5, f"{what}: error {float(err.max()):.3e} of the logits' spread at row {int(err.argmax())}"
        return
    bound = 0.03
    if rounding is not None and (float(err.median()) >= bound or int((err > 3 * bound).sum()) > len(err) // 10):
        bound = max(bound, 1.5 * float(rounding().median()))
    over = int((err > 3 * bound).sum())
    assert float(err.median()) < bound and over <= len(err) // 10, \
        f"{what}: median {float(err.median()):.3e}, {over} of {len(err)} positions beyond {3 * bound:.3f}, worst {float(err.max()):.3e}"


LENGTHS = {"K1": [70, 45, 131, 33, 64, 50, 1, 2], "K2": [65, 33, 97, 128, 80, 3, 35, 66], "K3": [50, 21, 1, 2, 34, 90]}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["K1", "K2", "K3"])
@pytest.mark.parametrize("family", ["whole", "tail_decode", "portions", "mixed"])
def test_cuttings_against_the_plain_implementation(dirs, name, dtype, family):
    """Whole prompts; most of a prompt and then token by token; portions down to two tokens; up to three live requests
    mixed, with a pool so small and so few state slots that pages and slots are used again.  The requests are longer than
    every chunk of K1 and K3, and cross several."""
    from pih_b200.engine.factory import create_runner
    requests = traces.make_requests(km.CONFIGS[name]["vocab"], LENGTHS[name], seed=21)
    kw = dict(max_live=3) if family == "mixed" else {}
    steps = getattr(traces, family)(requests, **kw)
    page = {"K1": 16, "K2": 8, "K3": 4}[name]
    _, model, cache, runner = create_runner(dirs[name], dtype, page_size=page,
                                            max_cache_tokens=traces.peak_tokens(steps, round_to=16), max_requests=3)
    got = traces.replay(runner, steps)
    model.rt.ops.check_errors()
    _check(got, km.plain_logits(dirs[name], requests), dtype, f"{name} {family} {dtype}")
    cache.check()
    assert all(f == cache.num_pages for f in cache.num_free_pages()) and cache.slots.num_free == 3
    if family == "mixed":
        assert all(g.pool.pages_handed_out > g.pool.num_pages for g in cache.groups)


def test_the_stream_behind_every_layer_run(dirs):
    """The residual stream behind every layer that runs (a looped layer each time) against the plain implementation, in
    32-bit: the blocks one by one through the model's own schedule and caches."""
    from pih_b200.engine import StepEntry
    from pih_b200.engine.factory import create_runner
    from pih_b200.parts import Pending
    for name in ("K1", "K2"):
        toks = traces.make_requests(km.CONFIGS[name]["vocab"], [53], seed=4)["r0"]
        cfg, w = km.load_plain(dirs[name])
        layers, _, _ = plain.model_layers(cfg, w, toks)
        _, model, cache, runner = create_runner(dirs[name], "float32", page_size=16, max_cache_tokens=64, max_requests=1)
        seen = []
        for block in model.blocks:
            inner = block.forward

            def spy(h, delta, step, c, inner=inner):
                h, delta = inner(h, delta, step, c)
                assert isinstance(delta, Pending) and delta.again is None and delta.vector is None
                y = delta.y if delta.bias is None else delta.y + delta.bias
                seen.append((h + delta.scale * y).double().cpu())
                return h, delta
            block.forward = spy
        runner.step([StepEntry("a", toks, [len(toks) - 1])])
        model.rt.ops.check_errors()
        assert len(seen) == layers.shape[0]
        for i, (got, ref) in enumerate(zip(seen, layers)):
            assert float((got - ref).abs().max()) < 2e-5 * float(ref.abs().max()), f"{name}: behind layer run {i}"


SCAN, LEFT, RIGHT = km.scan(40, 7, 5, 4), km.att(4, 2, 12, 20, 0.4, chunk=13, rot=4, base=50.0), km.dlt(2, 1, 12, 20, 3, 6, 9)


@pytest.mark.parametrize("mixer", [
    SCAN, km.scan(24, 1, 1, 1), km.scan(33, 70, 40, 6), km.scan(16, 130, 3, 2),
    km.pair(LEFT, RIGHT, 0.6, 1.4), km.pair(LEFT, RIGHT, 1.3, 0.0), km.pair(LEFT, RIGHT, 0.0, 0.7), km.pair(LEFT, RIGHT, -1.0, -0.4),
    km.pair(km.att(1, 1, 40, 8, 0.2, chunk=1, rot=40, base=3.0), km.dlt(1, 1, 20, 8, 1, 1, 1), 1.0, 1.0),
    km.pair(km.att(2, 2, 8, 24, 0.3), km.dlt(6, 2, 4, 40, 4, 40, 2), 0.5, 0.9),
    km.pair(km.att(3, 1, 16, 16, 0.5, chunk=1000, rot=2), km.dlt(3, 3, 64, 16, 2, 16, 16), 0.8, 0.6)])
@pytest.mark.parametrize("mlp", [None, km.ff(52)])
def test_a_layer_alone(tmp_path, mixer, mlp):
    """One layer, with a feed-forward and without, whole and token by token: scans of every spread of the states over
    lanes, either half of a pair alone (the other's scale is zero), negative scales, chunks of one place and wider than
    the requests, no chunks and no rotation, narrow projections of one number and wider than the heads."""
    from pih_b200.engine.factory import create_runner
    d = km.write_model(tmp_path / "m", km.single_layer(mixer, mlp), seed=3, sigma=0.2)
    requests = traces.make_requests(120, [40, 7], seed=2)
    truth = km.plain_logits(d, requests)
    for family in ("whole", "tail_decode"):
        _, model, cache, runner = create_runner(d, "float32", page_size=8, max_cache_tokens=64, max_requests=2)
        _check(traces.replay(runner, getattr(traces, family)(requests)), truth, "float32", family)
        model.rt.ops.check_errors()


@pytest.mark.parametrize("loop", [None, (0, 1, 1), (0, 1, 4), (0, 2, 2), (1, 2, 3)])
def test_loops(tmp_path, loop):
    """No loop, one pass, several passes of the first, of all and of the last layers; every pass finds its own keys and
    states again when the request goes on."""
    from pih_b200.engine.factory import create_runner
    raw = km.single_layer(km.pair(LEFT, RIGHT, 0.6, 1.4), km.ff(20))
    raw["layers"].append(km.layer(SCAN))
    if loop is not None:
        raw["loop"] = dict(zip(("start", "stop", "times"), loop))
    d = km.write_model(tmp_path / "m", raw, seed=6, sigma=0.2)
    requests = traces.make_requests(120, [30, 3], seed=2)
    for family in ("portions", "mixed"):
        _, model, cache, runner = create_runner(d, "float32", page_size=8, max_cache_tokens=128, max_requests=4)
        _check(traces.replay(runner, getattr(traces, family)(requests)), km.plain_logits(d, requests), "float32", family)
        model.rt.ops.check_errors()


def _step(positions, request_of_row, cu_q, slots=None):
    t = lambda v: torch.tensor(v, dtype=torch.int32, device=DEV)
    slots = list(range(len(cu_q) - 1)) if slots is None else slots
    return SimpleNamespace(positions=t(positions), request_of_row=t(request_of_row), cu_q=t(cu_q), state_slots=t(slots),
                           num_requests=len(slots), host_cu_q=list(cu_q),
                           host_q_start=[positions[c] if c < len(positions) else 0 for c in cu_q[:-1]],
                           q_start=t([positions[c] if c < len(positions) else 0 for c in cu_q[:-1]]), meta=None, attention_plans={})


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("states", [1, 2, 3, 5, 8, 16, 24, 33, 64, 100, 128, 200])
def test_selective_scan_of_every_state_size(states, dtype):
    """Every spread of the states over lanes, a number of channels that is no multiple of a block's, rows that are no
    multiple of a chunk's: two requests of unequal length (one of padding between them) in two steps, from strided views,
    into a strided view, against plain loops; nothing beyond the state and no other slot is touched."""
    ops = _ops()
    g = torch.Generator().manual_seed(states)
    inner, lens, cut = 37, [53, 18], 21
    T = sum(lens)
    u, z = (torch.randn(T, inner, generator=g).to(dtype) for _ in range(2))
    bc = torch.randn(T, 2 * states, generator=g).to(dtype)
    dt = torch.randn(T, inner, generator=g) * 2 - 1
    bias, D = torch.randn(inner, generator=g), torch.randn(inner, generator=g)
    A = -torch.exp(torch.randn(inner, states, generator=g))
    state = torch.zeros(4, inner * states + 5, device=DEV)
    wide = lambda x: torch.cat([x, torch.full((x.shape[0], 3), 77.0).to(x.dtype)], dim=1).to(DEV)[:, :x.shape[1]]
    out = torch.full((T, inner + 2), 5.0, dtype=dtype, device=DEV)
    got = torch.zeros(T, inner, dtype=F64)

    def run(rows, cu, slots):
        sel = torch.tensor(rows)
        ops.selective_scan(wide(u[sel]), wide(dt[sel]), wide(bc[sel]), wide(z[sel]), dt_bias=bias.to(DEV), A=A.to(DEV),
                           D=D.to(DEV), state=state, step=_step([0] * len(rows), [0] * len(rows), cu, slots), scale=0.75,
                           out=out[:len(rows), 1:inner + 1])
        assert bool((out[:, 0] == 5.0).all()) and bool((out[:, -1] == 5.0).all())
        got[sel] = out[:len(rows), 1:inner + 1].double().cpu()

    run(list(range(cut)) + list(range(lens[0], T)), [0, cut, cut, cut + lens[1]], [3, -1, 0])
    run(list(range(cut, lens[0])), [0, lens[0] - cut], [3])
    ops.check_errors()
    ref, S_end, at = [], [], 0
    for n in lens:
        rows = slice(at, at + n)
        y, S = plain.selective_scan(u[rows].double(), plain.softplus(dt[rows].double() + bias.double()), A.double(),
                                    bc[rows, :states].double(), bc[rows, states:].double(), D.double(),
                                    torch.zeros(inner, states, dtype=F64))
        ref.append(0.75 * y * plain.silu(z[rows].double()))
        S_end.append(S.flatten())
        at += n
    ref = torch.cat(ref)
    tol = 2e-5 if dtype == torch.float32 else 5e-3                # (bfloat16: the rounding of the output)
    assert float((got - ref).abs().max()) < tol * float(ref.abs().max())
    held = state.double().cpu()
    for slot, S in ((3, S_end[0]), (0, S_end[1])):
        assert float((held[slot, :inner * states] - S).abs().max()) < (2e-5 if dtype == torch.float32 else 1e-4) * float(S.abs().max())
    assert float(held[[1, 2]].abs().max()) == 0.0 and float(held[:, -5:].abs().max()) == 0.0


def test_selective_scan_keeps_a_state_over_a_thousand_tokens():
    """States whose decay lies next to one: an input at token 0 is still there 1500 tokens later, fed in portions and
    token by token, to full 32-bit precision; a row's result is the same bit by bit wherever the portions are cut."""
    ops = _ops()
    inner, n, T = 16, 8, 1500
    A = -torch.tensor([1e-6, 1e-5, 1e-4, 1e-3, 3e-3, 1e-2, 0.1, 1.0], dtype=F64).float()[None, :].repeat(inner, 1)
    u = torch.zeros(T, inner)
    u[0], u[700] = 1.0, -0.5
    dt = torch.full((T, inner), 0.3)
    ones = torch.ones(T, 2 * n)
    z = torch.full((T, inner), 2.0)
    zeros = torch.zeros(inner, device=DEV)

    def run(cuts):
        state, outs, at = torch.zeros(1, inner * n, device=DEV), [], 0
        for c in cuts:
            sl = slice(at, at + c)
            outs.append(ops.selective_scan(u[sl].to(DEV), dt[sl].to(DEV), ones[sl].to(DEV), z[sl].to(DEV), dt_bias=zeros,
                                           A=A.to(DEV), D=zeros, state=state, step=_step([0] * c, [0] * c, [0, c])))
            at += c
        ops.check_errors()
        return torch.cat(outs).cpu(), state.cpu()

    whole, end = run([T])
    cut, cut_end = run([640, 2, 63] + [1] * 40 + [755])
    assert torch.equal(whole, cut) and torch.equal(end, cut_end)
    ref, S = plain.selective_scan(u.double(), plain.softplus(dt.double()), A.double(), ones[:, :n].double(), ones[:, n:].double(),
                                  torch.zeros(inner, dtype=F64), torch.zeros(inner, n, dtype=F64))
    assert float(S[0, 0].abs()) > 0.3                                             # the slowest state still remembers
    assert float(((end.double().view(inner, n) - S).abs() / S.abs().clamp(min=1e-3)).max()) < 1e-4
    ref = ref * plain.silu(z.double())
    assert float((whole.double() - ref).abs().max()) < 1e-4 * float(ref.abs().max())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("dim, vdim", [(16, 24), (32, 32), (48, 40), (64, 70), (128, 128), (256, 64), (40, 8), (20, 7)])
@pytest.mark.parametrize("logits", ["rows", "wide"])
def test_delta_rule_with_a_decay_a_channel_of_every_key_size(dim, vdim, logits, dtype):
    """The register kernel's instances and the shared-memory kernel with one decay a head and key channel, decay logits of
    the rows' type and 32-bit ones, value sizes that are no multiple of a block's columns, two requests in two steps."""
    ops = _ops()
    g = torch.Generator().manual_seed(dim + vdim)
    heads, kv_heads, lens, cut = 4, 2, [37, 9], 20
    T, QK, VS = sum(lens), kv_heads * dim, heads * vdim
    qkv = (torch.randn(T, 2 * QK + VS, generator=g) * 0.7).to(dtype)
    beta = torch.randn(T, heads, generator=g).to(dtype)
    a = torch.randn(T, heads * dim, generator=g)
    a = a.to(dtype) if logits == "rows" else a
    log, bias = torch.randn(heads, generator=g) * 0.5 - 1.0, torch.randn(heads * dim, generator=g) * 0.5
    state = torch.zeros(3, heads * dim * vdim + 5, device=DEV)
    got = torch.zeros(T, heads, vdim, dtype=F64)

    def run(rows, cu, slots):
        sel = torch.tensor(rows)
        got[sel] = ops.gated_delta_rule(qkv[sel].to(DEV), beta[sel].to(DEV), a[sel].to(DEV), decay_log=log.to(DEV),
                                        decay_bias=bias.to(DEV), state=state, step=_step([0] * len(rows), [0] * len(rows), cu, slots),
                                        heads=heads, kv_heads=kv_heads, key_dim=dim, value_dim=vdim, unit_eps=1e-6,
                                        q_scale=dim ** -0.5).double().cpu()

    run(list(range(cut)) + list(range(lens[0], T)), [0, cut, cut + lens[1]], [2, 0])
    run(list(range(cut, lens[0])), [0, lens[0] - cut], [2])
    ops.check_errors()
    x = qkv.double()
    q = plain.unit(x[:, :QK].view(T, kv_heads, dim)) * dim ** -0.5
    k = plain.unit(x[:, QK:2 * QK].view(T, kv_heads, dim))
    dec = torch.exp(-torch.exp(log.double())[None, :, None] * plain.softplus(a.double() + bias.double()).view(T, heads, dim))
    ref, at = [], 0
    for n, slot in zip(lens, (2, 0)):
        r = slice(at, at + n)
        o, S = plain.delta_rule(q[r], k[r], x[r, 2 * QK:].view(n, heads, vdim), dec[r], torch.sigmoid(beta[r].double()),
                                torch.zeros(heads, dim, vdim, dtype=F64))
        ref.append(o)
        held = state[slot, :-5].double().cpu().view(heads, dim, vdim)
        assert float((held - S).abs().max()) < 1e-4 * max(1.0, float(S.abs().max()))
        at += n
    ref = torch.cat(ref)
    assert float((got - ref).abs().max()) < 2e-5 * max(1.0, float(ref.abs().max()))
    assert float(state[1].abs().max()) == 0.0 and float(state[:, -5:].abs().max()) == 0.0


def test_a_channel_that_forgets_beside_channels_that_remember():
    """Values written under orthogonal keys; one key channel decays away at once, the others do not decay: 200 tokens
    later, over several steps, the state returns every value but the one under the forgetting channel."""
    ops = _ops()
    D, V, n = 32, 20, 232
    g = torch.Generator().manual_seed(3)
    keys = torch.eye(D)
    v = torch.randn(n, 1, V, generator=g)
    v[D:] = 0.0                                                                   # later tokens write nothing ...
    k = keys[torch.arange(n) % D].clone()
    qkv = torch.cat([k, k, v.reshape(n, V)], dim=1).to(DEV)
    beta = torch.full((n, 1), -40.0)
    beta[:D] = 40.0                                                               # ... and with no strength
    a = torch.full((n, D), -40.0)
    a[:, 7] = 40.0
    state = torch.zeros(1, D * V, device=DEV)
    outs, at = [], 0
    for cut in (5, 90, 1, 1, 2, 133):
        outs.append(ops.gated_delta_rule(qkv[at:at + cut], beta[at:at + cut].to(DEV), a[at:at + cut].to(DEV),
                                         decay_log=torch.zeros(1, device=DEV), decay_bias=torch.zeros(D, device=DEV), state=state,
                                         step=_step([0] * cut, [0] * cut, [0, cut]), heads=1, kv_heads=1, key_dim=D, value_dim=V,
                                         unit_eps=1e-6, q_scale=1.0))
        at += cut
    ops.check_errors()
    out = torch.cat(outs)[:, 0].cpu()
    for t in range(n - D, n):
        want = torch.zeros(V) if t % D == 7 else v[t % D, 0]
        assert float((out[t] - want).abs().max()) < 1e-4, t
    assert float((out[7] - v[7, 0]).abs().max()) < 1e-4                           # (it was there when it was written)


def _plain_rows(q, K, V, positions, scale, chunk, gate, group, window=0, keep=0):
    """softmax(q k scale) v over the keys of the row's chunk (and window, and the kept first keys), times the gate."""
    out = torch.zeros(q.shape[0], q.shape[1], V.shape[-1], dtype=F64)
    for t, p in enumerate(positions):
        js = [j for j in range(p + 1) if ((not chunk or j // chunk == p // chunk) and (not window or p - j < window)) or j < keep]
        for h in range(q.shape[1]):
            s = (K[js, h // group] @ q[t, h]) * scale
            out[t, h] = torch.softmax(s, dim=0) @ V[js, h // group]
            if gate is not None:
                out[t, h] *= torch.sigmoid(gate[t, h])
    return out


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rows_of_step", [260, 17, 5, 1])
@pytest.mark.parametrize("chunk, window, keep, dim, vdim", [
    (64, 0, 0, 64, 64), (50, 0, 0, 64, 64), (7, 0, 0, 64, 40), (150, 0, 0, 96, 128), (299, 0, 0, 64, 64), (1, 0, 0, 32, 64),
    (300, 0, 0, 64, 64), (128, 40, 0, 64, 64), (90, 0, 5, 64, 64), (50, 0, 0, 72, 136)])
def test_keys_that_stand_out_at_the_edges_of_chunks(dtype, rows_of_step, chunk, window, keep, dim, vdim):
    """Keys that score high wherever they are seen: on head 0 the last key of every chunk (the next chunk's rows must not
    see it), on head 1 the first key of every chunk (seen from the whole chunk), on head 2 the keys at page borders.  A
    prompt of several row tiles (the tensor-core kernel in bf16), short portions and single rows (the warp kernel, its keys
    cut into parts); also with a window inside the chunk and kept first keys; the output goes into a strided view, scaled."""
    ops = _ops()
    heads, kv_heads, page, n = 6, 3, 16, 300
    g = torch.Generator().manual_seed(chunk)
    V = torch.randn(n, kv_heads, vdim, generator=g, dtype=F64)
    K = 0.05 * torch.randn(n, kv_heads, dim, generator=g, dtype=F64)
    unit = torch.zeros(dim, dtype=F64)
    unit[3] = 1.0
    K[chunk - 1::chunk, 0] += 6.0 * unit
    K[::chunk, 1] += 6.0 * unit
    K[page - 1::page, 2] += 4.0 * unit
    K[::page, 2] += 4.0 * unit
    first = n - rows_of_step
    positions = list(range(first, n))
    q = 0.05 * torch.randn(rows_of_step, heads, dim, generator=g, dtype=F64) + 3.0 * unit
    gate = torch.randn(rows_of_step, heads, generator=g, dtype=F64)
    qd, Kd, Vd, gd = (x.to(dtype).double() for x in (q, K, V, gate))
    want = 0.6 * _plain_rows(qd, Kd, Vd, positions, 0.5, chunk, gd, heads // kv_heads, window, keep)
    pages = -(-n // page)
    order = torch.randperm(pages + 3, generator=g)[:pages]
    cache = torch.zeros(pages + 3, page, kv_heads * (dim + vdim), dtype=dtype, device=DEV)
    flat = torch.cat([Kd.reshape(n, -1), Vd.reshape(n, -1)], dim=1).to(dtype).to(DEV)
    for i in range(pages):
        rows = flat[i * page:(i + 1) * page]
        cache[order[i], :rows.shape[0]] = rows
    table = order.to(torch.int32).clone()
    if keep == 0 and window == 0:
        table[:(first - first % chunk) // page] = -1               # pages of finished chunks were given back
    out = torch.full((rows_of_step, heads * vdim + 6), 9.0, dtype=dtype, device=DEV)
    ops.window_attention(qd.to(dtype).reshape(rows_of_step, -1).contiguous().to(DEV), cache=cache,
                         block_table=table.to(DEV).reshape(1, -1).contiguous(),
                         step=_step(positions, [0] * rows_of_step, [0, rows_of_step]), scale=0.5, window=window, keep_first=keep,
                         softcap=0.0, bias=None, sink=None, gate=gd.to(dtype).to(DEV), heads=heads, kv_heads=kv_heads,
                         key_dim=dim, value_dim=vdim, chunk=chunk, scale_out=0.6, out=out[:, 2:2 + heads * vdim])
    ops.check_errors()
    assert bool((out[:, :2] == 9.0).all()) and bool((out[:, -4:] == 9.0).all())
    got = out[:, 2:2 + heads * vdim].double().cpu().reshape(rows_of_step, heads, vdim)
    limit = 1e-5 if dtype == torch.float32 else 2e-2
    assert float((got - want).abs().max()) < limit * float(want.abs().max())
    if rows_of_step == 260 and chunk in (64, 50) and window == 0 and keep == 0:
        # the check would see a fault: chunks that are one place longer or shorter give something else
        for other in (chunk + 1, chunk - 1):
            moved = 0.6 * _plain_rows(qd, Kd, Vd, positions, 0.5, other, gd, heads // kv_heads)
            assert float((moved - want).abs().max()) > 0.2 * float(want.abs().max())


@pytest.mark.parametrize("width", [6, 72, 1000, 1024, 2050, 4096, 9001, 20480])
def test_the_norm_with_what_a_pass_of_the_loop_adds(width):
    """h += scale (y + bias) + factor table[ids] + vector, then the norm; stored back, or for gathered rows not stored; each
    part also alone; sizes in 16-byte pieces, odd ones, and ones beyond what a thread keeps in registers."""
    ops = _ops()
    g = torch.Generator().manual_seed(width)
    rows = 7
    h0, y = torch.randn(rows, width, generator=g), torch.randn(rows, width, generator=g)
    table, ids = torch.randn(11, width, generator=g), torch.tensor([3, 0, 10, 10, 5, 1, 2], dtype=torch.int32)
    bias, vector, w = (torch.randn(width, generator=g) for _ in range(3))
    pick = torch.tensor([6, 0, 3], dtype=torch.int32)
    for dtype in (torch.float32, torch.bfloat16):
        yd, td = y.to(dtype), table.to(dtype)
        for parts in ("dbav", "d", "db", "da", "av", "v", "a", ""):
            kw = {}
            want = h0.double()
            if "d" in parts:
                kw.update(delta=yd.to(DEV), scale=0.35)
                want = want + 0.35 * (yd.double() + (bias.double() if "b" in parts else 0.0))
            if "b" in parts:
                kw.update(bias=bias.to(DEV))
            if "a" in parts:
                kw.update(again=(td.to(DEV), ids.to(DEV), 1.5))
                want = want + 1.5 * td.double()[ids.long()]
            if "v" in parts:
                kw.update(vector=vector.to(DEV))
                want = want + vector.double()
            normed = plain.rms_unit(want, 1e-5) * w.double()
            h = h0.to(DEV)
            out = ops.rmsnorm_stream(h, w.to(DEV), 1e-5, out_dtype=dtype, **kw)
            assert float((h.double().cpu() - want).abs().max()) < 1e-5
            assert float((out.double().cpu() - normed).abs().max()) < (3e-5 if dtype == torch.float32 else 4e-2)
            h = h0.to(DEV)
            out = ops.rmsnorm_stream(h, w.to(DEV), 1e-5, out_dtype=dtype, rows=pick.to(DEV), **kw)
            assert torch.equal(h.cpu(), h0)
            assert float((out.double().cpu() - normed[pick.long()]).abs().max()) < (3e-5 if dtype == torch.float32 else 4e-2)
    scaled = ops.embedding(table.bfloat16().to(DEV), ids.to(DEV), out_dtype=torch.float32, scale=0.3)
    assert float((scaled.double().cpu() - 0.3 * table.bfloat16().double()[ids.long()]).abs().max()) < 1e-6
    ops.check_errors()


@pytest.mark.parametrize("rows", [1, 8, 13, 40])
def test_the_product_with_bias_and_gelu(rows):
    """The few-rows product with a bias and the exact GELU in its epilogue gives the bits of the product followed by the
    activation's kernel (which is also what many rows run), and the values of the plain computation; sizes that the
    few-rows product does not take; the gated norm with a sigmoid into a strided view."""
    ops = _ops()
    g = torch.Generator().manual_seed(rows)
    for n, k in ((96, 64), (520, 256), (4096, 1024), (37, 50)):
        x = (torch.randn(rows, k, generator=g) * 0.5).bfloat16().to(DEV)
        w = (torch.randn(n, k, generator=g) * (2.0 / math.sqrt(k))).bfloat16().to(DEV)
        bias = torch.randn(n, generator=g).to(DEV)
        got = ops.linear_bias_gelu(x, w, bias)
        assert torch.equal(got, ops.activation(ops.linear(x, w), "gelu_erf", bias))
        ref = plain.gelu((x.double() @ w.double().T).bfloat16().double() + bias.double())
        assert float((got.double() - ref).abs().max()) < 0.02 * float(ref.abs().max())
        x32, w32 = x.float(), w.float()
        got = ops.linear_bias_gelu(x32, w32, bias)
        ref = plain.gelu(x.double() @ w.double().T + bias.double())
        assert float((got.double() - ref).abs().max()) < 1e-5 * float(ref.abs().max())
    z = torch.linspace(-8, 8, 401, dtype=torch.float32, device=DEV)[None, :]
    assert float((ops.activation(z, "gelu_erf").double() - plain.gelu(z.double())).abs().max()) < 2e-6
    o, gate, wv = torch.randn(rows, 3, 20, generator=g), torch.randn(rows, 70, generator=g), torch.randn(20, generator=g)
    for gate_dtype, dtype in ((torch.float32, torch.float32), (torch.float32, torch.bfloat16), (torch.bfloat16, torch.bfloat16)):
        gt = gate.to(gate_dtype)
        out = torch.full((rows, 64), 3.0, dtype=dtype, device=DEV)
        ops.gated_rmsnorm(o.to(DEV), gt.to(DEV)[:, 4:64], wv.to(DEV), 1e-5, activation="sigmoid", scale=1.7, out=out[:, 2:62])
        ref = 1.7 * plain.rms_unit(o.double(), 1e-5) * wv.double() * torch.sigmoid(gt[:, 4:64].double()).view(rows, 3, 20)
        err = (out[:, 2:62].double().cpu() - ref.reshape(rows, 60)).abs().max()
        assert float(err) < (1e-5 if dtype == torch.float32 else 3e-2) and bool((out[:, :2] == 3.0).all()) and bool((out[:, 62:] == 3.0).all())
    ops.check_errors()


@pytest.mark.parametrize("name", ["K1", "K2"])
def test_batches_against_each_request_alone(dirs, name):
    """Unequal requests side by side in one step — a long portion, a short one, single tokens — give each request
    what it gets alone (32-bit: every reduction has an order fixed by the row)."""
    from pih_b200.engine import StepEntry
    from pih_b200.engine.factory import create_runner
    requests = traces.make_requests(km.CONFIGS[name]["vocab"], [61, 18, 40, 9], seed=8)
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


@pytest.mark.parametrize("seed", range(10))
def test_configurations_drawn_at_random(tmp_path, seed):
    """Sizes, orders of layers, loops and constants drawn at random (odd sizes and sizes that only the plain kernels take
    among them): a mixed schedule in 32-bit against the plain implementation position by position, and in bfloat16 within
    rounding."""
    from pih_b200.engine.factory import create_runner
    raw = km.random_config(seed)
    requests = traces.make_requests(raw["vocab"], [70, 45, 33, 18, 1, 2], seed=seed)
    steps = traces.mixed(requests, seed=seed, max_live=3)
    d = km.write_model(tmp_path / "m", raw, seed=seed, sigma=0.15)
    kw = dict(page_size=16, max_cache_tokens=traces.peak_tokens(steps, round_to=16), max_requests=3)
    for dtype in ("float32", "bfloat16"):
        _, model, cache, runner = create_runner(d, dtype, **kw)
        got = traces.replay(runner, steps)
        model.rt.ops.check_errors()

        def rounding():
            from fake_ops import FakeOps
            _, _, _, plain_runner = create_runner(d, dtype, device="cpu", ops=FakeOps(), **kw)
            return _errors(traces.replay(plain_runner, steps), km.plain_logits(d, requests))

        _check(got, km.plain_logits(d, requests), dtype, f"seed {seed} {dtype}", rounding=rounding)
        cache.check()


def test_long_decoding(dirs):
    """A short prompt and 300 tokens one by one: pages fill and go back chunk by chunk, the states run on."""
    from pih_b200.engine.factory import create_runner
    for name in ("K1", "K3"):
        requests = traces.make_requests(km.CONFIGS[name]["vocab"], [310], seed=9)
        steps = traces.tail_decode(requests, tail=300)
        _, model, cache, runner = create_runner(dirs[name], "float32", page_size=8, max_cache_tokens=320, max_requests=1)
        _check(traces.replay(runner, steps), km.plain_logits(dirs[name], requests), "float32", f"{name} long decoding")
        model.rt.ops.check_errors()


@pytest.mark.parametrize("cuda_graphs", [False, True])
@pytest.mark.parametrize("name", ["K1", "K2", "K3"])
def test_greedy_generation_through_the_engine(dirs, name, cuda_graphs):
    """Engine.complete (scheduler, cache, sampler, graphs, padded steps, ids fed on the device) against greedy decoding
    with the plain implementation; three requests at once with room for two, so they queue."""
    from pih_b200.engine import Engine
    cfg, w = km.load_plain(dirs[name])
    prompts = list(traces.make_requests(km.CONFIGS[name]["vocab"], [9, 21, 5], seed=13).values())
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
    requests = traces.make_requests(km.K1["vocab"], [33, 20, 47], seed=17)
    logits = []
    for graphs in (False, True):
        _, model, cache, runner = create_runner(dirs["K1"], dtype, page_size=16, max_cache_tokens=512, max_requests=4,
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
    """bin/pih-worker makes a random Kedavik model from a configuration file and generates from it; bin/trace_run replays
    a trace on it, in both precisions; all agree with the plain implementation."""
    import json
    import os
    import subprocess
    import sys

    import numpy as np
    from conftest import ROOT
    worker = [sys.executable, os.path.join(ROOT, "bin", "pih-worker")]
    cfg_file = tmp_path / "config.json"
    cfg_file.write_text(json.dumps(km.K2))
    folder = str(tmp_path / "made")
    proc = subprocess.run(worker + ["--random-model", folder, "--config", str(cfg_file), "--seed", "4", "--sigma", "0.15"],
                          capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    prompt = [5, 17, 3, 200, 9]
    proc = subprocess.run(worker + ["--model", folder, "--generate-tokens", ",".join(map(str, prompt)), "--max-tokens", "7",
                                    "--dtype", "float32", "--ignore-eos"], capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    res = json.loads(proc.stdout.strip().splitlines()[-1])
    cfg, w = km.load_plain(folder)
    toks = list(prompt)
    for _ in range(7):
        toks.append(int(plain.model_layers(cfg, w, toks)[1][-1].argmax()))
    assert res["token_ids"] == toks[len(prompt):]

    requests = traces.make_requests(km.K2["vocab"], [40, 9, 23], seed=6)
    steps = traces.mixed(requests, seed=1, max_live=3)
    for s_ in steps:
        for e in s_["entries"]:
            e["want"] = e["want"][-1:]                              # the last place of every portion
    truth = km.plain_logits(folder, requests)
    for dtype, tol in (("float32", 1e-4), ("bfloat16", 0.1)):
        out_dir = str(tmp_path / dtype)
        cmd = [sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", dtype, "--out", out_dir,
               "--max-tokens", str(traces.peak_tokens(steps))]
        proc = subprocess.run(cmd, input="\n".join(json.dumps(s_) for s_ in steps) + "\n", capture_output=True, text=True,
                              timeout=600)
        assert proc.returncode == 0, proc.stderr[-2000:]
        assert [l for l in proc.stdout.splitlines() if l.startswith("done ")] == [f"done {s_['step']}" for s_ in steps]
        at = {rid: 0 for rid in requests}
        for s_ in steps:
            got = np.fromfile(os.path.join(out_dir, f"{s_['step']}.f32"), dtype="<f4").reshape(-1, km.K2["vocab"])
            for j, e in enumerate(s_["entries"]):
                at[e["id"]] += len(e["tokens"])
                ref = truth[e["id"]][at[e["id"]] - 1].numpy()
                assert np.abs(got[j] - ref).max() < tol * max(1.0, np.abs(ref).max()), (s_["step"], e["id"])
