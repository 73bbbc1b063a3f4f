"""Getozen on the GPU: every mechanism against the plain implementation, then whole models
through the step function under every kind of schedule, the scheduler and the trace program."""

import copy

import pytest
import torch

import getozen_helpers as gh
import helpers
from plain import getozen_plain as plain

pytestmark = pytest.mark.gpu

DTYPES = [torch.float32, torch.bfloat16]
DEV = "cuda:0"


def _ops():
    from paged_attention_engine_b200.kernels import ops

    return ops


def _close(got, want, dtype, scale=1.0):
    tol = (2e-5 if dtype == torch.float32 else 2.0 ** -6) * scale * max(1.0, float(want.abs().max()))
    gap = float((got.double().cpu() - want.double()).abs().max())
    assert gap <= tol, f"max difference {gap} > {tol}"


dev = lambda t: t.to(DEV).contiguous()
ints = lambda values: torch.tensor(values, dtype=torch.int32, device=DEV)


# --------------------------------------------------------------------------- #
# Mechanisms alone
# --------------------------------------------------------------------------- #

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens, width, planes", [(1, 48, (1, 1)), (7, 64, (3, 24)), (5, 257, (9, 2)), (300, 1024, (2, 1))])
def test_two_norms_of_a_stream_and_the_sum_of_two_sublayers(dtype, tokens, width, planes):
    """x + a + b, the outputs tensors or planes of split products, and both norms of the sum in one
    kernel: the numbers of the single steps."""
    ops = _ops()
    gen = torch.Generator().manual_seed(tokens + width)
    x = torch.randn(tokens, width, generator=gen) * 2.0
    outs = [torch.randn(n, tokens, width, generator=gen) for n in planes]
    names = {}
    for n in ("a", "b"):
        names.update({n: torch.randn(width, generator=gen), f"{n}.alpha": torch.rand((), generator=gen) + 0.3,
                      f"{n}.b": torch.randn(width, generator=gen) * 0.3})
    norm = lambda n: (dev(names[f"{n}.alpha"].reshape(1)), dev(names[n]), dev(names[f"{n}.b"]))
    want = x.double() + sum(o.double().sum(0) for o in outs)
    sublayer = lambda o: ops.PendingSum(dev(o), None, None, torch.float32) if o.shape[0] > 1 else dev(o[0])
    pending = ops.residual_add(dev(x), sublayer(outs[0]), 1.0, y2=sublayer(outs[1]))
    a, b = ops.dyt_norm_pair(pending, norm("a"), norm("b"), dtype)
    _close(pending.value, want, torch.float32)
    _close(a, plain.dynamic_tanh(want, names, "a"), dtype)
    _close(b, plain.dynamic_tanh(want, names, "b"), dtype)
    alone = ops.dyt_norm_pair(pending.value, norm("a"), norm("b"), dtype)
    assert torch.equal(alone[0], a) and torch.equal(alone[1], b)
    assert torch.equal(ops.dyt_norm(pending.value, *norm("b"), dtype), b)
    again = ops.residual_add(dev(x), sublayer(outs[0]), 1.0, y2=sublayer(outs[1]))
    assert torch.equal(ops.materialized(again), pending.value)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("neighbours", [True, False])
@pytest.mark.parametrize("heads, kv_heads, d, dv, dims, tokens", [
    (4, 2, 64, 128, 64, 70), (3, 1, 24, 8, 16, 5), (2, 2, 12, 20, 8, 9), (1, 1, 8, 16, 2, 3), (5, 5, 48, 48, 0, 300), (2, 1, 128, 128, 96, 1)])
def test_rotation_in_both_pairings_into_pages_and_into_rows(dtype, neighbours, heads, kv_heads, d, dv, dims, tokens):
    """Sizes that split into pieces of eight channels and sizes that do not; a span shorter than the head; a
    projection that starts beyond column 0; queries as leading columns of wider rows; a token without a page."""
    ops = _ops()
    gen = torch.Generator().manual_seed(heads * d + dims)
    off = 8
    proj = torch.randn(tokens, off + (heads + kv_heads) * d + kv_heads * dv, generator=gen)
    first = 1000
    rot = gh.rot(dims, 5000.0, 3.0) if dims else None
    q = proj[:, off: off + heads * d].double().view(tokens, heads, d)
    k = proj[:, off + heads * d: off + (heads + kv_heads) * d].double().view(tokens, kv_heads, d)
    v = proj[:, off + (heads + kv_heads) * d:].view(tokens, kv_heads, dv)
    table = None
    if rot:
        q, k = plain.rotate(q, rot, neighbours, first), plain.rotate(k, rot, neighbours, first)
        freqs = torch.tensor(plain.frequencies(rot), dtype=torch.float64).float()
        table = ops.rotary_table(dev(torch.arange(first, first + tokens, dtype=torch.int32)), dev(freqs))
    page = 4
    pages = tokens // page + 2
    keys = torch.zeros(pages, kv_heads, page, d, dtype=dtype, device=DEV)
    values = torch.zeros(pages, kv_heads, page, dv, dtype=dtype, device=DEV)
    slots = torch.arange(page, page + tokens, dtype=torch.int32, device=DEV)
    slots[tokens // 2] = -1
    wide = torch.full((tokens, (heads + 2 * kv_heads) * d), 7.0, dtype=dtype, device=DEV)
    common = dict(q_off=off, k_off=off + heads * d, v_off=off + (heads + kv_heads) * d, heads=heads, kv_heads=kv_heads, q_dim=d, k_dim=d,
                  value_dim=dv, q_norm=None, k_norm=None, q_span=0, k_span=0, eps=0.0, table=table, interleaved=neighbours, q_rot0=0,
                  k_rot0=0, out_dtype=dtype)
    got = ops.head_prep(dev(proj), slots=slots, keys=keys, values=values, page_size=page, q_out=wide, **common)
    scale = 8.0                                     # the angle of a position of a thousand is a float32 product
    _close(got[:, : heads * d].reshape(tokens, heads, d), q, dtype, scale)
    assert bool((got[:, heads * d:] == 7.0).all())
    has_page = torch.arange(tokens) != tokens // 2
    stored = keys.permute(0, 2, 1, 3).reshape(-1, kv_heads, d)[page: page + tokens]
    _close(stored[has_page.to(DEV)], k[has_page], dtype, scale) if tokens > 1 else None
    assert not bool(stored[tokens // 2].any())
    stored_v = values.permute(0, 2, 1, 3).reshape(-1, kv_heads, dv)[page: page + tokens]
    assert torch.equal(stored_v[has_page.to(DEV)].cpu(), v[has_page].to(dtype))
    rows_k = torch.empty(tokens, kv_heads * d, dtype=dtype, device=DEV)
    rows_v = torch.empty(tokens, kv_heads * dv, dtype=dtype, device=DEV)
    direct = ops.head_prep(dev(proj), slots=None, keys=rows_k, values=rows_v, page_size=1, direct=True, **common)
    assert torch.equal(direct, got[:, : heads * d])
    _close(rows_k.view(tokens, kv_heads, d), k, dtype, scale)
    assert torch.equal(rows_v.view(tokens, kv_heads, dv).cpu(), v.to(dtype))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens, width, group, ld", [(1, 64, 1, 200), (33, 24, 1, 50), (300, 1024, 1, 2048), (9, 48, 12, 17)])
def test_gate_into_a_column_range(dtype, tokens, width, group, ld):
    ops = _ops()
    gen = torch.Generator().manual_seed(width)
    x = torch.randn(tokens, width, generator=gen).to(dtype)
    rows = torch.randn(tokens, ld, generator=gen) * 2.0
    gate_off, out_off = 8 if group == 1 else 5, 4
    want = 1.7 * x.double() * torch.sigmoid(rows[:, gate_off: gate_off + width // group].double()).repeat_interleave(group, dim=1)
    out = torch.full((tokens, width + 12), 3.0, dtype=dtype, device=DEV)
    ops.sigmoid_gate(dev(x), dev(rows), gate_off, group=group, mult=1.7, out=out, out_off=out_off)
    _close(out[:, out_off: out_off + width], want, dtype)
    assert bool((out[:, :out_off] == 3.0).all()) and bool((out[:, out_off + width:] == 3.0).all())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("tokens, inter, k", [(1, 64, 128), (8, 320, 192), (20, 256, 256), (40, 160, 64), (130, 256, 128), (5, 24, 36), (70, 40, 64)])
def test_gated_unit_of_a_rectifier(dtype, tokens, inter, k):
    """relu(x Wg) * (x Wu): inside the product for few and many tokens, in the sum of its splits, alone."""
    ops = _ops()
    gen = torch.Generator().manual_seed(tokens + inter)
    x = torch.randn(tokens, k, generator=gen).to(dtype)
    gate, up = ((torch.randn(inter, k, generator=gen) / k ** 0.5).to(dtype) for _ in range(2))
    want = torch.relu(x.double() @ gate.double().T) * (x.double() @ up.double().T)
    both = ops.linear(dev(x), dev(torch.cat([gate, up])))
    _close(ops.silu_mul(both, gate="relu"), want, dtype, 2.0)
    mixed = ops.interleave_gate_up(dev(gate), dev(up))
    if inter % 16:
        assert mixed is None
    else:
        _close(ops.linear_swiglu(dev(x), mixed, gate="relu"), want, dtype, 2.0)
    ops.check_device_errors()


# requests as (tokens before this step, tokens of this step)
MIXES = [
    [(0, 1)],
    [(5, 2), (0, 1), (300, 1), (0, 3)],
    [(0, 127), (9, 128), (0, 129), (4, 1)],
    [(0, 300), (130, 65), (7, 1), (0, 1), (33, 64)],
]


def _memory_case(seed, heads, groups, n, dv, requests, mode):
    """Operands of a whole sequence per request, and the plain outputs and states with every sequence
    cut where the step begins."""
    gen = torch.Generator().manual_seed(seed)
    case = {"q": [], "k": [], "v": [], "keep": [], "step": [], "want": [], "start": [], "end": []}
    group = [h // (heads // groups) for h in range(heads)]
    skip = torch.randn(heads, generator=gen)
    decay = torch.rand(heads, generator=gen) ** 0.05
    if heads > 1:
        decay[0], decay[1] = 1.0, 0.0                # one head that keeps everything, one that keeps nothing
    for past, new in requests:
        T = past + new
        q, k = (torch.randn(T, groups, n, generator=gen).to(torch.bfloat16) for _ in range(2))
        v = torch.randn(T, heads, dv, generator=gen).to(torch.bfloat16)
        if mode == "chosen":
            rate = torch.exp(torch.rand(heads, generator=gen) * 8.0 - 6.0)
            step = torch.rand(T, heads, generator=gen) * 2.0
            step[T // 2] = 60.0                         # a token after which hardly anything of the past is left
            log_decay = -rate * step
        else:
            step, log_decay = torch.full((T, heads), float(n) ** -0.5), torch.log(decay).expand(T, heads)
        keep = torch.exp(log_decay.double())
        o, _ = plain.decayed_memory(q.double()[:, group], step.double()[:, :, None] * k.double()[:, group], v.double(), keep)
        _, start = plain.decayed_memory(q.double()[:past, group], step.double()[:past, :, None] * k.double()[:past, group], v.double()[:past], keep[:past])
        _, end = plain.decayed_memory(q.double()[past:, group], step.double()[past:, :, None] * k.double()[past:, group], v.double()[past:], keep[past:], start)
        o = o + skip.double()[:, None] * v.double()
        for name, t in (("q", q), ("k", k), ("v", v), ("keep", log_decay), ("step", step), ("want", o)):
            case[name].append(t[past:])
        case["start"].append(start)
        case["end"].append(end)
    case.update(skip=skip, decay=decay)
    return case


@pytest.mark.parametrize("dtype, form", [(torch.float32, None), (torch.bfloat16, None), (torch.bfloat16, "scan")])
@pytest.mark.parametrize("mode", ["chosen", "fixed"])
@pytest.mark.parametrize("heads, groups, n, dv", [(4, 2, 32, 32), (3, 3, 64, 128), (6, 1, 16, 24), (2, 2, 136, 72), (4, 4, 10, 6), (1, 1, 7, 5),
                                                  (2, 1, 256, 64), (2, 1, 520, 16)])
def test_decaying_memory_in_every_form(dtype, form, mode, heads, groups, n, dv):
    """Single tokens, short and long portions on both sides of a chunk's end, from a state that earlier
    tokens left, in a pool whose other slots hold NaN and stay as they are."""
    ops = _ops()
    for seed, requests in enumerate(MIXES if n <= 136 else MIXES[1:3]):
        case = _memory_case(seed, heads, groups, n, dv, requests, mode)
        slots = torch.randperm(len(requests) + 3, generator=torch.Generator().manual_seed(seed)).tolist()[: len(requests)]
        pool = torch.full((len(requests) + 3, heads * n * dv + 8), float("nan"))
        for slot, start in zip(slots, case["start"]):
            pool[slot, : heads * n * dv] = start.float().flatten()
        pool = dev(pool)
        state = pool[:, : heads * n * dv]
        cat = lambda name, width: dev(torch.cat(case[name]).reshape(-1, width))
        # q, k and v as column ranges of one matrix
        rows = torch.cat([cat("v", heads * dv), cat("k", groups * n), cat("q", groups * n)], dim=1).to(dtype).contiguous()
        q_start = [0]
        for _, new in requests:
            q_start.append(q_start[-1] + new)
        lens = [new for _, new in requests]
        singles = sum(1 for x in lens if x == 1)
        multi = [i for i, x in enumerate(lens) if x > 1]
        extra = dict(log_decay=cat("keep", heads), step=cat("step", heads)) if mode == "chosen" else dict(
            head_decay=dev(case["decay"]), k_scale=float(n) ** -0.5)
        got = ops.decay_memory((rows, heads * dv + groups * n), (rows, heads * dv), (rows, 0), state, ints(q_start), ints(slots), len(requests),
                               heads, groups, n, dv, skip=dev(case["skip"]), max_q_len=max(lens), num_single=singles,
                               multi_index=ints(multi) if 0 < len(multi) < len(lens) else None, form=form, **extra)
        # bfloat16 operands are exact here: what is left is the arithmetic, which is not 16-bit in any form
        _close(got, torch.cat(case["want"]).reshape(-1, heads * dv), torch.float32, 3.0 if dtype == torch.bfloat16 else 1.0)
        for slot, end in zip(slots, case["end"]):
            _close(state[slot].view(heads, n, dv), end, torch.float32, 3.0 if dtype == torch.bfloat16 else 1.0)
        for slot in set(range(len(requests) + 3)) - set(slots):
            assert bool(torch.isnan(pool[slot]).all())
        assert bool(torch.isnan(pool[:, heads * n * dv:]).all())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads, dv, n, groups, taps, planes", [(4, 16, 8, 2, 4, 1), (3, 5, 7, 1, 3, 1), (2, 64, 64, 1, 2, 3), (8, 12, 4, 4, 1, 2),
                                                                (2, 8, 12, 1, 17, 1), (5, 4, 3, 5, 6, 2)])
def test_convolution_steps_and_decays_of_a_state_space(dtype, heads, dv, n, groups, taps, planes):
    """The convolution across portions of one, two and many tokens whose earlier rows are in the state, zeros
    before the start; steps and decays of small and large pre-activations; planes of a split product."""
    ops = _ops()
    gen = torch.Generator().manual_seed(heads * dv + taps)
    inner, channels = heads * dv, heads * dv + 2 * groups * n
    ld = 4 + inner + channels + heads
    w = torch.rand(channels, taps, generator=gen) * 2.0 - 1.0
    bias, dt_bias, a_log = torch.randn(channels, generator=gen), torch.randn(heads, generator=gen) * 3.0, torch.randn(heads, generator=gen)
    portions = [[1, 2, 40], [2, 1, 1], [17, 5, 33], [1, 1, 16]]          # per request, the tokens of each step
    rows = [torch.randn(sum(p), ld, generator=gen) * 3.0 for p in portions]
    for r in rows:
        r[0, -heads:] = 40.0                      # softplus of a large number is the number
    floats = (taps - 1) * channels
    pool = torch.full((7, floats + 3), float("nan"))
    slots = [5, 0, 3, 2]
    pool[slots, : floats] = 0.0
    pool = dev(pool)
    at = [0] * len(portions)
    for s in range(3):
        lens = [p[s] for p in portions]
        flat = torch.cat([r[a: a + n_] for r, a, n_ in zip(rows, at, lens)])
        proj = dev(flat)
        if planes > 1:
            parts = torch.randn(planes, *flat.shape, generator=gen)
            parts[-1] = flat - parts[:-1].sum(0)
            proj = ops.PendingSum(dev(parts), None, None, torch.float32)
        q_start = [0]
        for n_ in lens:
            q_start.append(q_start[-1] + n_)
        u, step, log_decay, (gate, gate_off) = ops.ssm_prepare(
            proj, 4, inner, 4 + inner, channels, 4 + inner + channels, heads, dev(w), dev(bias), dev(dt_bias), dev(a_log),
            pool[:, : floats], ints(q_start), ints(at), ints(slots), len(lens), max(lens), dtype)
        scale = 1.0 if planes == 1 else 4.0
        for i, (r, a, n_) in enumerate(zip(rows, at, lens)):
            here = slice(q_start[i], q_start[i + 1])
            want = plain.silu(plain.short_convolution(r[: a + n_, 4 + inner: 4 + inner + channels].double(), w, bias))[a:]
            _close(u[here], want, dtype, scale)
            dt = plain.softplus(r[a: a + n_, -heads:].double() + dt_bias.double())
            _close(step[here], dt, torch.float32, scale)
            _close(log_decay[here], -torch.exp(a_log.double()) * dt, torch.float32, scale)
            _close(gate[here, gate_off: gate_off + inner], r[a: a + n_, 4: 4 + inner].double(), torch.float32, scale)
        at = [a + n_ for a, n_ in zip(at, lens)]
    for slot in set(range(7)) - set(slots):
        assert bool(torch.isnan(pool[slot]).all())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("gate_first", [True, False])
@pytest.mark.parametrize("tokens, groups, size", [(1, 1, 64), (9, 3, 7), (300, 8, 384), (5, 2, 1500), (3, 1, 3072), (17, 12, 128)])
def test_norm_of_channel_groups_with_a_gate_before_or_after(dtype, gate_first, tokens, groups, size):
    ops = _ops()
    gen = torch.Generator().manual_seed(size)
    width = groups * size
    y = torch.randn(tokens, width, generator=gen) * torch.logspace(-3, 1, groups).repeat_interleave(size)      # groups of unequal size
    rows = torch.randn(tokens, width + 12, generator=gen) * 2.0
    weight = torch.randn(width, generator=gen)
    g = plain.silu(rows[:, 4: 4 + width].double())
    eps = 1e-3
    if gate_first:
        want = plain.unit_rms((y.double() * g).view(tokens, groups, size), eps).reshape(tokens, width) * weight.double()
    else:
        want = plain.unit_rms(y.double().view(tokens, groups, size), eps).reshape(tokens, width) * g
    out = torch.full((tokens, width + 8), 3.0, dtype=dtype, device=DEV)
    ops.gated_group_norm(dev(y), dev(rows), 4, groups, eps, dtype, weight=dev(weight) if gate_first else None, gate_first=gate_first, mult=0.6,
                         out=out, out_off=4)
    _close(out[:, 4: 4 + width], 0.6 * want, dtype)
    assert bool((out[:, :4] == 3.0).all()) and bool((out[:, 4 + width:] == 3.0).all())


# --------------------------------------------------------------------------- #
# Single parts of a model against the plain functions
# --------------------------------------------------------------------------- #

@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    root = tmp_path_factory.mktemp("getozen")
    return {name: gh.write_model(root / name, raw, seed) for name, (raw, _page, seed) in gh.SMALL.items()}


@pytest.fixture(scope="module")
def prompts(folders):
    """Per model: prompts and the plain model's logits for them."""
    out = {}
    for name, (raw, _page, seed) in gh.SMALL.items():
        requests = gh.random_requests(raw, [45, 9, 31, 1, 2, 150 if name in ("small_b", "wide") else 23], seed)
        out[name] = requests, {k: gh.plain_logits(folders[name], t) for k, t in requests.items()}
    return out


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name, index", [("small_a", 0), ("small_a", 1), ("small_a", 2), ("small_a", 5), ("small_b", 0), ("small_b", 1),
                                         ("small_b", 2), ("small_b", 3), ("ones", 0), ("ones", 2), ("wide", 0), ("wide", 1)])
def test_one_layer_mixer_in_portions(folders, name, index, dtype):
    """A mixer alone: a prompt in portions through its own pages and state, against the plain mixer."""
    from paged_attention_engine_b200.cache import CacheManager, PagedKVCache, plan_cache
    from paged_attention_engine_b200.config import resolve
    from paged_attention_engine_b200.engine.batch import BatchBuilder, StepEntry
    from paged_attention_engine_b200.parts import MIXERS, Runtime
    from paged_attention_engine_b200.weights import collect_tensor_specs, place_tensors

    raw, tensors = gh.read_model(folders[name])
    spec = resolve(raw)[1]
    ops = _ops()
    runtime = Runtime(ops, dtype, torch.device(DEV))
    entry = raw["layers"][index]
    position = index if "weights_of" not in entry else entry["weights_of"]
    layer = spec.layers[spec.schedule[index].layer]
    own = {k: v for k, v in place_tensors(tensors, spec, dtype, DEV).items() if k.startswith(f"l{position}.mix.")}
    assert set(own) == {k for k in collect_tensor_specs(spec) if k.startswith(f"l{position}.mix.")}
    part = MIXERS.get(layer.mixer.kind)(layer.mixer, own, runtime)
    gen = torch.Generator().manual_seed(index)
    h = (torch.randn(40, raw["width"], generator=gen)).to(dtype)
    want = plain.mixer(h.double(), tensors, f"l{position}.mix", entry["type"], entry["mixer"], raw["norm"]["eps"])
    plan = plan_cache(spec)
    manager = CacheManager(plan.groups, 24, 8, 2)
    cache = PagedKVCache(plan, manager, dtype, DEV)
    builder = BatchBuilder(manager, ops, dtype, DEV)
    slot = manager.create_request("r")
    cache.reset_state(slot)
    got, at = [], 0
    for n in (2, 1, 9, 1, 1, 2, 24):
        assert manager.reserve("r", n).ok
        ctx = builder.build([StepEntry("r", [0] * n, ())])
        y = part.forward(ctx, dev(h[at: at + n]), None, cache.entry_cache(index))
        got.append(ops.materialized(y).clone())
        assert got[-1].dtype == torch.float32
        manager.advance("r", n)
        at += n
    _close(torch.cat(got), want, dtype, scale=4.0)


# --------------------------------------------------------------------------- #
# Whole models through the step function
# --------------------------------------------------------------------------- #

def _check(folder, dtype, trace, requests, oracle, page, max_live=4, fragment=None, slack=1.0):
    from paged_attention_engine_b200.engine.llm import Engine
    from paged_attention_engine_b200.engine.replay import Replayer

    engine = Engine.from_pretrained(folder, dtype)
    replayer = Replayer(engine, helpers.max_live_tokens(trace, page), page, max_live)
    if fragment is not None and replayer.manager.groups:
        helpers.fragment_pool(replayer.manager, fragment)
    outputs = {}
    for record in trace:
        logits = replayer.run(record)
        if logits is not None:
            outputs[record["step"]] = logits.float().cpu()
    engine.runtime.ops.check_device_errors()
    got = helpers.collect(trace, outputs, requests)
    for key, want in oracle.items():
        gap = (got[key] - want).abs().max(dim=1).values
        allowed = slack * gh.row_tolerance(dtype, want, folder, requests[key])
        worst = int((gap - allowed).argmax())
        assert bool((gap <= allowed).all()), f"{key}: |dlogit| {float(gap[worst])} > {float(allowed[worst])} at position {worst}"
    assert not replayer.manager.live_requests()
    assert replayer.manager.num_free == replayer.manager.num_blocks
    return got


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(gh.SMALL))
def test_schedules_agree_with_the_plain_model(folders, prompts, name, dtype):
    """Prompts whole, decoded token by token, in portions down to two tokens, and in batches of
    unequal requests whose pages and state slots are used again."""
    raw, page, seed = gh.SMALL[name]
    requests, oracle = prompts[name]
    whole = _check(folders[name], dtype, helpers.trace_whole(requests), requests, oracle, page)
    tail = _check(folders[name], dtype, helpers.trace_tail(requests, tail=30), requests, oracle, page)
    chunks = _check(folders[name], dtype, helpers.trace_chunks(requests, seed), requests, oracle, page, fragment=seed)
    mixed = _check(folders[name], dtype, helpers.trace_mixed(requests, seed, live_limit=3, decode_tail=10), requests, oracle,
                   page, max_live=3, fragment=seed + 1)
    # How the tokens were cut, what else was in the batch and which pages and slots were used
    # changes a logit by rounding only.
    for key in requests:
        cut = 2e-5 * max(1.0, float(oracle[key].abs().max()))
        limit = torch.full((len(requests[key]),), cut) if dtype == torch.float32 else gh.row_tolerance(dtype, oracle[key], folders[name], requests[key])
        for other in (tail, chunks, mixed):
            assert bool(((other[key] - whole[key]).abs().max(dim=1).values <= limit).all())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["small_a", "small_b"])
def test_long_decoding_from_the_first_token(folders, name, dtype):
    raw, page, seed = gh.SMALL[name]
    requests = gh.random_requests(raw, [200], seed + 50)
    oracle = {"r0": gh.plain_logits(folders[name], requests["r0"])}
    _check(folders[name], dtype, helpers.trace_tail(requests, tail=199), requests, oracle, page)


def _portions(key, tokens, cuts):
    """A trace of one request whose portions end at `cuts`."""
    out = []
    for step, (a, b) in enumerate(zip([0] + list(cuts), list(cuts) + [len(tokens)])):
        out.append({"step": step, "entries": [helpers._entry(key, tokens[a:b])], "end": [key] if b == len(tokens) else []})
    return out


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_long_prompt_over_many_pages_and_chunks(folders, dtype):
    """600 tokens over 38 pages; cut on, just before and just after the borders of pages (16) and
    of the recurrence's chunks (128), which start anew with every portion."""
    raw, page, seed = gh.SMALL["small_b"]
    requests = gh.random_requests(raw, [600], seed + 9)
    oracle = {"r0": gh.plain_logits(folders["small_b"], requests["r0"])}
    runs = [helpers.trace_whole(requests), helpers.trace_tail(requests, tail=40)]
    runs += [_portions("r0", requests["r0"], cuts) for cuts in ((15, 16, 17, 144, 145, 273, 401), (128, 256, 257, 385, 512), (2, 4, 131, 260, 598))]
    results = [_check(folders["small_b"], dtype, trace, requests, oracle, page, fragment=3) for trace in runs]
    if dtype == torch.float32:
        cut = 2e-5 * max(1.0, float(oracle["r0"].abs().max()))
        for other in results[1:]:
            assert float((other["r0"] - results[0]["r0"]).abs().max()) <= cut


# --------------------------------------------------------------------------- #
# A token far back, through the keys and through each kind of state
# --------------------------------------------------------------------------- #

def _memory_model(tmp_path, kind):
    """One layer of one mechanism and a token that stands out: only its embedding has channel 0, and
    channel 1 is 0 in every embedding, so that behind the norm (bias 0 and 1 on these channels) channel 0
    is this token's alone and channel 1 the same constant for all. What it leaves is kept for good and
    read by every later token: an attention key that an unrotated channel of every query meets, a
    retention whose first head does not decay and whose unrotated channel it alone writes, a state space
    whose step is near zero except at this token."""
    from safetensors.torch import load_file, save_file

    if kind in ("left", "right"):
        layer = gh.parallel((2, 1, 32, 32, 0.18, gh.rot(16, 10000.0, 2.0)), (32, 32, (1.0, 1.0), gh.rot(16, 10000.0)),
                            (1.0, 0.0) if kind == "left" else (0.0, 1.0))
    else:
        layer = gh.mamba(2, 32, 16, 1, 3, 1)
    raw = gh.config(61, 64, [layer])
    folder = gh.write_model(tmp_path / kind, raw, 77)
    path = str(folder / "model.safetensors")
    tensors = load_file(path)
    inner = 64

    def write_in(t):
        t[2 * inner: 2 * inner + 16, 0] += 3.0       # B: the standing-out token writes with a weight of its own
        t[2 * inner + 16: 2 * inner + 32, 1] += 2.0  # C: every token reads it
        t[2 * inner + 32:].zero_()
        t[2 * inner + 32:, 0] = 8.0                  # the step: large at this token, tiny elsewhere (by its bias)

    changes = {"embed": lambda t: (t[:, 0].zero_(), t[:, 1].zero_(), t[60].mul_(3.0), t[60, 0].fill_(3.0)),
               "l0.norm1": lambda t: t[0].fill_(1.0), "l0.norm1.b": lambda t: (t[0].zero_(), t[1].fill_(1.0))}
    if kind in ("left", "right"):
        # channel 20 is beyond the rotated span of both: no position turns it
        changes.update({
            "l0.mix.left.k": lambda t: (t[20].zero_(), t[20, 0].fill_(6.0)), "l0.mix.left.k.b": lambda t: t[20].zero_(),
            "l0.mix.left.q": lambda t: (t[20].zero_(), t[20, 1].fill_(6.0), t[52].zero_(), t[52, 1].fill_(6.0)),
            "l0.mix.right.k": lambda t: (t.mul_(0.02), t[20].zero_(), t[20, 0].fill_(6.0), t[52].zero_(), t[52, 0].fill_(6.0)),
            "l0.mix.right.q": lambda t: (t.mul_(0.2), t[20, 1].fill_(6.0), t[52, 1].fill_(6.0)),
            "l0.mix.left.o": lambda t: t.mul_(10.0), "l0.mix.right.o": lambda t: t.mul_(10.0)})
    else:
        changes.update({"l0.mix.in": write_in, "l0.mix.dt_bias": lambda t: t.fill_(-9.0), "l0.mix.A_log": lambda t: t.fill_(-1.0),
                        "l0.mix.D": lambda t: t.mul_(0.02), "l0.mix.o": lambda t: t.mul_(10.0)})
    for name, change in changes.items():
        t = tensors[name].float()
        change(t)
        tensors[name] = t.to(torch.bfloat16)
    save_file(tensors, path)
    return raw, folder, tensors


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["left", "right", "mamba"])
@pytest.mark.parametrize("at, cuts", [(0, (1, 2, 150)), (15, (16, 128, 129, 131)), (127, (127, 128, 300)), (140, tuple(range(200, 330)))])
def test_a_token_far_back_is_still_there(tmp_path, dtype, kind, at, cuts):
    """The outstanding token stands first, before a page's end, at a chunk's end, inside a chunk; the
    portions part right at it, or later tokens come one by one. The logits hundreds of tokens on follow the plain
    model, and are far from the plain model of the same prompt without that token, so a lost state or key would show."""
    raw, folder, tensors = _memory_model(tmp_path, kind)
    tokens = gh.random_requests(dict(raw, vocab=60), [330], 5 + at)["r0"]
    without = list(tokens)
    tokens[at] = 60
    want = plain.forward(raw, tensors, tokens).float()
    lost = plain.forward(raw, tensors, without).float()
    got = _check(folder, dtype, _portions("r0", tokens, cuts), {"r0": tokens}, {"r0": want}, 16, fragment=at)["r0"]
    tol = gh.tolerance(torch.bfloat16, want)
    far = (lost[at + 150:] - got[at + 150:]).abs().max(dim=1).values
    assert float(far.median()) > 4.0 * tol, (kind, float(far.median()), tol)


# --------------------------------------------------------------------------- #
# Through the entry points
# --------------------------------------------------------------------------- #

def _plain_greedy(folder, prompt, count):
    raw, tensors = gh.read_model(folder)
    tokens = list(prompt)
    for _ in range(count):
        tokens.append(int(plain.forward(raw, tensors, tokens)[-1].argmax()))
    return tokens[len(prompt):]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["small_a", "small_b", "ones"])
def test_greedy_generation_through_the_entry_point(folders, name, dtype):
    from paged_attention_engine_b200 import LLM, Request

    raw, page, seed = gh.SMALL[name]
    llm = LLM.from_pretrained(folders[name], dtype=str(dtype).replace("torch.", ""), num_blocks=64, block_size=page,
                              max_num_seqs=3, max_num_batched_tokens=16, record_logits=True)
    prompts = list(gh.random_requests(raw, [5, 21, 12, 1, 33], seed + 20).values())
    for i, prompt in enumerate(prompts):
        assert llm.add_request(Request(f"g{i}", tuple(prompt), 7))
    out = llm.run_to_completion()
    for i, prompt in enumerate(prompts):
        tokens = list(out[f"g{i}"])
        assert len(tokens) == 7
        want = gh.plain_logits(folders[name], prompt + tokens)[len(prompt) - 1: -1]
        got = torch.stack(llm.scheduler.finished[f"g{i}"].step_logits)
        allowed = gh.row_tolerance(dtype, gh.plain_logits(folders[name], prompt + tokens[:-1]), folders[name], prompt + tokens[:-1])[-7:]
        assert bool(((got - want).abs().max(dim=1).values <= allowed).all())
        if dtype == torch.float32:
            assert tokens == _plain_greedy(folders[name], prompt, 7)


def test_preempted_requests_are_computed_again(folders):
    """A pool too small for all requests: some give everything back, state included, and start over."""
    from paged_attention_engine_b200 import LLM, Request
    from paged_attention_engine_b200.engine.scheduler import EventKind

    raw, page, seed = gh.SMALL["small_a"]
    outs = []
    for blocks in (96, 16):
        llm = LLM.from_pretrained(folders["small_a"], dtype="float32", num_blocks=blocks, block_size=page, max_num_seqs=4)
        for i, prompt in enumerate(gh.random_requests(raw, [14, 9, 17, 6], seed + 30).values()):
            assert llm.add_request(Request(f"p{i}", tuple(prompt), 20))
        outs.append(llm.run_to_completion())
    assert outs[0] == outs[1]
    assert llm.scheduler.events_of(EventKind.PREEMPT)


def test_trace_program_on_a_random_model(folders, prompts, tmp_path):
    raw, page, seed = gh.SMALL["small_a"]
    requests, oracle = prompts["small_a"]
    requests = {k: requests[k] for k in ("r1", "r2", "r4")}
    trace = helpers.trace_mixed(requests, seed, live_limit=2, decode_tail=6)
    outputs = helpers.run_trace_program(folders["small_a"], "bfloat16", trace, helpers.max_live_tokens(trace, page),
                                        tmp_path / "out", raw["vocab"], block_size=page)
    got = helpers.collect(trace, outputs, requests)
    for key in requests:
        allowed = gh.row_tolerance(torch.bfloat16, oracle[key], folders["small_a"], requests[key])
        assert bool(((got[key] - oracle[key]).abs().max(dim=1).values <= allowed).all())


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_tolerance_notices_a_fault_in_any_mechanism(folders, prompts, dtype, monkeypatch):
    """The plain model with one mechanism changed leaves the tolerance around the engine's logits:
    the comparisons above could tell."""
    raw, page, seed = gh.SMALL["small_a"]
    requests, oracle = prompts["small_a"]
    requests, oracle = {"r0": requests["r0"]}, {"r0": oracle["r0"]}
    got = _check(folders["small_a"], dtype, helpers.trace_whole(requests), requests, oracle, page)["r0"]
    config, tensors = gh.read_model(folders["small_a"])
    tol = gh.tolerance(dtype, oracle["r0"])

    def gap(changed_config=config, changed_tensors=tensors):
        return float((plain.forward(changed_config, changed_tensors, requests["r0"]).float() - got).abs().max())

    def changed(path, value):
        out = copy.deepcopy(config)
        node = out
        for key in path[:-1]:
            node = node[key]
        if value is None:
            node.pop(path[-1])
        else:
            node[path[-1]] = value
        return out

    def with_tensor(name, change):
        out = dict(tensors)
        out[name] = change(tensors[name].float()).to(tensors[name].dtype)
        return out

    left, right = ["layers", 0, "mixer", "left"], ["layers", 0, "mixer", "right"]
    faults = {
        "score scale": gap(changed(left + ["scale"], 0.2)),
        "rotation base": gap(changed(left + ["rot", "base"], 60.0)),
        "rotated channels": gap(changed(left + ["rot", "dims"], 6)),
        "no frequency scaling": gap(changed(left + ["rot", "scaling"], None)),
        "frequency factor": gap(changed(left + ["rot", "scaling", "factor"], 3.5)),
        "retention's rotation base": gap(changed(right + ["rot", "base"], 50.0)),
        "retention's rotated channels": gap(changed(right + ["rot", "dims"], 8)),
        "a head's decay": gap(changed(right + ["decay"], [0.5, 0.9, 1.0])),
        "left scale": gap(changed(["layers", 0, "mixer", "left_scale"], 1.0)),
        "right scale": gap(changed(["layers", 0, "mixer", "right_scale"], 1.0)),
        "norm groups": gap(changed(["layers", 1, "mixer", "norm_groups"], 6)),
        "key bias": gap(changed_tensors=with_tensor("l0.mix.left.k.b", torch.zeros_like)),
        "value bias": gap(changed_tensors=with_tensor("l0.mix.left.v.b", torch.zeros_like)),
        "output gate": gap(changed_tensors=with_tensor("l0.mix.left.g", torch.zeros_like)),
        "retention's gate": gap(changed_tensors=with_tensor("l0.mix.right.g", lambda t: t * 0.5)),
        "convolution bias": gap(changed_tensors=with_tensor("l1.mix.conv.b", torch.zeros_like)),
        "convolution taps reversed": gap(changed_tensors=with_tensor("l2.mix.conv", lambda t: t.flip(1))),
        "oldest tap": gap(changed_tensors=with_tensor("l2.mix.conv", lambda t: torch.cat([t[:, :1] * 0, t[:, 1:]], dim=1))),
        "step bias": gap(changed_tensors=with_tensor("l1.mix.dt_bias", lambda t: t + 0.3)),
        "rate": gap(changed_tensors=with_tensor("l1.mix.A_log", lambda t: t + 0.3)),
        "skip": gap(changed_tensors=with_tensor("l2.mix.D", torch.zeros_like)),
        "norm slope": gap(changed_tensors=with_tensor("l1.norm1.alpha", lambda t: t * 1.5)),
        "norm bias": gap(changed_tensors=with_tensor("l1.norm2.b", torch.zeros_like)),
        "the last layer again": gap(changed(["layers"], config["layers"][:-1])),
        "other weights again": gap(changed(["layers", 3], dict(config["layers"][2], weights_of=2))),
    }

    def fault(what, name, replacement):
        monkeypatch.setattr(plain, name, replacement)
        faults[what] = gap()
        monkeypatch.undo()

    plain_rotate, plain_memory, plain_unit = plain.rotate, plain.decayed_memory, plain.unit_rms
    fault("the other pairing", "rotate", lambda x, rot, neighbours, first=0: plain_rotate(x, rot, not neighbours, first))
    fault("queries one position on", "rotate", lambda x, rot, neighbours, first=0: plain_rotate(x, rot, neighbours, 1 if x.shape[1] == 4 else 0))
    fault("a read before the write", "decayed_memory", lambda q, k, v, keep, state=None: (
        torch.cat([torch.zeros_like(v[:1]), plain_memory(q.roll(-1, 0), k, v, keep)[0][:-1]]), None))
    fault("a state lost after 20 tokens", "decayed_memory", lambda q, k, v, keep, state=None: (
        torch.cat([plain_memory(q[a: a + 20], k[a: a + 20], v[a: a + 20], keep[a: a + 20])[0] for a in range(0, q.shape[0], 20)]), None))
    fault("a norm over all channels", "unit_rms", lambda x, eps: plain_unit(x.reshape(x.shape[0], -1), eps).reshape(x.shape))
    fault("silu in the feed-forward", "relu_glu", lambda h, t, name: (
        plain.silu(h @ t[f"{name}.gate"].double().T) * (h @ t[f"{name}.up"].double().T)) @ t[f"{name}.down"].double().T)
    plain_layer = plain.layer

    def one_after_the_other(x, t, name, entry, eps):
        x = plain_layer(x, t, name, dict(entry, mlp=None), eps)
        if entry.get("mlp"):
            x = x + plain.relu_glu(plain.dynamic_tanh(x, t, f"{name}.norm2"), t, f"{name}.mlp")
        return x

    fault("one sublayer after the other", "layer", one_after_the_other)

    def one_norm(x, t, name, entry, eps):
        t = dict(t)
        for end in ("", ".alpha", ".b"):
            if f"{name}.norm2{end}" in t:
                t[f"{name}.norm2{end}"] = t[f"{name}.norm1{end}"]
        return plain_layer(x, t, name, entry, eps)

    fault("one norm for both", "layer", one_norm)

    fault("the gate after the norm", "mamba2_mixer", _mamba_gate_after)
    assert gap() <= tol
    # bfloat16's tolerance is a thousand times wider: there the coarse faults must show, in float32 all of them
    coarse = ("left scale", "skip", "the last layer again", "a state lost after 20 tokens", "one norm for both", "silu in the feed-forward")
    unseen = {what: value for what, value in faults.items() if (dtype == torch.float32 or what in coarse) and not value > 1.5 * tol}
    assert not unseen, f"the plain model with these faults is within 1.5 x the tolerance {tol}: {unseen}"


def _mamba_gate_after(h, t, name, m, eps):
    T, H, dv, n, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner, silu = H * dv, plain.silu
    z, xbc, dt = (h @ t[f"{name}.in"].double().T).split([inner, inner + 2 * G * n, H], dim=1)
    x, B, C = silu(plain.short_convolution(xbc, t[f"{name}.conv"], t[f"{name}.conv.b"])).split([inner, G * n, G * n], dim=1)
    step = plain.softplus(dt + t[f"{name}.dt_bias"].double())
    y = plain.selective_memory(x.view(T, H, dv), B.view(T, G, n), C.view(T, G, n), step, torch.exp(t[f"{name}.A_log"].double()), t[f"{name}.D"].double())
    y = plain.unit_rms(y.reshape(T, m["norm_groups"], -1), eps).reshape(T, inner) * t[f"{name}.norm"].double() * silu(z)
    return y @ t[f"{name}.o"].double().T
