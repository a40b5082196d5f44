"""Each kernel behind Meronex's layers against the plain oracle, one mechanism at a time."""
import numpy as np
import pytest
import torch

from tests import meronex_oracle as oracle
from tests.test_gpu_reninex_ops import PAGE, _batch, _pages, _rel, _schedule
from tests.test_gpu_rigulorn_ops import _fill_slots, _pad8

pytestmark = pytest.mark.gpu

DTYPES = [torch.float32, torch.bfloat16]


def _gen(seed):
    g = torch.Generator().manual_seed(seed)
    return lambda *s, std=1.0: torch.randn(*s, generator=g) * std


# ---------------------------------------------------------------------------- residual
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W,groups,top", [(64, 1, 1), (256, 2, 3), (74, 37, 2), (33, 3, 5), (2052, 4, 6), (96, 16, 2), (12288, 8, 2), (160, 5, 1)])
def test_gated_residual_with_group_norm_and_two_sides(dtype, W, groups, top):
    from arctic_platform_b200.ops import serving
    rnd, T, eps, mult = _gen(W), 9, 1e-2, 0.37
    x, y, y2 = rnd(T, W), rnd(T, W), rnd(T, W, std=3.0)
    x[:, :W // groups] *= 5                                                    # groups of different size
    post, post2, pre, bias = ((1 + rnd(W, std=0.4)).to(dtype) for _ in range(4))
    wide = rnd(T, W + 8)
    eo = rnd(T * top, W).to(dtype)
    slots = torch.randperm(T * top, generator=torch.Generator().manual_seed(1)).view(T, top).int()
    slots[::3, 0] = -1
    f = lambda t: t.double()
    mixed = torch.where((slots >= 0)[..., None], f(eo)[slots.clamp(min=0).long()], torch.zeros((), dtype=torch.float64)).sum(1)
    mix = serving.ExpertMix(eo.cuda(), slots.cuda(), None, None, eo.cuda())
    tol = {torch.float32: 1e-5, torch.bfloat16: 0.05}[dtype]
    for sides, use_mix, gated, gate_type in ((1, 0, 1, dtype), (2, 0, 1, dtype), (0, 1, 1, torch.float32), (2, 0, 0, dtype), (1, 1, 1, torch.float32),
                                             (0, 0, 0, dtype)):
        gate = wide.to(gate_type)[:, 8:]
        s = (f(y) if sides else 0) + (mixed if use_mix else 0)
        if sides == 2:
            s = oracle.rms(f(y), eps) * f(post) + oracle.rms(f(y2), eps) * f(post2)
        ref = f(x) + mult * (oracle.sigmoid(f(gate) + f(bias)) if gated else 1.0) * s
        xc, yc, y2c = x.cuda(), y.cuda(), y2.cuda()
        args = dict(mix=mix if use_mix else None, offset=0.0, mult=mult, groups=groups, eps=eps)
        if sides == 2:
            args.update(y2=y2c, post2=post2.cuda())
        if gated:
            args.update(gate=wide.cuda().to(gate_type)[:, 8:], gate_bias=bias.cuda())
        first = yc if sides else None
        p = post.cuda() if sides == 2 else None
        look = serving.residual_step(xc, first, p, None, write=False, dtype=dtype, **args)
        assert torch.equal(xc.cpu(), x) and torch.equal(yc.cpu(), y) and _rel(look.cpu(), ref) < 5e-6
        h = serving.residual_step(xc, first, p, pre.cuda(), clear=True, **args)
        want = oracle.group_norm(ref, f(pre), groups, eps)
        assert h.dtype == dtype and _rel(h.cpu(), want) < tol and _rel(xc.cpu(), ref) < 5e-6
        assert groups == 1 or _rel(oracle.group_norm(ref, f(pre), 1, eps), want) > 0.3
        assert (yc == 0).all() if sides else torch.equal(yc.cpu(), y)
        assert (y2c == 0).all() if sides == 2 else torch.equal(y2c.cpu(), y2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W,groups", [(74, 1), (74, 2), (2048, 4), (90, 9), (512, 64)])
def test_final_norm_in_groups(dtype, W, groups):
    from arctic_platform_b200.ops import serving
    rnd = _gen(W)
    x, w = rnd(5, W), rnd(W).to(dtype)
    x[:, :W // groups] *= 7
    rows = torch.tensor([4, 0, 4], dtype=torch.int32, device="cuda")
    got = serving.gain_norm_rows(x.cuda(), rows, w.cuda(), 1e-3, groups=groups)
    assert _rel(got.cpu(), oracle.group_norm(x.double()[[4, 0, 4]], w.double(), groups, 1e-3)) < {torch.float32: 5e-6, torch.bfloat16: 0.03}[dtype]


# ---------------------------------------------------------------------------- recurrent mixers
def _rule_inputs(rule, dtype, shape, lens, seed, strong, taps):
    """Projections in one buffer with neighbours on both sides, weights, and the oracle's normed and gated output per sequence."""
    from arctic_platform_b200.ops import serving
    H, KH, D, E = shape
    rnd, eps = _gen(seed), 0.5                                   # a large eps: the scale of an output shows
    spec = serving.RecurrentSpec(rule, H, KH, D, E, eps, cap=4.0, silu=rule != "memory", shared_gain=rule == "delta")
    q, k, v = 8, 8 + KH * D, 8 + 2 * KH * D
    g = 8 + _pad8(spec.channels)
    a, b = g + _pad8(H * E), g + _pad8(H * E) + _pad8(H)
    ld = b + _pad8(H) + 8
    P = [rnd(n, ld).to(dtype) for n in lens]
    for p in P:
        p[:, a:a + H] *= 3 * strong
        p[:, b:b + H] *= 3 * strong
    gain = (1 + rnd(E if rule == "delta" else H * E, std=0.4)).to(dtype)
    Z, conv, want = [None] * len(lens), None, []
    if rule == "memory":
        w0, w1 = rnd(H, std=2.0).to(dtype), (2 + rnd(H)).to(dtype)
    elif rule == "delta":
        w0, w1, conv = (rnd(H) - 1).to(dtype), (rnd(H) - 2).to(dtype), rnd(taps, spec.channels, std=taps ** -0.5).to(dtype)
    else:
        w0, w1, Z = (rnd(H * D, std=strong) - 2).to(dtype), rnd(H * D, std=2.0).to(dtype), [rnd(n, H * D, std=strong) for n in lens]
    act = (lambda t: t.to(dtype).double()) if dtype == torch.bfloat16 else (lambda t: t)       # convolved columns are activations
    for p, z in zip(P, Z):
        d, n = p.double(), p.shape[0]
        x = d[:, q:q + spec.channels]
        if rule == "delta":
            x = act(oracle.short_conv(x, conv.double().t()))
        qq, kk, vv = x[:, :KH * D].view(n, KH, D), x[:, KH * D:2 * KH * D].view(n, KH, D), x[:, 2 * KH * D:].view(n, H, E)
        zi, zf = d[:, a:a + H], d[:, b:b + H]
        if rule == "memory":
            o = oracle.matrix_memory(qq * D ** -0.5, kk, vv, *oracle.memory_gates(zi + w0.double(), zf + w1.double(), spec.cap))
        elif rule == "delta":
            unit = lambda t: t / torch.sqrt((t * t).sum(-1, keepdim=True) + 1e-6)
            of = torch.arange(H) // (H // KH)
            dec = torch.exp(-torch.exp(w0.double()) * oracle.softplus(zi + w1.double()))
            o = oracle.delta_rule(unit(qq)[:, of] * D ** -0.5, unit(kk)[:, of], vv, oracle.sigmoid(zf), dec)
        else:
            w = torch.exp(-torch.exp(z.double() + w0.double())).view(n, H, D)
            o = oracle.channel_decay_recurrence(qq, kk, vv, w, w1.double().view(H, D))
        o = (oracle.rms(o, eps).reshape(n, H, E) * gain.double().view(-1, E)).reshape(n, H * E)
        gate = d[:, g:g + H * E]
        want.append(o * (oracle.silu(gate) if spec.silu else oracle.sigmoid(gate)))
    make = lambda p, z: serving.RecurrentInputs(p, q, k, v, g, w0.cuda(), w1.cuda(), gain.cuda(), a, b, z=z, conv=None if conv is None else conv.cuda())
    return spec, P, Z, make, want


def _run_rule(rule, dtype, shape, lens, cuts, seed=0, strong=1.0, taps=3):
    from arctic_platform_b200.ops import _lib, serving
    H, KH, D, E = shape
    spec, P, Z, make, want = _rule_inputs(rule, dtype, shape, lens, seed, strong, taps)
    n = len(lens)
    f32 = dict(device="cuda", dtype=torch.float32)
    # slots hold what other sequences left there
    state, aux = torch.full((n, H, D, E), 7.0, **f32), torch.full((n, H, D + 1), 7.0, **f32)
    hist = torch.full((n, 2, taps - 1, spec.channels), 7.0, **f32) if rule == "delta" and taps > 1 else None
    parity, prev = (torch.zeros(n, device="cuda", dtype=torch.int32) for _ in range(2))
    pages, _ = _pages(lens)
    got = [[] for _ in lens]
    for step in _schedule(lens, cuts):
        b = _batch([(i, np.zeros(c), a) for i, a, c in step], pages)
        p = torch.cat([P[i][a:a + c] for i, a, c in step]).cuda()
        z = torch.cat([Z[i][a:a + c] for i, a, c in step]).cuda() if rule == "time_mix" else None
        out = torch.full((b.rows, _pad8(H * E) + 16), 3.0, device="cuda", dtype=dtype)
        serving.recurrent(b, spec, make(p, z), state, out[:, 8:8 + H * E], aux=aux, hist=hist, parity=parity)
        assert (out[:, :8] == 3).all() and (out[:, 8 + H * E:] == 3).all()
        serving.commit(b, prev, parity)
        r = 0
        for i, a, c in step:
            got[i].append(out[r:r + c, 8:8 + H * E].cpu())
            r += c
    _lib.check_status(rule)
    return max(max(_rel(torch.cat(x), w), 15 * _rms_error(torch.cat(x), w)) for x, w in zip(got, want))


def _rms_error(got, want):
    return float(((got.double() - want).pow(2).mean() / want.pow(2).mean()).sqrt())


RULE_TOL = {torch.float32: 1e-4, torch.bfloat16: 0.2}
SHAPES = [(2, 2, 56, 80), (4, 2, 64, 64), (3, 1, 10, 13), (2, 1, 128, 128), (1, 1, 40, 72), (6, 3, 16, 8), (2, 2, 136, 24), (2, 1, 24, 200)]


def _shape(rule, s):
    H, KH, D, E = s
    return (H, KH, D, E) if rule == "delta" else (H, H, D, E)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("rule", ["memory", "delta", "time_mix"])
def test_recurrences_in_portions(rule, shape, dtype):
    for cuts in ([1000], [2, 33, 1, 16, 7, 48, 31], [64] + [1] * 11, [2], [32, 65]):
        err = _run_rule(rule, dtype, _shape(rule, shape), [100, 33, 70], cuts, seed=3)
        assert err < RULE_TOL[dtype], (cuts, err)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rule", ["memory", "delta", "time_mix"])
def test_gates_far_from_their_middle(rule, dtype):
    """Decays from none to total, gates at their caps."""
    for cuts in ([1000], [5, 1, 40]):
        err = _run_rule(rule, dtype, (2, 2, 32, 32), [120, 50], cuts, seed=5, strong=4.0)
        assert err < RULE_TOL[dtype], (cuts, err)


@pytest.mark.parametrize("rule,shape", [("memory", (1, 1, 64, 128)), ("memory", (2, 2, 24, 40)), ("time_mix", (1, 1, 64, 64)), ("time_mix", (2, 2, 128, 128)),
                                        ("delta", (4, 2, 64, 56)), ("delta", (1, 1, 128, 72))])
def test_long_entries_are_cut_into_segments(rule, shape):
    from arctic_platform_b200.ops import serving
    lens = [1500, 900]
    plan = serving.segment_plan(np.array([[0, 1500, 0, 0], [1500, 900, 1, 0]]), shape[0] * -(-shape[3] // 64), 2 * 148)
    assert rule == "delta" or len(plan["chains"]) == 2
    for cuts in ([5000], [700, 1, 400]):
        err = _run_rule(rule, torch.bfloat16, shape, lens, cuts, seed=7)
        assert err < RULE_TOL[torch.bfloat16], (cuts, err)


@pytest.mark.parametrize("taps", [1, 2, 4, 6])
@pytest.mark.parametrize("dtype", DTYPES)
def test_convolutions_of_any_length(dtype, taps):
    for shape in ((2, 1, 16, 24), (3, 3, 9, 7)):
        for cuts in ([1000], [2, 1, 1, 3, 17]):
            assert _run_rule("delta", dtype, shape, [40, 23], cuts, seed=9, taps=taps) < RULE_TOL[dtype], (shape, cuts)


@pytest.mark.parametrize("rule", ["memory", "delta", "time_mix"])
@pytest.mark.parametrize("strong", [1.0, 4.0])
def test_chunks_keep_the_states_of_the_token_by_token_kernels(monkeypatch, rule, strong):
    """The tensor-core kernels split their fp32 operands: the states they leave agree to that precision."""
    from arctic_platform_b200.ops import serving
    H, KH, D, E = shape = _shape(rule, (2, 1, 64, 80))
    lens = [600, 31, 2]
    spec, P, Z, make, _ = _rule_inputs(rule, torch.bfloat16, shape, lens, 11, strong, 4)
    pages, _ = _pages([n + 40 for n in lens])
    g = torch.Generator().manual_seed(1)
    start = [torch.randn(3, H, D, E, generator=g), torch.randn(3, H, D + 1, generator=g).abs(), torch.randn(3, 2, 3, spec.channels, generator=g)]
    p, z = torch.cat(P).cuda(), torch.cat(Z).cuda() if rule == "time_mix" else None
    left = []
    for rows in (128, 0):
        monkeypatch.setattr(serving, "MAX_MMA_STATE", rows)
        state, aux, hist = (t.cuda() for t in start)
        b = _batch([(i, np.zeros(n), 40 * (i < 2)) for i, n in enumerate(lens)], pages)
        out = torch.empty(b.rows, H * E, device="cuda", dtype=torch.bfloat16)
        serving.recurrent(b, spec, make(p, z), state, out, aux=aux, hist=hist, parity=torch.zeros(3, device="cuda", dtype=torch.int32))
        left.append((state, aux, hist))
    assert _rel(left[0][0].cpu(), left[1][0].cpu()) < 1e-3
    assert rule != "memory" or _rel(left[0][1].cpu(), left[1][1].cpu()) < 1e-4
    assert torch.equal(left[0][2], left[1][2])


# ---------------------------------------------------------------------------- inputs of time mixing
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W,cols", [(64, [24, 24, 24, 24, 16]), (74, [21, 21, 21, 21, 13]), (256, [128, 128, 128, 128, 200]), (128, [64, 64, 40])])
def test_token_shift_and_its_products(dtype, W, cols):
    from arctic_platform_b200.ops import serving
    rnd, lens, step = _gen(W), [70, 23, 41], _pad8(cols[0])
    n = len(cols)
    mu = torch.rand(n, W, generator=torch.Generator().manual_seed(2)).to(dtype)
    w = torch.zeros((n - 1) * step + (cols[-1] + 127) // 128 * 128, W, dtype=dtype)
    for s, c in enumerate(cols):
        w[s * step:s * step + c] = rnd(c, W, std=W ** -0.5).to(dtype)
    hs = [rnd(m, W).to(dtype) for m in lens]
    hist = torch.full((3, 2, 1, W), 9.0, device="cuda")
    parity, prev = (torch.zeros(3, device="cuda", dtype=torch.int32) for _ in range(2))
    pages, _ = _pages(lens)
    got = [[[] for _ in cols] for _ in lens]
    for batch in _schedule(lens, [2, 1, 33, 1, 16]):
        b = _batch([(i, np.zeros(c), a) for i, a, c in batch], pages)
        h = torch.cat([hs[i][a:a + c] for i, a, c in batch]).cuda()
        out = serving.token_shift(b, h, mu.cuda(), hist, parity, w.cuda(), step, cols)
        serving.commit(b, prev, parity)
        r = 0
        for i, a, c in batch:
            for s, m in enumerate(cols):
                got[i][s].append(out[s, r:r + c, :m].cpu())
            r += c
    act = lambda t: t.to(dtype).double()
    for i, h in enumerate(hs):
        for s, c in enumerate(cols):
            ref = act(oracle.token_shift(h.double(), mu[s].double())) @ w[s * step:s * step + c].double().t()
            assert _rel(torch.cat(got[i][s]), ref) < {torch.float32: 1e-5, torch.bfloat16: 0.03}[dtype]


def test_token_shift_of_many_rows():
    from arctic_platform_b200.ops import serving
    rnd, lens, W, cols = _gen(1), [1300, 1, 250], 128, [64, 64, 64, 64, 24]
    step, T = 64, 1551
    mu, w = torch.rand(5, W).bfloat16(), rnd(4 * step + 128, W, std=0.1).bfloat16()
    h = rnd(T, W).bfloat16()
    pages, _ = _pages(lens)
    b = _batch([(i, np.zeros(n), 0) for i, n in enumerate(lens)], pages)
    out = serving.token_shift(b, h.cuda(), mu.cuda(), torch.zeros(3, 2, 1, W, device="cuda"), torch.zeros(3, device="cuda", dtype=torch.int32),
                              w.cuda(), step, cols)
    at = 0
    for n in lens:
        for s, c in enumerate(cols):
            ref = oracle.token_shift(h[at:at + n].double(), mu[s].double()).bfloat16().double() @ w[s * step:s * step + c].double().t()
            assert _rel(out[s, at:at + n, :c].cpu(), ref) < 0.03
        at += n


@pytest.mark.parametrize("dtype", DTYPES)
def test_tanh_of_columns(dtype):
    from arctic_platform_b200.ops import serving
    x = _gen(0)(9, 40, std=2.0).to(dtype)
    y = x.cuda()
    serving.tanh_rows(y[:, 8:29])
    assert torch.equal(y[:, :8].cpu(), x[:, :8]) and torch.equal(y[:, 29:].cpu(), x[:, 29:])
    assert _rel(y[:, 8:29].cpu(), torch.tanh(x[:, 8:29].double())) < {torch.float32: 1e-6, torch.bfloat16: 0.01}[dtype]


# ---------------------------------------------------------------------------- attention
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,E,rot", [(4, 2, 32, 48, 16), (3, 1, 18, 13, 6), (2, 2, 128, 128, 128), (6, 3, 40, 24, 0), (1, 1, 8, 8, 2), (4, 4, 24, 200, 20)])
@pytest.mark.parametrize("normed", [False, True])
def test_half_rotation_value_norm_and_cache_rows(dtype, H, G, D, E, rot, normed):
    from arctic_platform_b200.ops import norm, serving
    rnd, lens, eps = _gen(D), [40, 23], 1e-2
    r = {"dims": rot, "base": 700.0, "scaling": {"factor": 3.0, "original": 32, "fast": 4.0, "slow": 1.0}}
    cols = (8, 8 + _pad8(H * D), 8 + _pad8(H * D) + _pad8(G * D))
    P = [rnd(n, cols[2] + _pad8(G * E), std=2.0).to(dtype) for n in lens]
    pages, pool = _pages(lens)
    rope = norm.rope_tables(64, max(2, rot), 700.0, "cuda", norm.Yarn(3.0, 32.0, 4.0, 1.0) if rot else None)
    kc = torch.full((pool, G, PAGE, D), 7.0, device="cuda", dtype=dtype)
    vc = torch.full((pool, G, PAGE, E), 7.0, device="cuda", dtype=dtype)
    got = [[], []]
    for step in _schedule(lens, [3, 1, 9]):
        b = _batch([(i, np.zeros(n), a) for i, a, n in step], pages)
        _fill_slots(b)
        p = torch.cat([P[i][a:a + n] for i, a, n in step]).cuda()
        serving.half_rope_cache(b, p, cols, rope, rot, H, kc, vc, eps if normed else None)
        at = 0
        for i, a, n in step:
            got[i].append(p[at:at + n].cpu())
            at += n
    tol = {torch.float32: 1e-5, torch.bfloat16: 0.03}[dtype]
    for i, n in enumerate(lens):
        out, src = torch.cat(got[i]), P[i].double()
        assert _rel(out[:, 8:8 + H * D].reshape(n, H, D), oracle.rotate(src[:, 8:8 + H * D].view(n, H, D), r)) < tol
        assert torch.equal(out[:, :8], P[i][:, :8]) and torch.equal(out[:, cols[1]:], P[i][:, cols[1]:])
        rows, off = torch.tensor([int(pages[i][t // PAGE]) for t in range(n)]), torch.arange(n) % PAGE
        assert _rel(kc.cpu()[rows, :, off], oracle.rotate(src[:, cols[1]:cols[1] + G * D].view(n, G, D), r)) < tol
        v = src[:, cols[2]:cols[2] + G * E].view(n, G, E)
        assert _rel(vc.cpu()[rows, :, off], oracle.rms(v, eps) if normed else v) < tol
    assert int((kc == 7).all(-1).sum()) >= kc[..., 0].numel() - sum(lens) * G


def _run_capped(dtype, heads, cap, lens, cuts, seed=0, hot=1.5, faults=()):
    """Every third query repeats an earlier key (page borders, itself, the first tokens, far back), which then stands out."""
    from arctic_platform_b200.ops import serving
    H, G, D, E = heads
    rnd, spec = _gen(seed + 1), serving.SoftmaxSpec(9.0 / D, cap=cap)
    ck, cv = _pad8(H * D), _pad8(H * D) + _pad8(G * D)
    P, want = [], []
    for n in lens:
        q, k = rnd(n, H, D), rnd(n, G, D)
        for m, i in enumerate(range(2, n, 3)):
            j = min(max([0, i // PAGE * PAGE, i // PAGE * PAGE - 1, i, i // 5, 1, i - 1][m % 7], 0), i)
            for h in range(H):
                q[i, h] = k[j, h // (H // G)] * hot
        p = torch.cat([torch.nn.functional.pad(t, (0, w - t.shape[1])) for t, w in ((q.reshape(n, -1), ck), (k.reshape(n, -1), cv - ck),
                                                                                   (rnd(n, G * E), _pad8(G * E)))], 1).to(dtype)
        P.append(p)
        d = p.double()
        want.append(oracle.capped_attention(d[:, :H * D].view(n, H, D), d[:, ck:ck + G * D].view(n, G, D), d[:, cv:cv + G * E].view(n, G, E),
                                            spec.scale, cap, faults))
    pages, pool = _pages(lens, seed)
    kc, vc = (torch.zeros(pool, G, PAGE, w, device="cuda", dtype=dtype) for w in (D, E))
    got = [[] for _ in lens]
    for step in _schedule(lens, cuts):
        b = _batch([(i, np.zeros(n), a) for i, a, n in step], pages)
        p = torch.cat([P[i][a:a + n] for i, a, n in step]).cuda()
        rows = torch.tensor([int(pages[i][t // PAGE]) for i, a, n in step for t in range(a, a + n)], device="cuda")
        off = torch.tensor([t % PAGE for i, a, n in step for t in range(a, a + n)], device="cuda")
        kc[rows, :, off], vc[rows, :, off] = p[:, ck:ck + G * D].view(-1, G, D), p[:, cv:cv + G * E].view(-1, G, E)
        out = torch.full((b.rows, _pad8(H * E) + 16), 3.0, device="cuda", dtype=dtype)
        serving.softmax_attention(b, p, H, kc, vc, spec, None, out[:, 8:])
        assert (out[:, :8] == 3).all() and (out[:, 8 + H * E:] == 3).all()
        r = 0
        for i, a, n in step:
            got[i].append(out[r:r + n, 8:8 + H * E].cpu())
            r += n
    return max(_rel(torch.cat(x), w) for x, w in zip(got, want))


CAP_TOL = {torch.float32: 5e-5, torch.bfloat16: 0.1}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cap", [5.0, 20.0, 60.0, 200.0])
@pytest.mark.parametrize("heads", [(4, 2, 64, 64), (6, 6, 48, 88), (3, 1, 18, 13), (2, 1, 128, 128), (4, 4, 40, 72)])
def test_capped_attention_over_pages(dtype, heads, cap):
    """Caps below, around and above the scores that stand out, references fixed and following."""
    for cuts in ([1000], [2, 33, 1, 16, 7, 48], [64] + [1] * 11):
        err = _run_capped(dtype, heads, cap, [150, 33, 97], cuts, seed=3)
        assert err < CAP_TOL[dtype], (cuts, err)


@pytest.mark.parametrize("cap,hot", [(8.0, 4.0), (50.0, 1.5), (50.0, 6.0), (300.0, 6.0)])
def test_capped_attention_over_long_sequences(cap, hot):
    """Many key blocks per tile, small scores beside scores far beyond the cap."""
    from arctic_platform_b200.ops import _lib
    for heads in ((4, 2, 64, 128), (6, 6, 48, 88), (3, 1, 128, 128)):
        for cuts in ([5000], [400, 129, 1, 255, 2]):
            err = _run_capped(torch.bfloat16, heads, cap, [1500, 517, 128], cuts, seed=5, hot=hot)
            assert err < CAP_TOL[torch.bfloat16], (heads, cuts, err)
    _lib.check_status("capped attention")


@pytest.mark.parametrize("fault", ["no_softcap", "cap_before_scale"])
def test_attention_inputs_show_a_mistake(fault):
    assert _run_capped(torch.float32, (4, 2, 64, 64), 8.0, [150], [1000], seed=3, faults=(fault,)) > 0.3


# ---------------------------------------------------------------------------- experts
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,W,E,top,ff,limit", [(9, 64, 6, 3, 48, 0.7), (1, 128, 5, 2, 64, 2.0), (200, 74, 3, 1, 22, 1.0), (300, 256, 64, 8, 64, 0.5),
                                                (64, 64, 1, 1, 32, 7.0), (2, 2048, 64, 5, 768, 1.5), (20, 64, 500, 4, 16, 1.0)])
def test_experts_that_weigh_their_input(dtype, T, W, E, top, ff, limit):
    from arctic_platform_b200.models.meronex import LayerSpec, MemorySpec, MeronexConfig, MoeSpec, _Mixture
    from arctic_platform_b200.ops import _lib, gemm, serving
    rnd = _gen(T)
    cfg = MeronexConfig(8, W, (LayerSpec(MemorySpec(1, 8, 8, 1.0), MoeSpec(E, top, ff, limit)),), 1e-5)
    mk = lambda *s: torch.nn.Parameter(torch.zeros(*s, device="cuda", dtype=dtype), requires_grad=False)
    moe = _Mixture(cfg, cfg.layers[0].mlp, mk)
    w = {}
    for e in range(E):
        for n, t in (("gate", rnd(ff, W, std=2 * W ** -0.5)), ("up", rnd(ff, W, std=2 * W ** -0.5)), ("down", rnd(W, ff, std=ff ** -0.5))):
            w[f"e{e}.{n}"] = t.to(dtype)
            moe.place(f"e{e}.{n}").copy_(w[f"e{e}.{n}"])
    h, z = rnd(T, W).to(dtype), rnd(T, E + 8, std=2.0)[:, 4:4 + E]
    W64 = {k: v.double() for k, v in w.items()}
    want = torch.zeros(T, W, dtype=torch.float64)
    s = oracle.sigmoid(z.double())
    chosen = torch.topk(s, top, dim=-1).indices
    for t in range(T):
        for e in chosen[t].tolist():
            x = (s[t, e] * h[t].double()).to(dtype).double()
            want[t] += oracle.clamped_glu(x, W64[f"e{e}.gate"], W64[f"e{e}.up"], W64[f"e{e}.down"], limit)
    live = torch.ones(T, dtype=torch.bool)
    live[3::7] = False
    pages, _ = _pages([T])
    b = _batch([(0, np.zeros(T), 0)], pages)
    b.kv_slot = torch.where(live, 1, -1).int().cuda()
    zc = rnd(T, E + 8).cuda()
    zc[:, 4:4 + E] = z.cuda()
    for _ in range(2):                                                # the counters are zero again for the second call
        mix = serving.experts(b, h.cuda(), zc[:, 4:4 + E], None, moe.counters, moe.w_gu, moe.w_down, E, E, top, ff, sigmoid=True, scale_input=True,
                              epi=gemm.EPI_CLAMP_GLU, limit=limit)
        x = torch.zeros(T, W, device="cuda")
        out = serving.residual_step(x, None, None, None, 1e-5, mix=mix, dtype=dtype, write=False).cpu()
        assert (moe.counters == 0).all() and mix.weights is None
        err = (out.double() - want)[live].abs().max() / want.pow(2).mean().sqrt()
        assert err < {torch.float32: 2e-5, torch.bfloat16: 0.06}[dtype], err
    _lib.check_status("experts")


def test_scores_that_round_to_one_keep_their_order():
    from arctic_platform_b200.ops import gemm, serving
    T, W, E, ff = 3, 64, 4, 16
    rnd = _gen(0)
    pages, _ = _pages([T])
    b = _batch([(0, np.zeros(T), 0)], pages)
    b.kv_slot = torch.ones(T, device="cuda", dtype=torch.int32)
    z = torch.tensor([[20.0, 30.0, 25.0, 40.0], [-90.0, -100.0, -95.0, -99.0], [5.0, 1.0, 50.0, 60.0]])
    h, gu, down = rnd(T, W), rnd(E * 2 * ff, W, std=W ** -0.5), rnd(E * W, ff, std=ff ** -0.5)
    mix = serving.experts(b, h.cuda(), z.cuda(), None, torch.zeros(E + 1, device="cuda", dtype=torch.int32), gu.cuda(), down.cuda(), E, E, 2, ff,
                          sigmoid=True, scale_input=True, epi=gemm.EPI_CLAMP_GLU, limit=2.0)
    got = serving.residual_step(torch.zeros(T, W, device="cuda"), None, None, None, 1e-5, mix=mix, dtype=torch.float32, write=False).cpu()
    for t, chosen in enumerate(([3, 1], [0, 2], [3, 2])):
        ref = sum(oracle.clamped_glu(oracle.sigmoid(z[t, e].double()) * h[t].double(), gu[2 * ff * e:2 * ff * (e + 1):2].double(),
                                     gu[2 * ff * e + 1:2 * ff * (e + 1):2].double(), down[W * e:W * (e + 1)].double(), 2.0) for e in chosen)
        assert float((got[t].double() - ref).abs().max()) < 1e-5, t
