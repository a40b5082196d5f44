"""Each kernel behind Rigulorn's layers against the plain oracle, one mechanism at a time."""
import numpy as np
import pytest
import torch

from tests import rigulorn_oracle as oracle
from tests.test_gpu_reninex_ops import PAGE, _batch, _pages, _rel, _schedule

pytestmark = pytest.mark.gpu

DTYPES = [torch.float32, torch.bfloat16]


def _pad8(n):
    return (n + 7) // 8 * 8


def _fill_slots(b):
    """The embedding kernel writes ``b.kv_slot``."""
    from arctic_platform_b200.ops import serving
    serving.embed(b, torch.zeros(4, 8, device="cuda"), None, None, torch.zeros(8, dtype=torch.int32, device="cuda"),
                  torch.empty(b.rows, 8, device="cuda"))


# ---------------------------------------------------------------------------- streams
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("S,W", [(1, 64), (2, 256), (3, 128), (4, 2052), (4, 74), (5, 96), (16, 33), (1, 7), (2, 12288)])
def test_stream_update_input_and_norm(dtype, S, W):
    from arctic_platform_b200.ops import serving
    g = torch.Generator().manual_seed(S * W)
    rnd = lambda *s: torch.randn(*s, generator=g)
    T, eps = 9, 1e-2
    x, y = rnd(T, S, W), rnd(T, W)
    mix, out, inw, gain = (rnd(*s).to(dtype) for s in ((S, S), (S,), (S,), (W,)))
    f = lambda t: t.double()
    ref = oracle.streams_out(f(x).transpose(0, 1), f(y), f(mix), f(out))
    u = oracle.streams_in(ref, f(inw))
    h = oracle.rms(u, eps) * f(gain)
    tol = {torch.float32: 3e-6, torch.bfloat16: 0.05}[dtype]
    args = [t.cuda() for t in (mix, out, inw, gain)]
    xc, yc = x.cuda(), y.cuda()
    got = serving.stream_step(xc, yc, *args, eps, clear=True)
    assert got.dtype == dtype and _rel(got.cpu(), h) < tol
    assert _rel(xc.cpu().transpose(0, 1), ref) < 3e-6 and (yc == 0).all()
    # without an output of a sublayer, the streams stay; without a gain, the raw sum in fp32
    xc = x.cuda()
    got = serving.stream_step(xc, None, None, None, *args[2:], eps)
    assert _rel(got.cpu(), oracle.rms(oracle.streams_in(f(x).transpose(0, 1), f(inw)), eps) * f(gain)) < tol
    yc = y.cuda()
    got = serving.stream_step(xc, yc, *args[:2], None, None, eps, write=False)
    assert got.dtype == torch.float32 and _rel(got.cpu(), ref.sum(0)) < 3e-6
    assert torch.equal(xc.cpu(), x) and torch.equal(yc.cpu(), y)


@pytest.mark.parametrize("dtype", DTYPES)
def test_scaled_embedding_fills_every_stream_and_the_final_norm_has_a_gain_per_channel(dtype):
    from arctic_platform_b200.ops import serving
    g = torch.Generator().manual_seed(0)
    table, gain = torch.randn(50, 74, generator=g).to(dtype), torch.randn(74, generator=g).to(dtype)
    pages, _ = _pages([20])
    b = _batch([(0, np.arange(20) * 7 % 50, 0)], pages)
    x = torch.empty(b.rows, 3, 74, device="cuda")
    serving.embed(b, table.cuda(), None, None, torch.zeros(1, dtype=torch.int32, device="cuda"), x, scale=2.5)
    ref = table.float()[torch.arange(20) * 7 % 50] * 2.5
    assert all(torch.equal(x[:, s].cpu(), ref) for s in range(3))
    rows = torch.tensor([7, 0], dtype=torch.int32, device="cuda")
    got = serving.gain_norm_rows(x[:, 0].contiguous(), rows, gain.cuda(), 1e-3)
    tol = {torch.float32: 2e-6, torch.bfloat16: 0.03}[dtype]
    assert _rel(got.cpu(), oracle.rms(ref[[7, 0]].double(), 1e-3) * gain.double()) < tol


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("M,N,K,limit", [(1, 64, 96, 1.0), (5, 130, 74, 7.0), (130, 272, 256, 0.5), (300, 40, 50, 2.0),
                                         (700, 4096, 512, 1.5), (64, 2048, 512, 1.0)])
def test_clamped_glu(dtype, M, N, K, limit):
    from arctic_platform_b200.ops import serving
    if dtype == torch.float32 and M * N > 1e6:
        M = 70
    g = torch.Generator().manual_seed(M)
    a, w = torch.randn(M, K, generator=g).to(dtype), (torch.randn(N, K, generator=g) * 2 * K ** -0.5).to(dtype)
    ref = a.double() @ w.double().t()
    want = oracle.clamped_glu(ref[:, 0::2], ref[:, 1::2], limit)
    assert _rel(oracle.clamped_glu(ref[:, 0::2], ref[:, 1::2], limit, ("no_limit",)), want) > 0.5 or limit > 5
    out = torch.zeros(M, N // 2 + 16, device="cuda", dtype=dtype)
    serving.gate_up_clamped(a.cuda(), w.cuda(), out[:, 8:8 + N // 2], limit)
    assert _rel(out[:, 8:8 + N // 2].cpu(), want) < {torch.float32: 3e-5, torch.bfloat16: 0.03}[dtype]
    assert (out[:, :8] == 0).all() and (out[:, 8 + N // 2:] == 0).all()


@pytest.mark.parametrize("M,N,K", [(1, 256, 512), (70, 256, 96), (128, 4096, 256), (3000, 1024, 64), (4, 70, 30)])
def test_project_adds_onto_zeros_or_overwrites(M, N, K):
    from arctic_platform_b200.ops import serving
    g = torch.Generator().manual_seed(M)
    a, w = torch.randn(M, K, generator=g).bfloat16().cuda(), (torch.randn(N, K, generator=g) * K ** -0.5).bfloat16().cuda()
    y = torch.zeros(M, N, device="cuda") if serving.accumulates(M, N, a.device) else torch.full((M, N), 9.0, device="cuda")
    serving.project(a, w, y)
    assert _rel(y.cpu(), (a.double() @ w.double().t()).cpu()) < 1e-5


# ---------------------------------------------------------------------------- rotation, cache, attention
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,maps,D,E,rot", [(4, 2, 2, 32, 48, 16), (3, 1, 2, 18, 13, 6), (2, 2, 2, 64, 128, 64), (4, 4, 1, 24, 40, 12),
                                              (2, 1, 2, 9, 5, 4), (2, 2, 2, 16, 16, 0), (6, 3, 2, 24, 8, 2)])
def test_pairwise_rotation_and_cache_rows(dtype, H, G, maps, D, E, rot):
    from arctic_platform_b200.ops import norm, serving
    g = torch.Generator().manual_seed(D)
    lens, base = [40, 23], 700.0
    cols = (8, 8 + _pad8(H * maps * D), 8 + _pad8(H * maps * D) + _pad8(G * maps * D))
    ld = cols[2] + _pad8(G * E)
    P = [torch.randn(n, ld, generator=g).to(dtype) for n in lens]
    pages, pool = _pages(lens)
    rope = norm.rope_tables(64, max(2, rot), base, "cuda")
    kc = torch.full((pool, G, PAGE, maps * D), 7.0, device="cuda", dtype=dtype)
    vc = torch.full((pool, G, PAGE, E), 7.0, device="cuda", dtype=dtype)
    got = [[], []]
    for step in _schedule(lens, [3, 1, 9]):
        b = _batch([(i, np.zeros(n), a) for i, a, n in step], pages)
        _fill_slots(b)
        p = torch.cat([P[i][a:a + n] for i, a, n in step]).cuda()
        only_q = p.clone()
        serving.rope_cache(b, only_q, cols[:1], rope, rot, H * maps, D, torch.empty_like(kc), torch.empty_like(vc), write=False)
        serving.rope_cache(b, p, cols, rope, rot, H * maps, D, kc, vc)
        assert torch.equal(p, only_q)
        r = 0
        for i, a, n in step:
            got[i].append(p[r:r + n].cpu())
            r += n
    tol = {torch.float32: 1e-5, torch.bfloat16: 0.02}[dtype]
    for i, n in enumerate(lens):
        out, src = torch.cat(got[i]), P[i]
        q = oracle.rotate_pairs(src[:, 8:8 + H * maps * D].double().view(n, H * maps, D), torch.arange(n), rot, base)
        assert _rel(out[:, 8:8 + H * maps * D].reshape(n, H * maps, D), q) < tol
        assert torch.equal(out[:, cols[1]:], src[:, cols[1]:]) and torch.equal(out[:, :8], src[:, :8])
        k = oracle.rotate_pairs(src[:, cols[1]:cols[1] + G * maps * D].double().view(n, G * maps, D), torch.arange(n), rot, base)
        rows = torch.tensor([int(pages[i][t // PAGE]) for t in range(n)])
        off = torch.arange(n) % PAGE
        assert _rel(kc.cpu()[rows, :, off].reshape(n, G * maps, D), k) < tol
        assert torch.equal(vc.cpu()[rows, :, off], src[:, cols[2]:cols[2] + G * E].view(n, G, E))
    written = sum(lens) * G * maps * D
    assert int((kc == 7).sum()) >= kc.numel() - written                     # nothing outside the sequences' rows


# heads, kv heads, maps, dim, vdim, cap, chunk
HEADS = [(4, 2, 2, 32, 64, 20.0, 60), (4, 4, 2, 64, 128, 50.0, 100), (6, 2, 2, 16, 48, 8.0, 0), (3, 1, 2, 18, 13, 10.0, 37),
         (8, 1, 2, 24, 24, 90.0, 33), (4, 2, 2, 48, 88, 30.0, 129), (2, 1, 2, 40, 72, 0.0, 50), (4, 2, 1, 64, 64, 12.0, 64),
         (2, 2, 1, 128, 96, 0.0, 0), (4, 2, 2, 128, 256, 30.0, 80), (24, 1, 2, 16, 16, 20.0, 17), (6, 2, 2, 32, 48, 6.0, 48), (2, 1, 2, 300, 260, 15.0, 45),
         (4, 1, 2, 64, 64, 64.0, 1), (2, 2, 2, 32, 8, 2.0, 128)]


def _spiky(T, H, G, maps, D, chunk, seed):
    """Random q, k; every third query repeats one key of its KV head in one of its maps: the first of its chunk, the last of
    the chunk before (which must not count), at page borders, itself, far back."""
    g = torch.Generator().manual_seed(seed)
    q, k = torch.randn(T, H, maps, D, generator=g), torch.randn(T, G, maps, D, generator=g)
    for n, i in enumerate(range(2, T, 3)):
        c = i // chunk * chunk if chunk else 0
        j = [c, i, max(0, c - 1), (i // PAGE) * PAGE, max(0, (i // PAGE) * PAGE - 1), i // 5, max(0, i - 1)][n % 7]
        for h in range(H):
            m = (h + n) % maps
            q[i, h, m] = k[j, h // (H // G), m] * 1.5
    return q, k


def _run_softmax(dtype, heads, lens, cuts, seed=0, faults=()):
    from arctic_platform_b200.ops import serving
    H, G, maps, D, E, cap, chunk = heads
    g = torch.Generator().manual_seed(seed + 1)
    spec = serving.SoftmaxSpec(9.0 / D, cap, chunk, maps, 0.7, 1e-4)
    lam = torch.tensor([0.6])
    P, want = [], []
    cols = (0, _pad8(H * maps * D), _pad8(H * maps * D) + _pad8(G * maps * D))
    ld = cols[2] + _pad8(G * E) + 8
    for i, n in enumerate(lens):
        q, k = _spiky(n, H, G, maps, D, chunk, seed + i)
        p = torch.zeros(n, ld, dtype=dtype)
        p[:, :H * maps * D], p[:, cols[1]:cols[1] + G * maps * D] = q.reshape(n, -1).to(dtype), k.reshape(n, -1).to(dtype)
        p[:, cols[2]:cols[2] + G * E] = torch.randn(n, G * E, generator=g).to(dtype)
        P.append(p)
        q, k = p[:, :H * maps * D].double().view(n, H, maps, D), p[:, cols[1]:cols[1] + G * maps * D].double().view(n, G, maps, D)
        v, seen = p[:, cols[2]:cols[2] + G * E].double().view(n, G, E), oracle.chunk_visible(n, chunk, faults)
        if maps == 2:
            want.append(oracle.two_map_attention(q, k, v, 0.6, 0.3, spec.scale, cap, seen, spec.eps, faults))
        else:
            want.append(oracle.softcapped_attention(q[:, :, 0], k[:, :, 0], v, spec.scale, cap, seen, faults))
    pages, pool = _pages(lens, seed)
    kc = torch.zeros(pool, G, PAGE, maps * D, device="cuda", dtype=dtype)
    vc = torch.zeros(pool, G, PAGE, E, device="cuda", dtype=dtype)
    got, none = [[] for _ in lens], torch.zeros(4096, 1, device="cuda")
    for step in _schedule(lens, cuts):
        b = _batch([(i, np.zeros(n), a) for i, a, n in step], pages)
        _fill_slots(b)
        p = torch.cat([P[i][a:a + n] for i, a, n in step]).cuda()
        out = torch.full((b.rows, _pad8(H * E) + 16), 3.0, device="cuda", dtype=dtype)
        serving.rope_cache(b, p, cols, (none, none), 0, H * maps, D, kc, vc)
        serving.softmax_attention(b, p, H, kc, vc, spec, lam.cuda() if maps == 2 else None, out[:, 8:])
        assert (out[:, :8] == 3).all() and (out[:, 8 + H * E:] == 3).all()
        r = 0
        for i, a, n in step:
            got[i].append(out[r:r + n, 8:8 + H * E].cpu())
            r += n
    return max(_rel(torch.cat(x).view(w.shape), w) for x, w in zip(got, want))


SOFT_TOL = {torch.float32: 5e-5, torch.bfloat16: 0.15}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads", HEADS)
def test_softmax_attention_over_pages(dtype, heads):
    from arctic_platform_b200.ops import _lib
    cuts = {"whole": [1000], "portions": [2, 33, 1, 16, 7, 48], "tokens": [64, 1, 1, 1, 1, 1, 1, 1, 1, 1, 1, 1]}
    for name, c in cuts.items():
        err = _run_softmax(dtype, heads, [150, 33, 97], c, seed=3)
        assert err < SOFT_TOL[dtype], (name, err)
    _lib.check_status("softmax attention")


@pytest.mark.parametrize("heads", [(4, 2, 2, 64, 128, 40.0, 0), (2, 2, 2, 32, 96, 20.0, 700), (4, 1, 2, 16, 120, 15.0, 257), (4, 2, 1, 64, 64, 0.0, 300)])
def test_softmax_attention_long_sequences(heads):
    """Many key blocks per query tile, tile and chunk borders inside portions, single tokens over a long context."""
    for cuts in ([5000], [400, 129, 1, 255, 2]):
        err = _run_softmax(torch.bfloat16, heads, [1500, 517, 128], cuts, seed=5)
        assert err < SOFT_TOL[torch.bfloat16], (cuts, err)


@pytest.mark.parametrize("fault", ["chunk_early", "chunk_late", "no_softcap", "one_map", "no_diff_scale"])
def test_softmax_attention_inputs_show_a_mistake(fault):
    assert _run_softmax(torch.float32, (4, 2, 2, 32, 64, 4.0, 60), [150], [1000], seed=3, faults=(fault,)) > 0.4


def test_a_lone_query_over_many_keys_is_split_and_merged():
    """One sequence: its keys are spread over several CTAs; some splits see nothing of a late chunk."""
    for heads in ((2, 2, 2, 32, 64, 20.0, 1000), (2, 1, 2, 16, 32, 0.0, 0), (1, 1, 1, 64, 64, 10.0, 1030)):
        err = _run_softmax(torch.bfloat16, heads, [1100], [995] + [1] * 8 + [20, 3] + [1] * 90, seed=9)
        assert err < SOFT_TOL[torch.bfloat16], (heads, err)


# ---------------------------------------------------------------------------- state space
def _run_ssm(dtype, H, E, G, N, taps, parts, lens, schedules, tol, a_lo=-3.0, a_hi=1.5):
    from arctic_platform_b200.ops import _lib, serving
    inner, ch, eps = H * E, H * E + 2 * G * N, 1e-3
    cols = (8, 8 + _pad8(inner), 8 + _pad8(inner) + _pad8(ch))
    ld = cols[2] + _pad8(H)
    state = torch.full((len(lens), H, N, E), 7.0, device="cuda")
    hist = torch.full((len(lens), 2, taps - 1, ch), 7.0, device="cuda") if taps > 1 else None
    prev, parity = (torch.zeros(len(lens), dtype=torch.int32, device="cuda") for _ in range(2))
    for rnd, cuts in enumerate(schedules):
        g = torch.Generator().manual_seed(rnd)
        r_ = lambda *s, std=1.0: (torch.randn(*s, generator=g) * std).to(dtype)
        conv, cb, db, D, gain = r_(taps, ch, std=0.6), r_(ch, std=0.3), r_(H) - 2.0, r_(H), r_(inner)
        A = (torch.rand(H, generator=g) * (a_hi - a_lo) + a_lo).to(dtype)
        P, want, pages = [], [], _pages(lens)[0]
        for n in lens:
            p = r_(n, ld)
            P.append(p)
            z, raw = p[:, 8:8 + inner].double(), p[:, cols[1]:cols[1] + ch].double()
            dt = oracle.softplus(p[:, cols[2]:cols[2] + H].double() + db.double())
            # the activation type's values, as the products see them: a value next to a rounding border may differ by an ulp
            act = oracle.silu(oracle.causal_conv(raw, conv.double().t(), cb.double())).to(dtype).double()
            x, B, C = torch.split(act, [inner, G * N, G * N], -1)
            y = oracle.state_space(x.reshape(n, H, E), B.reshape(n, G, N), C.reshape(n, G, N), dt, A.double(), D.double())
            y = y.reshape(n, -1)
            want.append((y, oracle.gated_group_norm(y, z, gain.double(), parts, eps)))
        w = serving.SsmWeights(*(t.cuda() for t in (conv, cb, db, A, D)))
        got = [[] for _ in lens]
        for step in _schedule(lens, cuts):
            b = _batch([(i, np.zeros(n), a) for i, a, n in step], pages)
            p = torch.cat([P[i][a:a + n] for i, a, n in step]).cuda()
            y = serving.state_space(b, p, cols[1], cols[2], w, G, hist, parity, state)
            out = torch.full((b.rows, _pad8(inner) + 8), 3.0, device="cuda", dtype=dtype)
            serving.gated_group_norm(y, p[:, 8:], gain.cuda(), parts, eps, out)
            serving.commit(b, prev, parity)
            assert (out[:, inner:] == 3).all()
            r = 0
            for i, a, n in step:
                got[i].append((y[r:r + n].cpu(), out[r:r + n, :inner].cpu()))
                r += n
        for i, (y, o) in enumerate(want):
            errs = [_rel(torch.cat([x[k] for x in got[i]]), ref) for k, ref in enumerate((y, o))]
            assert errs[0] < tol[0] and errs[1] < tol[1], (rnd, i, errs)
    _lib.check_status("state space")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,E,G,N,taps,parts", [(6, 32, 3, 48, 4, 2), (3, 10, 3, 21, 2, 5), (4, 72, 2, 16, 7, 1), (2, 136, 1, 128, 1, 4),
                                                (8, 64, 2, 64, 3, 8), (1, 8, 1, 8, 5, 1), (2, 40, 2, 200, 4, 2), (5, 64, 1, 128, 4, 1)])
def test_state_space_in_portions(dtype, H, E, G, N, taps, parts):
    cuts = ([1000], [2, 1, 31, 64, 5, 33], [100, 1, 1, 1, 1, 1, 1, 1, 1, 1, 1, 1], [65, 3], [2])
    _run_ssm(dtype, H, E, G, N, taps, parts, [130, 41, 90], cuts, {torch.float32: (2e-4, 2e-4), torch.bfloat16: (0.03, 0.12)}[dtype])


@pytest.mark.parametrize("E,N", [(64, 64), (136, 128)])
def test_state_space_over_segments(E, N):
    """Long entries are cut into segments whose states are chained; slow decays make a lost segment visible."""
    _run_ssm(torch.bfloat16, 2, E, 1, N, 4, 2, [1500, 700, 333], ([5000], [900, 1, 450, 2]), (0.03, 0.12), -8.0, -5.0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("inner,parts", [(12288, 1), (8192, 8), (30, 5), (16384, 1), (96, 96)])
def test_gate_before_the_grouped_norm(dtype, inner, parts):
    from arctic_platform_b200.ops import serving
    g = torch.Generator().manual_seed(inner)
    y, z, gain = torch.randn(5, inner, generator=g), torch.randn(5, inner + 6, generator=g).to(dtype), torch.randn(inner, generator=g).to(dtype)
    out = torch.zeros(5, inner, device="cuda", dtype=dtype)
    serving.gated_group_norm(y.cuda(), z.cuda()[:, :inner], gain.cuda(), parts, 1e-2, out)
    want = oracle.gated_group_norm(y.double(), z[:, :inner].double(), gain.double(), parts, 1e-2)
    assert _rel(out.cpu(), want) < {torch.float32: 1e-5, torch.bfloat16: 0.12}[dtype]


def test_oracle_without_the_carried_state_differs():
    g = torch.Generator().manual_seed(0)
    r_ = lambda *s: torch.randn(*s, generator=g).double()
    args = (r_(60, 2, 8), r_(60, 1, 16), r_(60, 1, 16), r_(60, 2).abs() * 0.1, torch.full((2,), -3.0).double(), r_(2))
    assert _rel(oracle.state_space(*args, ("state_reset:30",)), oracle.state_space(*args)) > 0.5
