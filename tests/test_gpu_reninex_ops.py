"""Each kernel of the ragged serving batch against the plain oracle, one mechanism at a time."""
import math

import numpy as np
import pytest
import torch

from tests import reninex_oracle as oracle

pytestmark = pytest.mark.gpu

DTYPES = [torch.float32, torch.bfloat16]
PAGE = 16


def _batch(work, pages_of):
    """``work``: (slot, tokens, pos0) per entry; ``pages_of[slot]``: its pages."""
    from arctic_platform_b200.ops.serving import StepBatch, StepEntry
    return StepBatch.build([StepEntry(s, np.asarray(t), p, pages_of[s]) for s, t, p in work], "cuda")


def _pages(lens, seed=0, spare=3):
    """Shuffled, interleaved pages for sequences of the given lengths; returns the table and the pool size."""
    need = [(n + PAGE - 1) // PAGE for n in lens]
    ids = np.random.default_rng(seed).permutation(sum(need) + spare).astype(np.int32)
    cut = np.cumsum([0] + need)
    return [ids[a:b] for a, b in zip(cut, cut[1:])], sum(need) + spare


def _schedule(lens, cuts):
    """Steps that advance all sequences together, sequence i in portions cycling through ``cuts`` from offset i."""
    at, k = [0] * len(lens), 0
    while any(a < n for a, n in zip(at, lens)):
        step = []
        for i, n in enumerate(lens):
            take = min(cuts[(k + i) % len(cuts)], n - at[i])
            if take:
                step.append((i, at[i], take))
                at[i] += take
        k += 1
        yield step


def _rel(got, want):
    return float((got.double() - want.double()).abs().max() / want.double().pow(2).mean().sqrt())


@pytest.mark.parametrize("dtype", DTYPES)
def test_hashed_embedding_in_portions(dtype):
    from arctic_platform_b200.ops import serving
    V, W, spec = 131, 74, (29, 1000003, 999983)
    g = torch.Generator().manual_seed(0)
    table, big = torch.randn(V, W, generator=g).to(dtype), torch.randn(spec[0] + 1, W, generator=g).to(dtype)
    lens = [23, 40]
    toks = [np.random.default_rng(i).integers(0, V, n) for i, n in enumerate(lens)]
    want = [oracle.embedding(table.float(), torch.as_tensor(t), big.float(),
                             dict(zip(("buckets", "mul_prev", "mul_cur"), spec))) for t in toks]
    pages, _ = _pages(lens)
    prev, parity = torch.full((2,), 77, dtype=torch.int32, device="cuda"), torch.zeros(2, dtype=torch.int32, device="cuda")
    for step in _schedule(lens, [1, 2, 9, 1]):
        b = _batch([(i, toks[i][a:a + n], a) for i, a, n in step], pages)
        x = torch.empty(b.rows, W, device="cuda")
        x0 = torch.zeros(b.rows, 2 * W, device="cuda", dtype=dtype)
        serving.embed(b, table.cuda(), big.cuda(), spec, prev, x, x0[:, W:])
        serving.commit(b, prev, parity)
        ref = torch.cat([want[i][a:a + n] for i, a, n in step])
        assert torch.equal(x.cpu(), ref) and torch.equal(x0[:, W:].cpu(), ref.to(dtype)) and (x0[:, :W] == 0).all()
        slots = [int(pages[i][p // PAGE]) * PAGE + p % PAGE for i, a, n in step for p in range(a, a + n)]
        assert b.kv_slot.tolist() == slots
    assert prev.tolist() == [int(t[-1]) for t in toks]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("taps,W", [(1, 64), (2, 74), (4, 256), (5, 130), (9, 64)])
def test_norm_and_input_convolutions_in_portions(dtype, taps, W):
    from arctic_platform_b200.ops import serving
    g = torch.Generator().manual_seed(taps)
    gain = torch.tensor([1.3], dtype=dtype)
    w1, w2 = (torch.randn(taps, W, generator=g).to(dtype) for _ in range(2))
    eps, lens, tol = 1e-3, [37, 30, 8], {torch.float32: 2e-6, torch.bfloat16: 0.03}[dtype]
    for reuse in range(2):                         # the second round finds the states the first one left
        xs = [torch.randn(n, W, generator=g) * (1 + i) for i, n in enumerate(lens)]
        hs = [oracle.rms(x.double(), eps) * gain.double() for x in xs]
        outs = [[h + oracle.causal_conv(h, w.double().t()) for h in hs] for w in (w1, w2)]
        if not reuse:
            state = torch.randn(3, 2, max(1, taps - 1), W).cuda() if taps > 1 else None
            prev, parity = (torch.zeros(3, dtype=torch.int32, device="cuda") for _ in range(2))
        pages, _ = _pages(lens)
        for step in _schedule(lens, [1, 2, 11, 8, 3]):
            b = _batch([(i, np.zeros(n), a) for i, a, n in step], pages)
            x = torch.cat([xs[i][a:a + n] for i, a, n in step]).cuda()
            o1, o2 = serving.norm_conv(b, x, gain.cuda(), w1.cuda(), w2.cuda(), True, state, parity, taps, eps)
            serving.commit(b, prev, parity)
            for o, ref in ((o1, outs[0]), (o2, outs[1])):
                assert _rel(o.cpu(), torch.cat([ref[i][a:a + n] for i, a, n in step])) < tol
    # without weights: the norm alone
    o1, o2 = serving.norm_conv(b, x, gain.cuda(), None, None, False, state, parity, taps, eps)
    assert o2 is None and _rel(o1.cpu(), oracle.rms(x.cpu().double(), eps) * gain.double()) < tol
    rows = torch.tensor([x.shape[0] - 1, 0], dtype=torch.int32, device="cuda")
    f = serving.gain_norm_rows(x, rows, gain.cuda(), eps)
    assert _rel(f.cpu(), oracle.rms(x[rows.long()].cpu().double(), eps) * gain.double()) < tol


@pytest.mark.parametrize("dtype", DTYPES)
def test_loop_begin(dtype):
    from arctic_platform_b200.ops import serving
    x, init = torch.randn(9, 70, device="cuda"), torch.randn(70, device="cuda").to(dtype)
    out, ref = torch.zeros(9, 140, device="cuda", dtype=dtype), x.to(dtype).clone()
    serving.loop_begin(x, init, out)
    assert torch.equal(out[:, :70], ref) and (out[:, 70:] == 0).all() and torch.equal(x, init.float().expand(9, 70))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("M,N,K", [(1, 64, 96), (5, 131, 74), (130, 264, 256), (300, 40, 50), (33, 256, 1024)])
def test_products(dtype, M, N, K):
    from arctic_platform_b200.ops import serving
    g = torch.Generator().manual_seed(M)
    a, w = torch.randn(M, K, generator=g).to(dtype), (torch.randn(N, K, generator=g) * K ** -0.5).to(dtype)
    ref = a.double() @ w.double().t()
    tol = {torch.float32: 1e-5, torch.bfloat16: 0.03}[dtype]
    ac, wc = a.cuda(), w.cuda()
    assert _rel(serving.linear(ac, wc).cpu(), ref) < tol
    assert _rel(serving.linear(ac, wc, out_dtype=torch.float32).cpu(), ref) < 1e-5
    x = torch.randn(M, N, generator=g)
    xc = x.cuda()
    serving.linear(ac, wc, xc, accumulate=True)
    assert _rel(xc.cpu(), ref + x.double()) < 1e-5
    wide = torch.zeros(M, N // 2 + 16, device="cuda", dtype=dtype)
    serving.gate_up_gelu(ac, wc[:N // 2 * 2], wide[:, 8:8 + N // 2])
    want = oracle.gelu_tanh(ref[:, 0:N // 2 * 2:2]) * ref[:, 1::2][:, :N // 2]
    assert _rel(wide[:, 8:8 + N // 2].cpu(), want) < 4 * tol
    assert (wide[:, :8] == 0).all() and (wide[:, 8 + N // 2:] == 0).all()


# ---------------------------------------------------------------------------- sigmoid attention
HEADS = [(4, 2, 64, 32), (9, 3, 96, 88), (3, 1, 20, 12), (8, 1, 128, 128), (2, 2, 72, 136), (5, 5, 16, 16),
         (4, 4, 192, 160), (16, 2, 128, 64), (24, 1, 32, 32), (2, 1, 300, 260)]


def _spiky(T, H, G, D, seed):
    """Unit-scale random q, k in which some queries repeat a key's direction: far back, at page borders, the first key,
    themselves.  Values are large on the repeated keys only, so a lost key shows."""
    g = torch.Generator().manual_seed(seed)
    q, k = torch.randn(T, H, D, generator=g), torch.randn(T, G, D, generator=g)
    hits = []
    for n, i in enumerate(range(2, T, 3)):
        j = [0, i, max(0, i - 1), (i // PAGE) * PAGE, max(0, (i // PAGE) * PAGE - 1), i // 5][n % 6]
        k[j] = torch.randn(G, D, generator=g) if j not in hits else k[j]
        hits.append(j)
        for h in range(H):
            q[i, h] = k[j, h // (H // G)] * 1.5
    return q, k


def _run_sigmoid(dtype, heads, lens, cuts, seed=0, out_scale=0.8):
    from arctic_platform_b200.ops import serving
    H, G, D, E = heads
    g = torch.Generator().manual_seed(seed + 1)
    bias = (torch.randn(H, generator=g) * 0.3 - 6.0).to(dtype)
    scale, eps = 13.0 / D, 1e-5
    pad8 = lambda n: (n + 7) // 8 * 8
    cols = (0, pad8(H * D), pad8(H * D) + pad8(G * D))
    ld = cols[2] + pad8(G * E) + 8
    P, want = [], []
    for i, n in enumerate(lens):
        q, k = _spiky(n, H, G, D, seed + i)
        v = torch.randn(n, G, E, generator=g)
        p = torch.zeros(n, ld, dtype=dtype)
        p[:, :H * D], p[:, cols[1]:cols[1] + G * D] = q.reshape(n, -1).to(dtype), k.reshape(n, -1).to(dtype)
        p[:, cols[2]:cols[2] + G * E] = v.reshape(n, -1).to(dtype)
        P.append(p)
        qn = oracle.rms(p[:, :H * D].double().view(n, H, D), eps)
        kn = oracle.rms(p[:, cols[1]:cols[1] + G * D].double().view(n, G, D), eps)
        vv = p[:, cols[2]:cols[2] + G * E].double().view(n, G, E)
        want.append(oracle.sigmoid_attention(qn, kn, vv, bias.double(), scale) * out_scale)
    pages, pool = _pages(lens, seed)
    kc = torch.zeros(pool, G, PAGE, D, device="cuda", dtype=dtype)
    vc = torch.zeros(pool, G, PAGE, E, device="cuda", dtype=dtype)
    prev = torch.zeros(len(lens), dtype=torch.int32, device="cuda")
    table = torch.zeros(4, 8, device="cuda", dtype=dtype)
    got = [[] for _ in lens]
    for step in _schedule(lens, cuts):
        b = _batch([(i, np.zeros(n), a) for i, a, n in step], pages)
        serving.embed(b, table, None, None, prev, torch.empty(b.rows, 8, device="cuda"))        # fills b.kv_slot
        p = torch.cat([P[i][a:a + n] for i, a, n in step]).cuda()
        out = torch.full((b.rows, pad8(H * E) + 16), 3.0, device="cuda", dtype=dtype)
        serving.qk_norm_cache(b, p, cols, kc, vc, H, eps)
        serving.sigmoid_attention(b, p, H, kc, vc, bias.cuda(), scale, out[:, 8:], out_scale)
        assert (out[:, :8] == 3).all() and (out[:, 8 + H * E:] == 3).all()
        r = 0
        for i, a, n in step:
            got[i].append(out[r:r + n, 8:8 + H * E].cpu())
            r += n
    return max(_rel(torch.cat(x).view(w.shape), w) for x, w in zip(got, want))


SIG_TOL = {torch.float32: 3e-5, torch.bfloat16: 0.12}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads", HEADS)
def test_sigmoid_attention_over_pages(dtype, heads):
    from arctic_platform_b200.ops import _lib
    cuts = {"whole": [1000], "portions": [2, 33, 1, 16, 7, 48], "tokens": [64, 1, 1, 1, 1, 1, 1, 1, 1, 1, 1, 1]}
    for name, c in cuts.items():
        err = _run_sigmoid(dtype, heads, [150, 33, 97], c, seed=3)
        assert err < SIG_TOL[dtype], (name, err)
    _lib.check_status("sigmoid attention")


@pytest.mark.parametrize("heads", [(4, 2, 128, 128), (4, 2, 96, 112), (2, 1, 64, 120)])
def test_sigmoid_attention_long_sequences(heads):
    """Many key blocks per query tile, tile borders inside portions, single tokens over a long context."""
    for cuts in ([5000], [400, 129, 1, 255, 2]):
        err = _run_sigmoid(torch.bfloat16, heads, [900, 517, 128], cuts, seed=5)
        assert err < SIG_TOL[torch.bfloat16], (cuts, err)


def test_sigmoid_attention_inputs_show_a_lost_key():
    """The oracle without the far keys differs by far more than the tolerance on the inputs used above."""
    q, k = _spiky(150, 4, 2, 64, 3)
    v = torch.randn(150, 2, 32, generator=torch.Generator().manual_seed(0)).double()
    q, k = oracle.rms(q.double(), 1e-5), oracle.rms(k.double(), 1e-5)
    bias = torch.full((4,), -6.0).double()
    good = oracle.sigmoid_attention(q, k, v, bias, 13.0 / 64)
    assert _rel(oracle.sigmoid_attention(q, k, v, bias, 13.0 / 64, ("window:100",)), good) > 1.0


# ---------------------------------------------------------------------------- retention
def _run_retention(dtype, H, D, E, rot, base, decay, lens, schedules, tol):
    from arctic_platform_b200.ops import _lib, norm, serving
    l2 = torch.tensor([math.log2(x) if x else float("-inf") for x in decay], device="cuda")
    eps, ks, out_scale = 1e-5, D ** -0.5, 0.6
    rope = norm.rope_tables(max(lens), max(2, rot), base, "cuda")
    pad8 = lambda n: (n + 7) // 8 * 8
    cols, o = [], 8
    for n in (H * D, H * D, H * E, H * E):
        cols.append(o)
        o += pad8(n)
    state = torch.full((len(lens), H, D, E), 7.0, device="cuda")
    for rnd, cuts in enumerate(schedules):
        g = torch.Generator().manual_seed(rnd)
        P, want, pages = [], [], _pages(lens)[0]
        for n in lens:
            p = torch.randn(n, o, generator=g).to(dtype)
            P.append(p)
            q, k = (p[:, c:c + H * D].double().view(n, H, D) for c in cols[:2])
            v, gate = (p[:, c:c + H * E].double().view(n, H, E) for c in cols[2:])
            pos = torch.arange(n)
            r = oracle.retention(oracle.rotate(q, pos, rot, base), oracle.rotate(k, pos, rot, base) * ks, v, decay)
            want.append((oracle.rms(r, eps) * oracle.silu(gate) * out_scale).reshape(n, -1))
        got = [[] for _ in lens]
        for step in _schedule(lens, cuts):
            b = _batch([(i, np.zeros(n), a) for i, a, n in step], pages)
            p = torch.cat([P[i][a:a + n] for i, a, n in step]).cuda()
            out = torch.full((b.rows, pad8(H * E) + 8), 3.0, device="cuda", dtype=dtype)
            serving.retention(b, p, tuple(cols), rope, rot, l2, state, out, eps, ks, out_scale)
            assert (out[:, H * E:] == 3).all()
            r = 0
            for i, a, n in step:
                got[i].append(out[r:r + n, :H * E].cpu())
                r += n
        for i, w in enumerate(want):
            assert _rel(torch.cat(got[i]), w) < tol, (rnd, i, _rel(torch.cat(got[i]), w))
    _lib.check_status("retention")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,D,E,rot,base", [(4, 32, 72, 24, 2e5), (3, 22, 10, 6, 100.0), (2, 128, 128, 64, 1e4),
                                            (1, 64, 200, 0, 1e4), (2, 48, 256, 48, 500.0), (2, 192, 96, 128, 1e4),
                                            (2, 40, 24, 8, 50.0), (1, 8, 8, 2, 10.0)])
def test_retention_in_portions(dtype, H, D, E, rot, base):
    decay = [1.0, 0.97, 0.5, 0.0][:H] if H > 1 else [0.995]
    cuts = ([1000], [2, 1, 31, 64, 5, 33], [100, 1, 1, 1, 1, 1, 1, 1, 1, 1, 1, 1], [65, 3])
    _run_retention(dtype, H, D, E, rot, base, decay, [200, 41, 90], cuts, {torch.float32: 2e-4, torch.bfloat16: 0.06}[dtype])


@pytest.mark.parametrize("D,E", [(64, 64), (128, 192)])
def test_retention_over_segments(D, E):
    """Long entries are cut into segments whose states are chained; slow decays make a lost segment visible."""
    _run_retention(torch.bfloat16, 2, D, E, D, 1e4, [0.9995, 0.97], [1500, 700, 333], ([5000], [900, 1, 450, 2]), 0.06)
