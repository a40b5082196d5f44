"""Each kernel behind Titatar's layers against the plain oracle, one mechanism at a time."""
import numpy as np
import pytest
import torch

from tests import titatar_oracle as oracle
from tests.test_gpu_reninex_ops import PAGE, _batch, _pages, _rel, _schedule
from tests.test_gpu_rigulorn_ops import _fill_slots, _pad8

pytestmark = pytest.mark.gpu

DTYPES = [torch.float32, torch.bfloat16]


def _gen(seed):
    g = torch.Generator().manual_seed(seed)
    return lambda *s, std=1.0: torch.randn(*s, generator=g) * std


# ---------------------------------------------------------------------------- residual
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W,top", [(64, 1), (256, 3), (74, 2), (33, 5), (2052, 6), (12288, 2), (7, 8)])
def test_residual_update_with_norms_on_both_sides(dtype, W, top):
    from arctic_platform_b200.ops import serving
    rnd, T, eps = _gen(W), 9, 1e-2
    x, y, hin = rnd(T, W), rnd(T, W), rnd(T, W).to(dtype)
    post, pre = rnd(W, std=0.4).to(dtype), rnd(W, std=0.4).to(dtype)
    table, tok = rnd(11, W).to(dtype), torch.arange(T, dtype=torch.int32) * 5 % 11
    eo = rnd(T * top, W).to(dtype)
    slots = torch.randperm(T * top, generator=torch.Generator().manual_seed(1)).view(T, top).int()
    slots[::3, 0] = -1
    wts, ident = rnd(T, top), rnd(T)
    ident[2::3] = 0
    f = lambda t: t.double()
    chosen = torch.where((slots >= 0)[..., None], f(eo)[slots.clamp(min=0).long()], torch.zeros((), dtype=torch.float64))
    mixed = (f(wts)[..., None] * chosen).sum(1) + f(ident)[:, None] * f(hin)
    mix = serving.ExpertMix(eo.cuda(), slots.cuda(), wts.cuda(), ident.cuda(), hin.cuda())
    again = (tok.cuda(), table.cuda(), 1.75)
    tol = {torch.float32: 5e-6, torch.bfloat16: 0.05}[dtype]
    norm = lambda t, w: oracle.layer_norm(t, f(w), eps)
    for use_y, use_mix, use_again, use_post in ((1, 0, 0, 1), (0, 1, 0, 1), (1, 1, 1, 1), (0, 0, 1, 1), (1, 0, 0, 0), (0, 0, 0, 1)):
        s = (f(y) if use_y else 0) + (mixed if use_mix else 0)
        ref = f(x)
        if use_y or use_mix:
            ref = ref + (norm(s, post) if use_post else s)
        if use_again:
            ref = ref + f(table)[tok.long()] * 1.75
        args = dict(mix=mix if use_mix else None, again=again if use_again else None)
        xc, yc = x.cuda(), y.cuda()
        p = post.cuda() if use_post else None
        look = serving.residual_step(xc, yc if use_y else None, p, None, eps, write=False, dtype=dtype, **args)
        assert look.dtype == torch.float32 and torch.equal(xc.cpu(), x) and torch.equal(yc.cpu(), y)
        assert _rel(look.cpu(), ref) < 5e-6
        h = serving.residual_step(xc, yc if use_y else None, p, pre.cuda(), eps, clear=True, **args)
        assert h.dtype == dtype and _rel(h.cpu(), norm(ref, pre)) < tol and _rel(xc.cpu(), ref) < 5e-6
        assert (yc == 0).all() if use_y else torch.equal(yc.cpu(), y)


@pytest.mark.parametrize("dtype", DTYPES)
def test_final_norm_with_an_offset(dtype):
    from arctic_platform_b200.ops import serving
    rnd = _gen(0)
    x, w = rnd(5, 74), rnd(74).to(dtype)
    rows = torch.tensor([4, 0, 4], dtype=torch.int32, device="cuda")
    got = serving.gain_norm_rows(x.cuda(), rows, w.cuda(), 1e-3, 1.0)
    assert _rel(got.cpu(), oracle.layer_norm(x.double()[[4, 0, 4]], w.double(), 1e-3)) < {torch.float32: 2e-6, torch.bfloat16: 0.03}[dtype]


# ---------------------------------------------------------------------------- grouped attention
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,E,rot", [(4, 2, 32, 48, 16), (3, 1, 18, 13, 6), (2, 2, 128, 128, 128), (6, 3, 40, 24, 0), (1, 1, 8, 8, 2),
                                         (16, 4, 64, 80, 32), (4, 4, 24, 16, 24)])
def test_projection_norm_rotation_and_cache_rows(dtype, H, G, D, E, rot):
    from arctic_platform_b200.ops import norm, serving
    rnd, lens, base, eps = _gen(D), [40, 23], 700.0, 1e-2
    cols = (8, 8 + _pad8(H * D), 8 + _pad8(H * D) + _pad8(G * D))
    ld = cols[2] + _pad8(G * E)
    P = [rnd(n, ld, std=2.0).to(dtype) for n in lens]
    wq, wk = (1 + rnd(H * D, std=0.3)).to(dtype), (1 + rnd(G * D, std=0.3)).to(dtype)
    pages, pool = _pages(lens)
    rope = norm.rope_tables(64, max(2, rot), base, "cuda")
    kc = torch.full((pool, G, PAGE, D), 7.0, device="cuda", dtype=dtype)
    vc = torch.full((pool, G, PAGE, E), 7.0, device="cuda", dtype=dtype)
    got = [[], []]
    for step in _schedule(lens, [3, 1, 9]):
        b = _batch([(i, np.zeros(n), a) for i, a, n in step], pages)
        _fill_slots(b)
        p = torch.cat([P[i][a:a + n] for i, a, n in step]).cuda()
        serving.row_norm_rope_cache(b, p, cols, wq.cuda(), wk.cuda(), rope, rot, H, kc, vc, eps)
        r = 0
        for i, a, n in step:
            got[i].append(p[r:r + n].cpu())
            r += n
    tol = {torch.float32: 1e-5, torch.bfloat16: 0.03}[dtype]
    r = {"dims": rot, "base": base}
    for i, n in enumerate(lens):
        out, src = torch.cat(got[i]), P[i].double()
        nq = oracle.rms(src[:, 8:8 + H * D], eps) * wq.double()
        nk = oracle.rms(src[:, cols[1]:cols[1] + G * D], eps) * wk.double()
        pos = torch.arange(n)
        assert _rel(out[:, 8:8 + H * D].reshape(n, H, D), oracle.rotate(nq.view(n, H, D), pos, r, False)) < tol
        assert torch.equal(out[:, :8], P[i][:, :8])
        rows, off = torch.tensor([int(pages[i][t // PAGE]) for t in range(n)]), pos % PAGE
        assert _rel(kc.cpu()[rows, :, off].reshape(n, G, D), oracle.rotate(nk.view(n, G, D), pos, r, False)) < tol
        assert torch.equal(vc.cpu()[rows, :, off], P[i][:, cols[2]:cols[2] + G * E].view(n, G, E))
    assert int((kc == 7).all(-1).sum()) >= kc[..., 0].numel() - sum(lens) * G


def _targets(T, window, spots=(0,)):
    """For every third query the key it repeats: the first of its window, the last one outside of it (which must not count),
    itself, around page borders, far back, given positions."""
    out = []
    for n, i in enumerate(range(2, T, 3)):
        w = window or T
        j = [i - w + 1, i - w, i, i // PAGE * PAGE, i // PAGE * PAGE - 1, i // 5, i - 1, spots[n % len(spots)]][n % 8]
        out.append((i, min(max(j, 0), i)))
    return out


# heads, kv heads, dim, value dim (negative: the values are the first columns of the key row), window, sink, gate (0, 1 per head, 2 per column)
HEADS = [(4, 2, 64, 64, 37, 1, 1), (4, 4, 128, 128, 100, 1, 1), (6, 2, 32, 48, 1, 0, 2), (3, 1, 18, 13, 20, 1, 1), (8, 1, 24, 24, 0, 1, 2),
         (4, 2, 48, 88, 129, 0, 0), (2, 1, 40, 72, 50, 1, 2), (2, 2, 128, 96, 16, 1, 1), (4, 2, 256, 256, 33, 1, 1), (24, 1, 16, 16, 17, 1, 1),
         (2, 1, 300, 260, 45, 1, 1), (4, 1, 80, -64, 0, 1, 0), (3, 1, 30, -21, 25, 1, 2), (8, 1, 96, -96, 0, 0, 1), (5, 1, 600, -512, 0, 1, 0),
         (16, 1, 320, -256, 0, 1, 0), (32, 1, 576, -512, 0, 1, 0), (20, 1, 144, -80, 0, 1, 0)]


def _run_softmax(dtype, heads, lens, cuts, seed=0, faults=()):
    from arctic_platform_b200.ops import serving
    H, G, D, E, window, with_sink, gate = heads
    own, E = E > 0, abs(E)
    rnd = _gen(seed + 1)
    spec = serving.SoftmaxSpec(9.0 / D, window=window)
    sink = rnd(H, std=2.0) + 4.0 if with_sink else None
    cq, ck, cv = 0, _pad8(H * D), _pad8(H * D) + _pad8(G * D)
    cg = cv + (_pad8(G * E) if own else 0)
    cols = {0: 0, 1: H, 2: H * E}[gate]
    ld = cg + _pad8(cols) + 8
    P, want, keys = [], [], []
    for i, n in enumerate(lens):
        q, k = rnd(n, H, D), rnd(n, G, D)
        for a, j in _targets(n, window):
            for h in range(H):
                q[a, h] = k[j, h // (H // G)] * 1.5
        p = rnd(n, ld).to(dtype)
        p[:, :H * D], p[:, ck:ck + G * D] = q.reshape(n, -1).to(dtype), k.reshape(n, -1).to(dtype)
        P.append(p)
        d = p.double()
        q, k = d[:, :H * D].view(n, H, D), d[:, ck:ck + G * D].view(n, G, D)
        v = d[:, cv:cv + G * E].view(n, G, E) if own else k[..., :E]
        seen, out = oracle.visible(n, window, faults), []
        for h in range(H):
            s = None if sink is None or "no_sink" in faults else sink[h].double() * (spec.scale if "sink_scaled" in faults else 1.0)
            o = oracle.sink_softmax(q[:, h] @ k[:, h // (H // G)].t() * spec.scale, seen, s) @ v[:, h // (H // G)]
            if gate and "no_gate" not in faults:
                o = o * oracle.sigmoid(d[:, cg + h:cg + h + 1] if gate == 1 else d[:, cg + h * E:cg + (h + 1) * E])
            out.append(o)
        want.append(torch.cat(out, -1))
    pages, pool = _pages(lens, seed)
    kc = torch.zeros(pool, G, PAGE, D if own else serving.shared_row(D, E, dtype), device="cuda", dtype=dtype)
    vc = torch.zeros(pool, G, PAGE, E, device="cuda", dtype=dtype)
    got = [[] for _ in lens]
    for step in _schedule(lens, cuts):
        b = _batch([(i, np.zeros(n), a) for i, a, n in step], pages)
        p = torch.cat([P[i][a:a + n] for i, a, n in step]).cuda()
        rows = torch.tensor([int(pages[i][t // PAGE]) for i, a, n in step for t in range(a, a + n)], device="cuda")
        off = torch.tensor([t % PAGE for i, a, n in step for t in range(a, a + n)], device="cuda")
        kc[rows, :, off, :D] = p[:, ck:ck + G * D].view(-1, G, D)
        if own:
            vc[rows, :, off] = p[:, cv:cv + G * E].view(-1, G, E)
        out = torch.full((b.rows, _pad8(H * E) + 16), 3.0, device="cuda", dtype=dtype)
        serving.softmax_attention(b, p, H, kc, vc if own else None, spec, None, out[:, 8:], dim=D, vdim=E,
                                  sink=None if sink is None else sink.cuda(), gate=p[:, cg:] if gate else None, gate_cols=1 if gate == 1 else E)
        assert (out[:, :8] == 3).all() and (out[:, 8 + H * E:] == 3).all()
        r = 0
        for i, a, n in step:
            got[i].append(out[r:r + n, 8:8 + H * E].cpu())
            r += n
    return max(_rel(torch.cat(x), w) for x, w in zip(got, want))


SOFT_TOL = {torch.float32: 5e-5, torch.bfloat16: 0.1}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads", HEADS)
def test_windows_sinks_and_gates_over_pages(dtype, heads):
    from arctic_platform_b200.ops import _lib
    cuts = {"whole": [1000], "portions": [2, 33, 1, 16, 7, 48], "tokens": [64, 1, 1, 1, 1, 1, 1, 1, 1, 1, 1, 1]}
    for name, c in cuts.items():
        err = _run_softmax(dtype, heads, [150, 33, 97], c, seed=3)
        assert err < SOFT_TOL[dtype], (name, err)
    _lib.check_status("softmax attention")


@pytest.mark.parametrize("heads", [(4, 2, 64, 128, 0, 1, 1), (2, 2, 128, 128, 700, 1, 1), (4, 1, 64, 96, 129, 1, 2), (8, 2, 128, 80, 257, 1, 1),
                                   (2, 1, 192, 128, 128, 0, 0), (3, 1, 96, 64, 1000, 1, 1), (16, 1, 576, -512, 0, 1, 0)])
def test_attention_over_long_sequences(heads):
    """Many key blocks per query tile, tile and window borders inside portions, single tokens over a long context."""
    for cuts in ([5000], [400, 129, 1, 255, 2]):
        err = _run_softmax(torch.bfloat16, heads, [1500, 517, 128], cuts, seed=5)
        assert err < SOFT_TOL[torch.bfloat16], (cuts, err)


@pytest.mark.parametrize("fault", ["window_early", "window_late", "no_window", "no_sink", "sink_scaled", "no_gate"])
def test_attention_inputs_show_a_mistake(fault):
    assert _run_softmax(torch.float32, (4, 2, 64, 64, 37, 1, 1), [150], [1000], seed=3, faults=(fault,)) > 0.4


@pytest.mark.parametrize("heads", [(2, 2, 64, 64, 1000, 1, 1), (2, 1, 32, 32, 0, 1, 0), (1, 1, 64, 64, 1030, 1, 1), (8, 1, 160, -128, 0, 1, 0),
                                   (4, 1, 288, -256, 0, 1, 1)])
def test_a_lone_query_over_many_keys_is_split_and_merged(heads):
    """One sequence: its keys are spread over several CTAs; some splits see nothing of a late window; a sink counts once."""
    err = _run_softmax(torch.bfloat16, heads, [1100], [995] + [1] * 8 + [20, 3] + [1] * 90, seed=9)
    assert err < SOFT_TOL[torch.bfloat16], err


# ---------------------------------------------------------------------------- latent attention
# heads, dim, rot, vdim, q rank, kv rank
LATENT = [(4, 32, 16, 40, 72, 48), (3, 14, 6, 11, 29, 21), (8, 128, 64, 128, 192, 256), (1, 24, 8, 32, 40, 64), (2, 64, 64, 64, 96, 512),
          (16, 128, 64, 128, 256, 512), (5, 48, 32, 96, 64, 72), (12, 64, 16, 64, 64, 64)]


def _run_latent(dtype, shape, lens, cuts, seed=0, faults=()):
    """Everything between the first projections and the output projection, on the framework's fused layouts."""
    from arctic_platform_b200.models.titatar import RotSpec, LatentAttnSpec, TitatarConfig, LayerSpec, _LatentMixer
    from arctic_platform_b200.ops import norm, serving
    H, D, R, E, Q, C = shape
    rnd, eps, W = _gen(seed), 1e-3, Q + C + R + H * E + 8
    rot = {"base": 2000.0, "dims": R, "scaling": {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0}}
    m = {"heads": H, "dim": D, "rot_dim": R, "vdim": E, "q_rank": Q, "kv_rank": C, "scale": 9.0 / D, "rot": rot}
    yarn = norm.Yarn(4.0, 64.0, 8.0, 1.0)
    spec = LatentAttnSpec(H, D, R, E, Q, C, 9.0 / D, RotSpec(R, 2000.0, yarn))
    cfg = TitatarConfig(8, W, (LayerSpec(spec),), eps)
    mk = lambda *s: torch.nn.Parameter(torch.zeros(*s, device="cuda", dtype=dtype), requires_grad=False)
    mixer = _LatentMixer(cfg, spec, mk)
    r = min(Q, C)
    uk, uq = rnd(H, D, C, std=0.3 * C ** -0.5), rnd(H, D + R, Q, std=Q ** -0.5)
    uk[..., :r] = rnd(H, D, r, std=r ** -0.5)
    uq[:, :D] = 0
    uq[:, :D, :r] = uk[..., :r]
    eye = torch.eye(W)
    w = {"dq": eye[:Q], "dkv": eye[Q:Q + C + R], "g": eye[Q + C + R:Q + C + R + H * E], "dq.norm": 1 + rnd(Q, std=0.2),
         "dkv.norm": 1 + rnd(C, std=0.2), "uq": uq.reshape(-1, Q), "uk": uk.reshape(-1, C), "uv": rnd(H * E, C, std=C ** -0.5),
         "sink": rnd(H, std=1.0) + 3.0, "o": torch.zeros(W, H * E)}
    for n, t in w.items():
        w[n] = t.to(dtype)
        mixer.place(n).copy_(w[n])
        mixer.refresh(n)
    hs, want = [], []
    for i, n in enumerate(lens):
        h = rnd(n, W)
        for a, j in _targets(n, 0, (0, 1)):                     # the query latent repeats an earlier key latent
            h[a, :r] = h[j, Q:Q + r] * 1.3
        h = h.to(dtype)
        hs.append(h)
        W64 = {k: v.double() for k, v in w.items()}
        W64["o"] = torch.eye(H * E, dtype=torch.float64)
        want.append(oracle.latent_attention_mixer(m, W64, "", h.double(), eps, faults))
    pages, pool = _pages(lens, seed)
    rope = norm.rope_tables(max(lens), R, 2000.0, "cuda", yarn)
    cache = torch.zeros(pool, 1, PAGE, serving.shared_row(C + R, C, dtype), device="cuda", dtype=dtype)
    got = [[] for _ in lens]
    c = mixer.in_cols
    for step in _schedule(lens, cuts):
        b = _batch([(i, np.zeros(n), a) for i, a, n in step], pages)
        _fill_slots(b)
        h = torch.cat([hs[i][a:a + n] for i, a, n in step]).cuda()
        p = torch.zeros(b.rows, mixer.w_in.shape[0], device="cuda", dtype=dtype)
        at = 0
        for n in ("dq", "dkv", "g"):
            o, k = c[n]
            p[:, o:o + k] = h[:, at:at + k]
            at += k
        serving.latent_norm_cache(b, p, c["dq"][0], c["dkv"][0], mixer.q_norm, mixer.kv_norm, rope, cache, eps, R)
        q = serving.linear(p[:, c["dq"][0]:c["dq"][0] + Q], mixer.w_q[:, :Q])
        out = torch.full((b.rows, _pad8(H * E) + 16), 3.0, device="cuda", dtype=dtype)
        serving.latent_attention(b, q, mixer.spec, cache, mixer.w_absorb, mixer.w_expand, mixer.sink32, p[:, c["g"][0]:], rope, out[:, 8:])
        assert (out[:, :8] == 3).all() and (out[:, 8 + H * E:] == 3).all()
        at = 0
        for i, a, n in step:
            got[i].append(out[at:at + n, 8:8 + H * E].cpu())
            at += n
    return max(_rel(torch.cat(x), w) for x, w in zip(got, want))


LATENT_TOL = {torch.float32: 5e-5, torch.bfloat16: 0.15}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", LATENT)
def test_latent_attention_over_pages(dtype, shape):
    from arctic_platform_b200.ops import _lib
    for c in ([1000], [2, 33, 1, 16, 7, 48], [64] + [1] * 11):
        err = _run_latent(dtype, shape, [150, 33, 97], c, seed=3)
        assert err < LATENT_TOL[dtype], (c, err)
    _lib.check_status("latent attention")


@pytest.mark.parametrize("shape", [(4, 32, 16, 40, 72, 48), (6, 128, 64, 128, 192, 512), (3, 64, 32, 64, 64, 128)])
def test_latent_attention_over_long_sequences(shape):
    for cuts in ([5000], [400, 129, 1, 255, 2, 17]):
        err = _run_latent(torch.bfloat16, shape, [1500, 517, 128], cuts, seed=5)
        assert err < LATENT_TOL[torch.bfloat16], (cuts, err)


@pytest.mark.parametrize("fault", ["no_head_sink", "sink_scaled", "no_gate", "half_pairs", "no_yarn", "yarn_scale", "rot_normed", "no_latent_norm"])
def test_latent_attention_inputs_show_a_mistake(fault):
    assert _run_latent(torch.float32, (4, 32, 16, 40, 72, 48), [150], [1000], seed=3, faults=(fault,)) > 0.3


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("M,N,K,H,gated", [(5, 48, 32, 4, 0), (130, 512, 128, 3, 0), (1, 13, 21, 2, 1), (200, 128, 64, 8, 1), (70, 72, 24, 5, 1)])
def test_products_per_head(dtype, M, N, K, H, gated):
    from arctic_platform_b200.ops import serving
    rnd = _gen(M)
    step, out_step = _pad8(K) + 8, _pad8(N) + (0 if gated else 16)
    a, w = rnd(M, H * step).to(dtype), torch.zeros(H * N, _pad8(K), dtype=dtype)
    w[:, :K] = rnd(H * N, K, std=K ** -0.5).to(dtype)
    gate = rnd(M, H * out_step + 8).to(dtype).cuda() if gated else None
    out = torch.full((M, H * out_step), 3.0, device="cuda", dtype=dtype)
    serving.heads_linear(a.cuda(), step, w.cuda(), H, K, out, out_step, gate)
    for h in range(H):
        ref = a[:, h * step:h * step + K].double() @ w[h * N:(h + 1) * N, :K].double().t()
        if gated:
            ref = ref * oracle.sigmoid(gate[:, h * out_step:h * out_step + N].cpu().double())
        assert _rel(out[:, h * out_step:h * out_step + N].cpu(), ref) < {torch.float32: 1e-5, torch.bfloat16: 0.03}[dtype]
        assert (out[:, h * out_step + N:(h + 1) * out_step] == 3).all()


# ---------------------------------------------------------------------------- feed-forward
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,W,E,ident,top,ff,decided", [(9, 64, 6, 3, 3, 48, 0), (1, 128, 5, 0, 2, 64, 0), (200, 74, 3, 4, 5, 22, 0),
                                                        (300, 256, 40, 24, 8, 64, 0), (37, 64, 100, 60, 32, 16, 0), (64, 64, 1, 1, 1, 32, 0),
                                                        (500, 128, 8, 2, 2, 96, 1), (2, 2048, 64, 16, 6, 768, 0), (20, 64, 500, 12, 4, 16, 0)])
def test_mixture_of_experts(dtype, T, W, E, ident, top, ff, decided):
    """Routed, identity and shared parts; every weight, rows that are not live, experts without rows, one expert with all rows."""
    from arctic_platform_b200.models.titatar import LayerSpec, MoeSpec, RotSpec, TitatarConfig, WindowAttnSpec, _Mixture
    from arctic_platform_b200.ops import _lib, serving
    rnd = _gen(T)
    cfg = TitatarConfig(8, W, (LayerSpec(WindowAttnSpec(1, 1, 8, 8, 1.0, 0, RotSpec(0, 1.0)), MoeSpec(E, ident, top, ff)),), 1e-5)
    mk = lambda *s: torch.nn.Parameter(torch.zeros(*s, device="cuda", dtype=dtype), requires_grad=False)
    moe = _Mixture(cfg, cfg.layers[0].mlp, mk)
    w = {"correction": rnd(E + ident, std=0.1), "router": torch.zeros(E + ident, W)}
    if decided:
        w["correction"] = torch.arange(E + ident).float()
    for e in range(E):
        w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"] = rnd(ff, W, std=W ** -0.5), rnd(ff, W, std=W ** -0.5), rnd(W, ff, std=ff ** -0.5)
    for n in w:
        w[n] = w[n].to(dtype)
        moe.place(n).copy_(w[n])
    h, z = rnd(T, W).to(dtype), rnd(T, E + ident, std=2.0)
    p = oracle.route(z.double(), w["correction"].double(), top)
    live = torch.ones(T, dtype=torch.bool)
    live[3::7] = False
    y = p[:, E:].sum(-1, keepdim=True) * h.double()
    for e in range(E):
        y += p[:, e:e + 1] * oracle.glu({k: v.double() for k, v in w.items()}, f"e{e}.", h.double())
    pages, _ = _pages([T])
    b = _batch([(0, np.zeros(T), 0)], pages)
    b.kv_slot = torch.where(live, 1, -1).int().cuda()
    for rnd_ in range(2):                                             # the counters are zero again for the second call
        mix = serving.experts(b, h.cuda(), z.cuda(), moe.correction, moe.counters, moe.w_gu, moe.w_down, E + ident, E, top, ff)
        x = torch.zeros(T, W, device="cuda")
        out = serving.residual_step(x, None, None, None, 1e-5, mix=mix, dtype=dtype, write=False).cpu()
        assert (moe.counters == 0).all()
        err = (out.double() - y)[live].abs().max() / y.pow(2).mean().sqrt()
        assert err < {torch.float32: 1e-5, torch.bfloat16: 0.06}[dtype], err
        s, wt = mix.slots.cpu(), mix.weights.cpu()
        chosen = torch.zeros(T, dtype=torch.int32) + (s >= 0).sum(-1)
        assert (chosen[live] == (p[:, :E] > 0).sum(-1)[live]).all() and (chosen[~live] == 0).all()
        used = s[s >= 0]
        assert sorted(used.tolist()) == list(range(len(used)))        # every slot once, no gaps
        assert torch.allclose((wt * (s >= 0)).sum(-1)[live].double(), p[:, :E].sum(-1)[live], atol=1e-6)
    _lib.check_status("mixture of experts")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("M,N,K", [(1, 64, 96), (5, 130, 74), (130, 272, 256), (300, 40, 50), (64, 2048, 512)])
def test_gated_silu(dtype, M, N, K):
    from arctic_platform_b200.ops import serving
    rnd = _gen(M)
    a, w = rnd(M, K).to(dtype), rnd(N, K, std=2 * K ** -0.5).to(dtype)
    z = a.double() @ w.double().t()
    want = z[:, 0::2] * oracle.sigmoid(z[:, 0::2]) * z[:, 1::2]
    out = torch.zeros(M, N // 2 + 16, device="cuda", dtype=dtype)
    serving.gate_up_silu(a.cuda(), w.cuda(), out[:, 8:8 + N // 2])
    assert _rel(out[:, 8:8 + N // 2].cpu(), want) < {torch.float32: 3e-5, torch.bfloat16: 0.03}[dtype]
    assert (out[:, :8] == 0).all() and (out[:, 8 + N // 2:] == 0).all()
