"""Small Titatar configurations, random weights and engines for the tests."""
import torch

from tests import titatar_oracle as oracle
from tests.reninex_helpers import TOL, error, feed, save, tokens


def attention(heads=4, kv=2, dim=32, vdim=48, scale=None, window=37, rot=16, base=3000.0):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": 9.0 / dim if scale is None else scale,
         "rot": {"base": base, "dims": rot}}
    if window:
        m["mask"] = {"size": window}
    return {"type": "attention", "mixer": m}


def latent(heads=4, dim=32, rot_dim=16, vdim=40, q_rank=72, kv_rank=48, scale=None, base=2000.0, yarn=(4.0, 64.0, 8.0, 1.0)):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
         "scale": 9.0 / dim if scale is None else scale, "rot": {"base": base, "dims": rot_dim}}
    if yarn:
        m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
    return {"type": "latent_attention", "mixer": m}


def dense(layer, ff=96):
    return {**layer, "mlp": {"kind": "dense", "ff": ff}}


def moe(layer, experts=6, identity=3, top=3, ff=48, shared=40):
    mlp = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "identity": identity, "top": top}}
    if shared:
        mlp["shared"] = {"ff": shared}
    return {**layer, "mlp": mlp}


def bare(layer):
    return {**layer, "mlp": None}


def config(layers, width=128, vocab=200, eps=3e-5, scale=2.5, loop=None):
    d = {"architecture": "Titatar", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale},
         "layers": layers}
    if loop:
        d["loop"] = dict(zip(("start", "stop", "times"), loop))
    return d


CONFIGS = {
    # aligned sizes; every kind of layer, a loop over two of them
    "mixed-layers": config([dense(latent()), moe(attention()), moe(latent(heads=6, vdim=24, q_rank=48, kv_rank=64), shared=0),
                            bare(attention(heads=6, window=21, rot=8)), moe(attention(heads=2, kv=2, window=50), top=1)],
                           loop=(1, 3, 3)),
    # nothing is a multiple of 8; a loop over everything; no identity experts
    "odd-sizes": config([moe(attention(heads=3, kv=1, dim=18, vdim=13, window=19, rot=6), experts=5, identity=0, top=2, ff=30, shared=22),
                         moe(latent(heads=3, dim=14, rot_dim=6, vdim=11, q_rank=29, kv_rank=21, scale=0.6), experts=3, identity=4,
                             top=5, ff=22, shared=0)], width=74, vocab=131, scale=3.0, loop=(0, 2, 2)),
    # no rotation scaling, no window, one head, one pass; a router over more experts than a warp has lanes
    "plain": config([moe(latent(heads=1, dim=24, rot_dim=8, vdim=32, yarn=None), experts=36, identity=5, top=7, ff=16),
                     dense(attention(heads=8, kv=1, dim=16, vdim=24, window=0, rot=0), ff=128)], width=64, vocab=96, loop=(1, 2, 1)),
    # wide heads and latents (several 64-column tiles), nearby windows, a loop at the end
    "wide-heads": config([dense(attention(heads=4, kv=2, dim=128, vdim=128, window=129, rot=96, base=2e5), ff=160),
                          moe(latent(heads=8, dim=128, rot_dim=64, vdim=128, q_rank=192, kv_rank=256, base=2e5, yarn=(8.0, 90.0, 16.0, 2.0)),
                              ff=64, shared=96),
                          moe(attention(heads=4, kv=4, dim=64, vdim=96, window=64, rot=64, base=2e5), ff=64)],
                         width=256, vocab=456, loop=(1, 3, 2)),
    # long windows, so that long-range keys stay visible; a latent as wide as the query's
    "far-keys": config([moe(attention(dim=48, vdim=96, window=300)), dense(latent(dim=64, rot_dim=32, vdim=64, q_rank=128, kv_rank=128), ff=64),
                        moe(latent(heads=16, dim=64, rot_dim=64, vdim=64, q_rank=128, kv_rank=512, yarn=(2.5, 200.0, 4.0, 1.0)), identity=2)],
                       width=160, vocab=320),
}


def weights(cfg, seed=0, decided=False):
    """Random checkpoint tensors (bf16 values).  The key projections repeat rows of the query projections (for latent attention
    in the latents' common columns), so a token that comes back matches itself across any distance; sinks, corrections, identity
    weights and the rotated parts are large enough to show.  ``decided``: corrections so far apart that every token of a layer takes
    the same experts -- a test in 16 bits must not rest on a close call."""
    g = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]
    rnd = lambda *s, std=1.0: (torch.randn(*s, generator=g) * std).to(torch.bfloat16)
    uni = lambda *s, lo=0.0, hi=1.0: (torch.rand(*s, generator=g) * (hi - lo) + lo).to(torch.bfloat16)
    t = {"embed": rnd(V, W, std=0.5), "head": rnd(V, W, std=W ** -0.5), "final.norm": uni(W, lo=-0.3, hi=0.3)}
    std = W ** -0.5

    def glu(p, ff, gain=1.0):
        t[p + "gate"], t[p + "up"] = rnd(ff, W, std=1.5 * std), rnd(ff, W, std=1.5 * std)
        t[p + "down"] = rnd(W, ff, std=gain * ff ** -0.5)

    for i, s in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", s["mixer"], s["mlp"]
        for n in ("norm1", "norm2") if f else ("norm1",):
            t[p + n], t[p + n + "b"] = uni(W, lo=-0.3, hi=0.3), uni(W, lo=-0.6, hi=0.0)
        H, D, E = m["heads"], m["dim"], m["vdim"]
        if s["type"] == "attention":
            G = m["kv_heads"]
            q = rnd(H, D, W, std=std)
            t[p + "mix.q"], t[p + "mix.k"] = q.reshape(-1, W), q[::H // G].reshape(-1, W).clone()
            t[p + "mix.v"] = rnd(G * E, W, std=std)
            t[p + "mix.q.norm"], t[p + "mix.k.norm"] = uni(H * D, lo=0.5, hi=1.5), uni(G * D, lo=0.5, hi=1.5)
            t[p + "mix.g"] = rnd(H, W, std=2 * std)
        else:
            R, Q, C = m["rot_dim"], m["q_rank"], m["kv_rank"]
            r = min(Q, C)
            dq = rnd(Q, W, std=std)
            dkv = rnd(C + R, W, std=std)
            dkv[:r] = dq[:r]
            uk = rnd(H, D, C, std=0.3 * C ** -0.5)
            uk[..., :r] = rnd(H, D, r, std=r ** -0.5)
            uq = rnd(H, D + R, Q, std=1.5 * Q ** -0.5)
            uq[:, :D] = 0
            uq[:, :D, :r] = uk[..., :r]
            t[p + "mix.dq"], t[p + "mix.dkv"], t[p + "mix.uq"], t[p + "mix.uk"] = dq, dkv, uq.reshape(-1, Q), uk.reshape(-1, C)
            t[p + "mix.dq.norm"], t[p + "mix.dkv.norm"] = uni(Q, lo=0.5, hi=1.5), uni(C, lo=0.5, hi=1.5)
            t[p + "mix.uv"] = rnd(H * E, C, std=C ** -0.5)
            t[p + "mix.sink"] = uni(H, lo=3.0, hi=8.0)
            t[p + "mix.g"] = rnd(H * E, W, std=2 * std)
        t[p + "mix.o"] = rnd(W, H * E, std=(H * E) ** -0.5)
        if f and f["kind"] == "dense":
            glu(p + "mlp.", f["ff"])
        elif f:
            r = f["router"]
            n = r["experts"] + r["identity"]
            for e in range(r["experts"]):
                glu(p + f"mlp.e{e}.", f["expert"]["ff"], 3.0)
            t[p + "mlp.router"], t[p + "mlp.correction"] = rnd(n, W, std=1.5 * std), uni(n, lo=-0.3, hi=0.3)
            if decided:
                t[p + "mlp.correction"] = (torch.randperm(n, generator=g) * 1.5).to(torch.bfloat16)
            if f.get("shared"):
                glu(p + "mlp.shared.", f["shared"]["ff"])
    return t


def engine(cfg, tensors, dtype, tokens=2048, slots=4, max_seq_len=1024, **kw):
    from arctic_platform_b200.engine.stateful_sampler import StatefulSampler
    from arctic_platform_b200.models.titatar import TitatarConfig, TitatarLM
    rc = TitatarConfig.from_dict(cfg)
    model = TitatarLM(rc, "cuda", dtype)
    for n, t in tensors.items():
        model.load_named_tensor(n, t)
    return StatefulSampler(rc, "cuda", model=model, kv_cache_tokens=tokens, max_batch=slots, max_seq_len=max_seq_len, **kw)


def expected(cfg, tensors, toks, faults=()):
    return oracle.forward(cfg, tensors, toks, torch.float64, faults)[0]


__all__ = ["CONFIGS", "TOL", "attention", "config", "engine", "error", "expected", "feed", "latent", "oracle", "save", "tokens",
           "weights"]
