"""Small Meronex configurations, random weights and engines for the tests."""
import torch

from tests import meronex_oracle as oracle
from tests.reninex_helpers import TOL, error, feed, save, tokens

RANK = {"odd-sizes": 13, "wide-heads": 72, "long-range": 130}     # of the decay projections (24 elsewhere): in the tensors' shapes only


def mlstm(heads=3, dim=32, vdim=48, cap=7.0):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}}


def delta(heads=4, kv=2, dim=32, vdim=40, taps=3):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": taps}}


def parallel(heads=4, kv=2, dim=32, vdim=48, scale=None, softcap=18.0, rot=16, base=3000.0, yarn=(4.0, 64.0, 8.0, 1.0), r_heads=3,
             r_dim=24):
    left = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": 9.0 / dim if scale is None else scale,
            "rot": {"base": base, "dims": rot}}
    if softcap:
        left["softcap"] = softcap
    if yarn:
        left["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
    return {"type": "parallel", "mixer": {"left": left, "right": {"heads": r_heads, "dim": r_dim}}}


def moe(layer, experts=6, top=2, ff=48, limit=1.3):
    return {**layer, "mlp": {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}}


def bare(layer):
    return {**layer, "mlp": None}


def config(layers, width=128, vocab=200, eps=3e-5, groups=4, mult=0.4):
    return {"architecture": "Meronex", "vocab": vocab, "width": width, "norm": {"eps": eps, "groups": groups}, "residual_mult": mult,
            "layers": layers}


CONFIGS = {
    # aligned sizes; every kind of layer, one without a feed-forward
    "mixed-layers": config([moe(parallel()), moe(mlstm(), top=3), bare(delta()), moe(delta(heads=3, kv=3, dim=48, vdim=32, taps=4), limit=0.8),
                            moe(parallel(heads=6, kv=2, softcap=90.0, r_heads=2, r_dim=40), experts=5, top=1), moe(mlstm(heads=2, vdim=24))]),
    # nothing is a multiple of 8
    "odd-sizes": config([moe(mlstm(heads=3, dim=14, vdim=11, cap=3.5), experts=5, ff=30), moe(delta(heads=3, kv=1, dim=10, vdim=13, taps=5), ff=22),
                         moe(parallel(heads=3, kv=1, dim=18, vdim=13, rot=6, r_heads=3, r_dim=7), experts=3, top=3, ff=18)],
                        width=74, vocab=131, groups=2, mult=0.35),
    # one of everything: one head, one group, one tap, one expert; no rotation scaling, no cap; a router wider than a warp
    "plain": config([moe(delta(heads=1, kv=1, dim=24, vdim=16, taps=1), experts=1, top=1, ff=32), moe(mlstm(heads=1, dim=16, vdim=16), experts=36, top=7, ff=16),
                     bare(parallel(heads=2, kv=2, dim=24, vdim=24, scale=0.15, softcap=0.0, rot=24, yarn=None, r_heads=1, r_dim=16))],
                    width=64, vocab=96, groups=1, mult=1.0),
    # wide heads, values wider than keys and the other way round, rank larger than the heads
    "wide-heads": config([moe(parallel(heads=4, kv=2, dim=128, vdim=128, softcap=40.0, rot=96, base=2e5, yarn=(8.0, 90.0, 16.0, 2.0), r_heads=2, r_dim=64)),
                          moe(delta(heads=4, kv=2, dim=128, vdim=128, taps=4), limit=2.0), moe(mlstm(heads=2, dim=128, vdim=160, cap=15.0)),
                          moe(mlstm(heads=2, dim=136, vdim=64), ff=64), moe(parallel(heads=2, kv=1, dim=64, vdim=96, rot=64, r_heads=1, r_dim=128))],
                         width=256, vocab=456, groups=8),
    # many positions: keys far back beside states that last
    "long-range": config([moe(mlstm(heads=2, dim=64, vdim=64)), moe(parallel(heads=4, kv=1, dim=48, vdim=88, r_heads=2, r_dim=64)),
                          moe(delta(heads=2, kv=2, dim=64, vdim=96))], width=160, vocab=320, groups=5),
}


def weights(cfg, seed=0, decided=False, rank=None):
    """Random checkpoint tensors (bf16 values).  The key projections of attention repeat rows of the query projections, so a token that
    comes back matches itself across any distance; gates, decays and step sizes spread from states that last to states that forget at
    once, and gate biases, bonuses and gains are large enough to show.  ``decided``: one channel of the residual is a constant that the
    router reads, so every token of a layer takes the same experts -- a test in 16 bits must not rest on a close call."""
    g = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]
    rank = rank or next((r for n, r in RANK.items() if cfg is CONFIGS[n]), 24)
    rnd = lambda *s, std=1.0: (torch.randn(*s, generator=g) * std).to(torch.bfloat16)
    uni = lambda *s, lo=0.0, hi=1.0: (torch.rand(*s, generator=g) * (hi - lo) + lo).to(torch.bfloat16)
    std = W ** -0.5
    t = {"embed": rnd(V, W, std=1.5), "head": rnd(V, W, std=std), "final.norm": uni(W, lo=0.6, hi=1.4)}
    if decided:
        t["embed"][:, 0] = 3.0
    for i, s in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", s["mixer"], s["mlp"]
        for n in ("1", "2") if f else ("1",):
            t[p + "norm" + n], t[p + f"rg{n}"], t[p + f"rg{n}.b"] = uni(W, lo=0.6, hi=1.4), rnd(W, W, std=1.5 * std), uni(W, lo=-1.0, hi=2.5)
        if s["type"] == "mlstm":
            H, D, E = m["heads"], m["dim"], m["vdim"]
            for n, rows in (("q", H * D), ("k", H * D), ("v", H * E), ("g", H * E)):
                t[p + "mix." + n] = rnd(rows, W, std=1.5 * std)
            t[p + "mix.o"], t[p + "mix.norm"] = rnd(W, H * E, std=(H * E) ** -0.5), uni(H * E, lo=0.5, hi=1.5)
            t[p + "mix.i"], t[p + "mix.f"] = rnd(H, W, std=3 * std), rnd(H, W, std=2 * std)
            t[p + "mix.i.b"], t[p + "mix.f.b"] = uni(H, lo=-5.0, hi=3.0), uni(H, lo=0.0, hi=5.0)
        elif s["type"] == "delta":
            H, G, D, E, taps = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
            for n, rows in (("q", G * D), ("k", G * D), ("v", H * E)):
                t[p + "mix." + n], t[p + f"mix.{n}.conv"] = rnd(rows, W, std=1.5 * std), rnd(rows, taps, std=taps ** -0.5)
            t[p + "mix.g"], t[p + "mix.o"], t[p + "mix.norm"] = rnd(H * E, W, std=std), rnd(W, H * E, std=(H * E) ** -0.5), uni(E, lo=0.5, hi=1.5)
            t[p + "mix.a"], t[p + "mix.b"] = rnd(H, W, std=std), rnd(H, W, std=2 * std)
            t[p + "mix.A_log"], t[p + "mix.dt_bias"] = uni(H, lo=-1.5, hi=1.0), uni(H, lo=-4.0, hi=1.0)
        else:
            L, R = m["left"], m["right"]
            q = rnd(L["heads"], L["dim"], W, std=std)
            l, r = p + "mix.left.", p + "mix.right."
            t[l + "q"], t[l + "k"] = q.reshape(-1, W), q[::L["heads"] // L["kv_heads"]].reshape(-1, W).clone()
            t[l + "v"] = rnd(L["kv_heads"] * L["vdim"], W, std=2 * std) * uni(L["kv_heads"] * L["vdim"], 1, lo=0.3, hi=2.0)
            t[l + "o"] = rnd(W, L["heads"] * L["vdim"], std=3.0 * (L["heads"] * L["vdim"]) ** -0.5)
            n = R["heads"] * R["dim"]
            for x in "rkvg":
                t[r + x] = rnd(n, W, std=std)
            for x in "rkvgw":
                t[r + "mu." + x] = uni(W)
            t[r + "w1"], t[r + "w2"] = rnd(rank, W, std=2.5 * std), rnd(n, rank, std=1.5 * rank ** -0.5)
            t[r + "w0"], t[r + "u"] = uni(n, lo=-5.0, hi=1.0), rnd(R["heads"], R["dim"], std=2.0)
            t[r + "norm"], t[r + "o"] = uni(n, lo=0.5, hi=1.5), rnd(W, n, std=0.3 * n ** -0.5)
            t[l + "out"], t[r + "out"] = uni(W, lo=0.4, hi=1.6), uni(W, lo=0.4, hi=1.6)
        if f:
            n, ff = f["router"]["experts"], f["expert"]["ff"]
            for e in range(n):
                x = p + f"mlp.e{e}."
                t[x + "gate"], t[x + "up"], t[x + "down"] = rnd(ff, W, std=2 * std), rnd(ff, W, std=2 * std), rnd(W, ff, std=ff ** -0.5)
            t[p + "mlp.router"] = rnd(n, W, std=1.5 * std)
        if decided:
            for n in [k for k in t if k.startswith(p)]:
                leaf = n[len(p):]
                if leaf == "mix.o" or leaf.endswith((".down", "left.out", "right.out")) and not leaf.endswith("right.o"):
                    t[n][0] = 0
            if f:
                t[p + "mlp.router"] = rnd(n_experts := f["router"]["experts"], W, std=0.1 * std)
                t[p + "mlp.router"][:, 0] = torch.randperm(n_experts, generator=g).to(torch.bfloat16) * 0.6 - 0.3 * n_experts
                t[p + "norm2"][0] = 1.0
    return t


def engine(cfg, tensors, dtype, tokens=2048, slots=4, max_seq_len=1024, **kw):
    from arctic_platform_b200.engine.stateful_sampler import StatefulSampler
    from arctic_platform_b200.models.meronex import MeronexConfig, MeronexLM
    rc = MeronexConfig.from_dict(cfg)
    model = MeronexLM(rc, "cuda", dtype)
    for n, t in tensors.items():
        model.load_named_tensor(n, t)
    return StatefulSampler(rc, "cuda", model=model, kv_cache_tokens=tokens, max_batch=slots, max_seq_len=max_seq_len, **kw)


def expected(cfg, tensors, toks, faults=()):
    return oracle.forward(cfg, tensors, toks, torch.float64, faults)[0]


__all__ = ["CONFIGS", "RANK", "TOL", "config", "engine", "error", "expected", "feed", "oracle", "save", "tokens", "weights"]
