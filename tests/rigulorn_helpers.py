"""Small Rigulorn configurations, random weights and engines for the tests."""
import torch

from tests import rigulorn_oracle as oracle
from tests.reninex_helpers import TOL, error, feed, save, tokens


def attention(heads=4, kv=2, dim=32, vdim=48, scale=None, cap=6.0, diff=0.25, chunk=70, rot=None, base=3000.0, kv_from=None,
              ff=96, limit=1.5):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": 9.0 / dim if scale is None else scale,
         "softcap": cap, "diff": diff, "mask": {"size": chunk}, "rot": {"base": base, "dims": dim // 4 * 2 if rot is None else rot}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": {"kind": "dense", "ff": ff, "limit": limit} if ff else None}


def mamba(heads=6, vdim=32, state=48, groups=3, taps=4, norm_groups=2, ff=None, limit=2.5):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": taps,
                                        "norm_groups": norm_groups},
            "mlp": {"kind": "dense", "ff": ff, "limit": limit} if ff else None}


def config(layers, width=128, vocab=200, eps=3e-5, streams=3, scale=2.5):
    return {"architecture": "Rigulorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "streams": streams,
            "embedding": {"scale": scale}, "layers": layers}


CONFIGS = {
    # aligned sizes; chunks of different sizes, borrowed keys, every layer with and without a feed-forward
    "mixed-layers": config([attention(), mamba(ff=64), attention(heads=6, chunk=48, ff=None),
                            attention(heads=4, chunk=33, kv_from=2, ff=72, diff=0.6, cap=7.0), mamba(groups=1, norm_groups=3)],
                           streams=3),
    # nothing is a multiple of 8; two taps, one stream, a head per group
    "odd-sizes": config([mamba(heads=3, vdim=10, state=21, groups=3, taps=2, norm_groups=5, ff=50),
                         attention(heads=3, kv=1, dim=18, vdim=13, chunk=37, rot=6, ff=30),
                         attention(heads=2, kv=1, dim=18, vdim=13, chunk=90, rot=6, kv_from=1, ff=None)],
                        width=74, vocab=131, streams=1, scale=3.0),
    # a large cap (running maximum), no rotation, five streams, seven taps
    "large-cap": config([attention(heads=8, kv=1, dim=24, vdim=24, cap=90.0, chunk=64, rot=0, ff=128, scale=0.5),
                         mamba(heads=4, vdim=72, state=16, groups=2, taps=7, norm_groups=1)], width=64, vocab=96, streams=5),
    # wide heads (two 64-column chunks per tile), wide state, four streams, one tap, keys borrowed twice
    "wide-heads": config([mamba(heads=2, vdim=136, state=128, groups=1, taps=1, norm_groups=4),
                          attention(heads=4, kv=4, dim=64, vdim=128, chunk=100, base=2e5, ff=160),
                          attention(heads=4, kv=4, dim=64, vdim=128, chunk=64, base=2e5, kv_from=1, rot=32, ff=96),
                          attention(heads=8, kv=4, dim=64, vdim=128, chunk=129, base=2e5, kv_from=1, rot=32)],
                         width=256, vocab=456, streams=4),
    # long chunks, so that long-range keys stay visible; few streams
    "far-keys": config([attention(dim=48, vdim=96, chunk=4096, ff=64), mamba(heads=8, vdim=64, state=64, groups=2),
                        attention(heads=4, kv=1, dim=16, vdim=24, chunk=512)], width=160, vocab=320, streams=2),
}
# a borrower's rotation is its source's
for _c in CONFIGS.values():
    for _l in _c["layers"]:
        if _l["mixer"].get("kv_from") is not None:
            _l["mixer"]["rot"] = dict(_c["layers"][_l["mixer"]["kv_from"]]["mixer"]["rot"])
            _l["mixer"].update({n: _c["layers"][_l["mixer"]["kv_from"]]["mixer"][n] for n in ("kv_heads", "dim", "vdim")})


def weights(cfg, seed=0):
    """Random checkpoint tensors (bf16 values).  The key projections repeat rows of the query projection (of the borrower too),
    so a token that comes back matches itself across any distance in the dimensions that are not rotated; the second map's
    keys are independent.  Feed-forward inputs are wide enough to reach their limits."""
    g = torch.Generator().manual_seed(seed)
    W, V, S = cfg["width"], cfg["vocab"], cfg["streams"]
    rnd = lambda *s, std=1.0: (torch.randn(*s, generator=g) * std).to(torch.bfloat16)
    uni = lambda *s, lo=0.0, hi=1.0: (torch.rand(*s, generator=g) * (hi - lo) + lo).to(torch.bfloat16)
    t = {"embed": rnd(V, W, std=0.5), "head": rnd(V, W, std=W ** -0.5), "final.norm": uni(W, lo=0.7, hi=1.3)}
    std = W ** -0.5
    for i, s in enumerate(cfg["layers"]):
        p, m = f"l{i}.", s["mixer"]
        t[p + "norm1"] = uni(W, lo=0.7, hi=1.3)
        if s["type"] == "attention":
            H, G, D, E = (m[n] for n in ("heads", "kv_heads", "dim", "vdim"))
            if m.get("kv_from") is None:
                q = rnd(H, 2, D, W, std=std)
                k = q[::H // G].clone()
                k[:, 1] = rnd(G, D, W, std=std)
                t[p + "mix.k"], t[p + "mix.v"] = k.reshape(-1, W), rnd(G * E, W, std=std)
            else:
                k = t[f"l{m['kv_from']}.mix.k"].view(G, 2, D, W)
                q = k.repeat_interleave(H // G, 0).clone() + rnd(H, 2, D, W, std=0.2 * std)
            t[p + "mix.q"] = q.reshape(-1, W)
            for n in ("lq1", "lk1", "lq2", "lk2"):
                t[p + "mix." + n] = rnd(D, std=0.5 * D ** -0.25)
            t[p + "mix.o"] = rnd(W, H * E, std=(H * E) ** -0.5)
        else:
            inner = m["heads"] * m["vdim"]
            ch = inner + 2 * m["groups"] * m["state"]
            t[p + "mix.in"] = rnd(inner + ch + m["heads"], W, std=std)
            t[p + "mix.conv"], t[p + "mix.conv.b"] = rnd(ch, m["conv"], std=0.6), rnd(ch, std=0.2)
            t[p + "mix.dt_bias"] = uni(m["heads"], lo=-4.0, hi=-0.5)
            t[p + "mix.A_log"] = uni(m["heads"], lo=-3.0, hi=1.5)
            t[p + "mix.D"], t[p + "mix.norm"] = rnd(m["heads"]), uni(inner, lo=0.6, hi=1.4)
            t[p + "mix.o"] = rnd(W, inner, std=inner ** -0.5)
        if s["mlp"]:
            ff = s["mlp"]["ff"]
            t[p + "norm2"] = uni(W, lo=0.7, hi=1.3)
            t[p + "mlp.gate"], t[p + "mlp.up"] = rnd(ff, W, std=1.5 * std), rnd(ff, W, std=1.5 * std)
            t[p + "mlp.down"] = rnd(W, ff, std=0.6 * ff ** -0.5)
        for q in (1, 2) if s["mlp"] else (1,):
            t[p + f"hc{q}.in"] = uni(S, lo=0.2, hi=1.0)
            t[p + f"hc{q}.out"] = uni(S, lo=0.4, hi=1.4)
            t[p + f"hc{q}.mix"] = ((torch.eye(S) * 0.5 + torch.rand(S, S, generator=g) / S)).to(torch.bfloat16)
    return t


def engine(cfg, tensors, dtype, tokens=2048, slots=4, max_seq_len=1024, **kw):
    from arctic_platform_b200.engine.stateful_sampler import StatefulSampler
    from arctic_platform_b200.models.rigulorn import RigulornConfig, RigulornLM
    rc = RigulornConfig.from_dict(cfg)
    model = RigulornLM(rc, "cuda", dtype)
    for n, t in tensors.items():
        model.load_named_tensor(n, t)
    return StatefulSampler(rc, "cuda", model=model, kv_cache_tokens=tokens, max_batch=slots, max_seq_len=max_seq_len, **kw)


def expected(cfg, tensors, toks, faults=()):
    return oracle.forward(cfg, tensors, toks, torch.float64, faults)[0]


__all__ = ["CONFIGS", "TOL", "attention", "config", "engine", "error", "expected", "feed", "mamba", "oracle", "save", "tokens",
           "weights"]
