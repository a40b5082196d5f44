"""Small Reninex configurations, random weights and engines for the tests."""
import json
from pathlib import Path

import numpy as np
import torch

from tests import reninex_oracle as oracle


def layer(heads=4, kv=2, dim=64, vdim=32, scale=None, r_heads=3, r_dim=32, r_vdim=48, rot=16, base=5000.0,
          decay=None, ls=0.75, rs=0.6, ff=96):
    decay = list(decay) if decay is not None else [1.0 - 0.3 / (2 + 3 * i) for i in range(r_heads)]
    return {"type": "parallel",
            "mixer": {"left": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim,
                               "scale": 12.0 / dim if scale is None else scale},
                      "right": {"heads": r_heads, "dim": r_dim, "vdim": r_vdim, "decay": decay,
                                "rot": {"base": base, "dims": rot}},
                      "left_scale": ls, "right_scale": rs},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(layers, width=128, vocab=200, eps=2e-5, taps=3, bigram=(53, 211, 17), loop=(1, 2, 3)):
    d = {"architecture": "Reninex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if taps:
        d["canon"] = {"taps": taps}
    if bigram:
        d["embedding"] = {"bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))}
    if loop:
        d["loop"] = dict(zip(("start", "stop", "times"), loop))
    return d


CONFIGS = {
    # aligned sizes; different layers, a loop over the middle one
    "mixed-layers": config([layer(), layer(heads=2, kv=2, dim=128, vdim=128, r_heads=2, r_dim=64, r_vdim=64, rot=64, ff=160),
                            layer(heads=6, kv=2, dim=32, vdim=64, ff=64)]),
    # nothing is a multiple of 8; hashing with large multipliers; loop over everything
    "odd-sizes": config([layer(heads=3, kv=1, dim=20, vdim=12, r_heads=3, r_dim=22, r_vdim=10, rot=6, ff=50),
                         layer(heads=3, kv=3, dim=36, vdim=20, r_heads=1, r_dim=18, r_vdim=26, rot=18, ff=None)],
                        width=74, vocab=131, taps=5, bigram=(29, 1000003, 999983), loop=(0, 2, 2)),
    # no loop, no bigram, no input convolutions, unrotated retention, decays 1 and 0
    "bare": config([layer(heads=8, kv=1, dim=16, vdim=16, r_heads=4, r_dim=16, r_vdim=32, rot=0,
                          decay=[1.0, 0.9, 0.0, 0.5], ls=1.0, rs=1.0)], width=64, vocab=96, taps=0, bigram=None, loop=None),
    # wide heads, two taps, a loop that starts with the first layer and leaves one after it
    "wide-heads": config([layer(heads=4, kv=2, dim=96, vdim=96, r_heads=2, r_dim=128, r_vdim=128, rot=96, base=2e5),
                          layer(heads=2, kv=1, dim=192, vdim=160, r_heads=2, r_dim=48, r_vdim=80, rot=48)],
                         width=256, vocab=456, taps=2, loop=(0, 1, 2)),
}


def weights(cfg, seed=0):
    """Random checkpoint tensors (bf16 values).  The key projection of the left mixer repeats rows of the query
    projection, so a token that comes back matches itself across any distance: with the default scale one key then
    weighs about 1 among keys of weight e^-6."""
    g = torch.Generator().manual_seed(seed)
    W, V = cfg["width"], cfg["vocab"]
    rnd = lambda *s, std=1.0: (torch.randn(*s, generator=g) * std).to(torch.bfloat16)
    t = {"embed": rnd(V, W), "head": rnd(V, W, std=W ** -0.5), "final.norm": torch.tensor(1.25, dtype=torch.bfloat16)}
    bg = (cfg.get("embedding") or {}).get("bigram")
    if bg:
        t["bigram"] = rnd(bg["buckets"] + 1, W, std=0.4)
    if cfg.get("loop"):
        t["loop.in"] = torch.cat([rnd(W, W, std=0.3 * W ** -0.5) + torch.eye(W).to(torch.bfloat16),
                                  rnd(W, W, std=0.4 * W ** -0.5)], 1)
        t["loop.step"] = rnd(cfg["loop"]["times"], W, std=0.5)
    for i, s in enumerate(cfg["layers"]):
        p, L, R = f"l{i}.", s["mixer"]["left"], s["mixer"]["right"]
        std = W ** -0.5
        t[p + "norm1"] = torch.tensor(0.9 + 0.1 * i, dtype=torch.bfloat16)
        q = rnd(L["heads"], L["dim"], W, std=std)
        t[p + "mix.left.q"] = q.reshape(-1, W)
        t[p + "mix.left.k"] = q[::L["heads"] // L["kv_heads"]].reshape(-1, W).clone()
        t[p + "mix.left.v"] = rnd(L["kv_heads"] * L["vdim"], W, std=std)
        t[p + "mix.left.pb"] = rnd(L["heads"], std=0.3) - 6.0
        t[p + "mix.left.o"] = rnd(W, L["heads"] * L["vdim"], std=(L["heads"] * L["vdim"]) ** -0.5)
        for n, rows in (("q", R["heads"] * R["dim"]), ("k", R["heads"] * R["dim"]), ("v", R["heads"] * R["vdim"]),
                        ("g", R["heads"] * R["vdim"])):
            t[p + "mix.right." + n] = rnd(rows, W, std=std)
        t[p + "mix.right.o"] = rnd(W, R["heads"] * R["vdim"], std=(R["heads"] * R["vdim"]) ** -0.5)
        if s["mlp"]:
            ff = s["mlp"]["ff"]
            t[p + "mlp.gate"], t[p + "mlp.up"] = rnd(ff, W, std=std), rnd(ff, W, std=std)
            t[p + "mlp.down"] = rnd(W, ff, std=ff ** -0.5)
        if cfg.get("canon"):
            t[p + "canon1"] = rnd(W, cfg["canon"]["taps"], std=0.4)
            if s["mlp"]:
                t[p + "canon2"] = rnd(W, cfg["canon"]["taps"], std=0.4)
    return t


def tokens(cfg, n, seed=0):
    """Random ids in which every seventh token repeats one from far back."""
    r = np.random.default_rng(seed)
    t = r.integers(0, cfg["vocab"], size=n)
    for i in range(7, n, 7):
        t[i] = t[r.integers(0, max(1, i // 3))]
    return t.tolist()


def save(cfg, tensors, path):
    from arctic_platform_b200.models.hf_io import write_safetensors
    path = Path(path)
    path.mkdir(parents=True, exist_ok=True)
    (path / "config.json").write_text(json.dumps(cfg))
    write_safetensors(path / "model.safetensors", tensors)
    return path


def engine(cfg, tensors, dtype, tokens=2048, slots=4, max_seq_len=1024, **kw):
    from arctic_platform_b200.engine.stateful_sampler import StatefulSampler
    from arctic_platform_b200.models.reninex import ReninexConfig, ReninexLM
    rc = ReninexConfig.from_dict(cfg)
    model = ReninexLM(rc, "cuda", dtype)
    for n, t in tensors.items():
        model.load_named_tensor(n, t)
    return StatefulSampler(rc, "cuda", model=model, kv_cache_tokens=tokens, max_batch=slots, max_seq_len=max_seq_len, **kw)


def feed(eng, toks, cuts, slot=None):
    """Feeds a sequence in portions of the given sizes (the last size repeats); logits of every position, on the CPU."""
    s = eng.open_sequence() if slot is None else slot
    out, at, i = [], 0, 0
    while at < len(toks):
        n = min(cuts[min(i, len(cuts) - 1)], len(toks) - at)
        out.append(eng.step([(s, toks[at:at + n], list(range(n)))]).cpu())
        at, i = at + n, i + 1
    if slot is None:
        eng.close_sequence(s)
    return torch.cat(out)


def error(got, want):
    """Largest row error: root mean square of the mean-free difference over that of the expected logits."""
    d = got.double() - want.double()
    d = d - d.mean(-1, keepdim=True)
    w = want.double() - want.double().mean(-1, keepdim=True)
    return float(d.pow(2).mean(-1).sqrt().max() / w.pow(2).mean().sqrt())


TOL = {torch.bfloat16: 0.08, torch.float32: 5e-5}


def expected(cfg, tensors, toks, faults=()):
    return oracle.forward(cfg, tensors, toks, torch.float64, faults)[0]


__all__ = ["CONFIGS", "TOL", "config", "engine", "error", "expected", "feed", "layer", "oracle", "save", "tokens",
           "weights"]
