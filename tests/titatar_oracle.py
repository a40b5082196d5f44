"""Plain, slow Titatar decoder: the oracle of the kernel and engine tests.

One function per mechanism, each written as the textbook expression over ONE whole sequence (no cache, no absorbed
projections, no blocks, no batching, experts one by one), in the dtype of its inputs -- the tests use float64 on the CPU.  It
shares no code with the package.  ``forward(cfg, tensors, tokens)`` takes the parsed config.json and the checkpoint's tensors
by name and returns ``(logits [T, V], residual stream after every layer run [runs, T, width])``.

``faults`` (a set of names) plants a deliberate mistake, so that a test can show that its inputs would reveal one:
``window_early`` / ``window_late`` (the window one token shorter / longer), ``no_window``, ``no_sink``, ``no_head_sink``,
``sink_scaled`` (a learned sink multiplied like a score), ``no_gate``, ``head_norm`` (q and k normalised per head), ``norm_after_rotation``, ``neighbour_pairs`` (pairs (2i, 2i + 1) in the
grouped attention), ``half_pairs`` (pairs (i, i + dims/2) in the latent attention), ``no_yarn``, ``no_yarn_gain``,
``yarn_scale`` (the score scale multiplied by the squared gain too), ``first_rotated`` (the rotated part in front of a query
head), ``rot_normed`` (the norm of the latent spans the rotated key part), ``no_latent_norm``, ``plain_gain`` (layer norms
without the one), ``no_post_norm``, ``no_loop_input``, ``loop_input_every_layer``, ``loop_input_first`` (added before the first
pass too), ``shared_pass_keys`` (every pass of a looped layer sees the first pass's keys), ``no_correction``,
``corrected_weights``, ``renormed``, ``scores_of_experts`` (softmax without the identity experts), ``no_identity``,
``no_shared``."""
from __future__ import annotations

import math

import torch


def rms(x, eps):
    """x divided by its root mean square over the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def layer_norm(x, w, eps, faults=()):
    """Weight stored around zero."""
    return rms(x, eps) * (w if "plain_gain" in faults else 1.0 + w)


# ---------------------------------------------------------------------------- rotation
def frequencies(rot, faults=()):
    """``(frequencies, gain of cos and sin)``; YaRN blends every frequency between itself and itself / factor."""
    dims, base, sc = rot["dims"], float(rot["base"]), rot.get("scaling")
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not sc or "no_yarn" in faults:
        return f, 1.0

    def dim(turns):
        return dims * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo, hi = max(math.floor(dim(sc["fast"])), 0), min(math.ceil(dim(sc["slow"])), dims - 1)
    out = []
    for i, v in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(v / sc["factor"] * r + v * (1.0 - r))
    return out, 1.0 if "no_yarn_gain" in faults else 0.1 * math.log(sc["factor"]) + 1.0


def rotate(x, positions, rot, neighbours, faults=()):
    """``x [T, H, D]``: the first dims of every head, pairs (2i, 2i + 1) or (i, i + dims/2)."""
    y = x.clone()
    half = rot["dims"] // 2
    freqs, gain = frequencies(rot, faults)
    for i, f in enumerate(freqs):
        a = positions.to(torch.float64) * f
        c, s = (torch.cos(a) * gain).to(x.dtype)[:, None], (torch.sin(a) * gain).to(x.dtype)[:, None]
        m, n = (2 * i, 2 * i + 1) if neighbours else (i, i + half)
        y[..., m] = x[..., m] * c - x[..., n] * s
        y[..., n] = x[..., n] * c + x[..., m] * s
    return y


# ---------------------------------------------------------------------------- attention
def visible(T, window, faults=()):
    """``[T, T]`` bool: key j of query i with 0 <= i - j < window (0: plain causal)."""
    d = torch.arange(T)[:, None] - torch.arange(T)[None]
    seen = d >= 0
    if window and "no_window" not in faults:
        seen = seen & (d < window - ("window_early" in faults) + ("window_late" in faults))
    return seen


def sink_softmax(s, seen, sink):
    """``s [T, T]``; ``sink`` (a score without a key, or None) counts once in the denominator."""
    s = torch.where(seen, s, torch.full_like(s, float("-inf")))
    top = s.max(-1, keepdim=True).values
    if sink is not None:
        top = torch.clamp(top, min=float(sink))
    p = torch.exp(s - top)
    den = p.sum(-1, keepdim=True)
    if sink is not None:
        den = den + torch.exp(sink - top)
    return p / den


def attention_mixer(m, W, p, h, eps, faults=(), held=None):
    """``held``: dict in which a pass finds (or leaves) the keys and values of the first one (fault ``shared_pass_keys``)."""
    T, H, G, D = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    pos = torch.arange(T)
    q, k, v = (h @ W[p + n].t() for n in "qkv")
    wq, wk = W[p + "q.norm"], W[p + "k.norm"]
    near = "neighbour_pairs" in faults
    if "norm_after_rotation" in faults:
        q = rms(rotate(q.view(T, H, D), pos, m["rot"], near).reshape(T, -1), eps) * wq
        k = rms(rotate(k.view(T, G, D), pos, m["rot"], near).reshape(T, -1), eps) * wk
        q, k = q.view(T, H, D), k.view(T, G, D)
    else:
        if "head_norm" in faults:
            q, k = rms(q.view(T, H, D), eps).reshape(T, -1) * wq, rms(k.view(T, G, D), eps).reshape(T, -1) * wk
        else:
            q, k = rms(q, eps) * wq, rms(k, eps) * wk
        q, k = rotate(q.view(T, H, D), pos, m["rot"], near), rotate(k.view(T, G, D), pos, m["rot"], near)
    v = v.view(T, G, m["vdim"])
    if held is not None:
        k, v = held.setdefault(p, (k, v))
    seen = visible(T, (m.get("mask") or {}).get("size", 0), faults)
    gate = sigmoid(h @ W[p + "g"].t())
    out = []
    for i in range(H):
        g = i // (H // G)
        sink = None if "no_sink" in faults else torch.zeros((), dtype=h.dtype)
        o = sink_softmax(q[:, i] @ k[:, g].t() * m["scale"], seen, sink) @ v[:, g]
        out.append(o if "no_gate" in faults else o * gate[:, i:i + 1])
    return torch.cat(out, -1) @ W[p + "o"].t()


def latent_attention_mixer(m, W, p, h, eps, faults=(), held=None):
    T, H, D, R, E, C = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(T)
    cq = rms(h @ W[p + "dq"].t(), eps) * W[p + "dq.norm"]
    q = (cq @ W[p + "uq"].t()).view(T, H, D + R)
    qn, qr = (q[..., R:], q[..., :R]) if "first_rotated" in faults else (q[..., :D], q[..., D:])
    dkv = h @ W[p + "dkv"].t()
    if "rot_normed" in faults:
        dkv = rms(dkv, eps)
        c, kr = dkv[:, :C] * W[p + "dkv.norm"], dkv[:, C:]
    else:
        c, kr = dkv[:, :C], dkv[:, C:]
        if "no_latent_norm" not in faults:
            c = rms(c, eps) * W[p + "dkv.norm"]
    near = "half_pairs" not in faults
    qr = rotate(qr, pos, m["rot"], near, faults)
    kr = rotate(kr[:, None], pos, m["rot"], near, faults)[:, 0]
    if held is not None:
        c, kr = held.setdefault(p, (c, kr))
    k, v = (c @ W[p + "uk"].t()).view(T, H, D), (c @ W[p + "uv"].t()).view(T, H, E)
    scale = m["scale"] * (frequencies(m["rot"])[1] ** 2 if "yarn_scale" in faults else 1.0)
    seen, out = visible(T, 0), []
    for i in range(H):
        sink = None if "no_head_sink" in faults else W[p + "sink"][i] * (scale if "sink_scaled" in faults else 1.0)
        out.append(sink_softmax((qn[:, i] @ k[:, i].t() + qr[:, i] @ kr.t()) * scale, seen, sink) @ v[:, i])
    o = torch.cat(out, -1)
    if "no_gate" not in faults:
        o = o * sigmoid(h @ W[p + "g"].t())
    return o @ W[p + "o"].t()


# ---------------------------------------------------------------------------- feed-forward
def glu(W, p, h):
    g = h @ W[p + "gate"].t()
    return (g * sigmoid(g) * (h @ W[p + "up"].t())) @ W[p + "down"].t()


def route(z, correction, top, faults=()):
    """Logits ``[T, N]`` -> ``[T, N]`` weights, zero for the experts that are not chosen."""
    s = torch.softmax(z, -1)
    pick = s if "no_correction" in faults else s + correction
    idx = torch.argsort(pick, -1, descending=True)[:, :top]
    w = torch.zeros_like(s).scatter(1, idx, (pick if "corrected_weights" in faults else s).gather(1, idx))
    return w / w.sum(-1, keepdim=True) if "renormed" in faults else w


def mixture(m, W, p, h, faults=()):
    r = m["router"]
    n, ident = r["experts"], r.get("identity", 0)
    z = h @ W[p + "router"].t()
    if "scores_of_experts" in faults:
        w = torch.cat([route(z[:, :n], W[p + "correction"][:n], r["top"]), torch.zeros_like(z[:, n:])], 1)
    else:
        w = route(z, W[p + "correction"], r["top"], faults)
    y = torch.zeros_like(h)
    for e in range(n):
        y = y + w[:, e:e + 1] * glu(W, p + f"e{e}.", h)
    if "no_identity" not in faults:
        y = y + w[:, n:n + ident].sum(-1, keepdim=True) * h
    if m.get("shared") and "no_shared" not in faults:
        y = y + glu(W, p + "shared.", h)
    return y


# ---------------------------------------------------------------------------- model
def layer_order(cfg):
    """``(layer, pass)`` in the order of execution; pass is given on a pass's first layer only."""
    n, lp = len(cfg["layers"]), cfg.get("loop")
    a, b, times = (lp["start"], lp["stop"], lp["times"]) if lp else (0, 0, 0)
    return [(i, None) for i in range(a)] + [(i, t if i == a else -1 - t) for t in range(times) for i in range(a, b)] + \
        [(i, None) for i in range(b, n)]


@torch.no_grad()
def forward(cfg, tensors, tokens, dtype=torch.float64, faults=()):
    W = {k: v.to(dtype) if v.is_floating_point() else v for k, v in tensors.items()}
    eps = cfg["norm"]["eps"]
    x = x0 = W["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    after, held = [], {} if "shared_pass_keys" in faults else None
    post = (lambda y, w: y) if "no_post_norm" in faults else (lambda y, w: layer_norm(y, w, eps, faults))
    for i, t in layer_order(cfg):
        s, p = cfg["layers"][i], f"l{i}."
        later = t is not None and (t > 0 or (t == 0 and "loop_input_first" in faults))
        inside = t is not None and t < -1 and "loop_input_every_layer" in faults
        if (later or inside) and "no_loop_input" not in faults:
            x = x + x0
        mixer = attention_mixer if s["type"] == "attention" else latent_attention_mixer
        y = mixer(s["mixer"], W, p + "mix.", layer_norm(x, W[p + "norm1"], eps, faults), eps, faults, held)
        x = x + post(y, W[p + "norm1b"])
        if s.get("mlp") is not None:
            h = layer_norm(x, W[p + "norm2"], eps, faults)
            y = mixture(s["mlp"], W, p + "mlp.", h, faults) if s["mlp"]["kind"] == "moe" else glu(W, p + "mlp.", h)
            x = x + post(y, W[p + "norm2b"])
        after.append(x)
    return layer_norm(x, W["final.norm"], eps, faults) @ W["head"].t(), torch.stack(after)
